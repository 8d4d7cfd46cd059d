// Shared helpers of the sm_100a kernels: storage types, conversions, reductions,
// and the device-side error word.
//
// Storage type T is float or __nv_bfloat16.  Arithmetic that the model's
// numerics depend on (sums, softmax, norms, angles, residual adds) is done in
// float; `store<T>` rounds to nearest even at the operator's edge, as the
// reference rounds to its storage type at every operator boundary
// (rust/engine/README.md:430-447).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define LAB_EXPORT extern "C" __attribute__((visibility("default")))

enum LabDtype : int { LAB_F32 = 0, LAB_BF16 = 1 };

// Error codes a kernel may leave in the error word (first one wins).
enum LabDeviceError : int {
  LAB_OK = 0,
  LAB_ERR_PAGE_RANGE = 1,      // a page or slot index outside the pool
  LAB_ERR_WAIT_TIMEOUT = 2,    // a bounded wait on an mbarrier ran out
  LAB_ERR_ROW_RANGE = 3,       // a gathered row index outside the batch
};

// One copy per shared library (each library is built from one .cu file).
static __device__ int g_lab_error_word;

__device__ __forceinline__ void lab_set_error(int code) { atomicCAS(&g_lab_error_word, 0, code); }

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Round a float to the storage type and back: the value an operator boundary leaves.
template <typename T> __device__ __forceinline__ float round_to(float v) { return to_f32<T>(from_f32<T>(v)); }

// Split-half rotary pair: (lo, hi) are elements i and i + rotary_dim / 2 of a head, (cs, sn) the cosine
// and sine of the pair's angle (rust/engine/src/runner/model/qwen2/kernels.rs:587-631).  One spelling
// for every kernel that rotates, so that all of them round alike.
__device__ __forceinline__ void rope_rotate(float lo, float hi, float cs, float sn, float& out_lo, float& out_hi) {
  out_lo = __fmaf_rn(lo, cs, -__fmul_rn(hi, sn));
  out_hi = __fmaf_rn(hi, cs, __fmul_rn(lo, sn));
}

// The first key a query at position `pos` sees, by the mask's span: 0, every key from 0 on; a positive
// span, the last `span` keys (a sliding window); a negative one, the keys of the query's own chunk of
// -span positions, chunks counted from position 0 of the sequence.  The last key is `pos` in every case.
// Monotonic in `pos`, which the tile loops of the attention kernels rely on.
__host__ __device__ __forceinline__ int lab_first_key(int pos, int span) {
  if (span > 0) return pos - span + 1 > 0 ? pos - span + 1 : 0;
  if (span < 0) return pos < 0 ? 0 : (pos / (-span)) * (-span);
  return 0;
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
// 2^x by the hardware approximation (relative error about 2^-22; -inf gives 0).
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// A score under a soft cap: cap * tanh(raw * scale / cap) in log2 units, by the hardware's 2^x and reciprocal
// approximations (absolute error about 2^-21 of the cap): tanh(y) = 1 - 2 / (1 + e^2y).  cap_log2 = cap * log2(e),
// arg_log2 = 2 * log2(e) * scale / cap.
__device__ __forceinline__ float softcapped_log2(float raw, float arg_log2, float cap_log2) {
  return fmaf(-2.f * cap_log2, __fdividef(1.f, 1.f + fast_exp2(raw * arg_log2)), cap_log2);
}
// ---- thread-block clusters ---------------------------------------------------------------
__device__ __forceinline__ uint32_t cluster_rank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// The address, in the cluster's shared window, of `addr` (shared, this CTA) in CTA `rank` of the cluster.
__device__ __forceinline__ uint32_t map_to_rank(uint32_t addr, int rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
  return r;
}
__device__ __forceinline__ void st_cluster_f32(uint32_t addr, float v) {
  asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(addr), "f"(v) : "memory");
}

// The tanh form of GELU: 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))).  One spelling for the
// activation kernel and the matrix products' epilogues, so that all of them round alike.
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float inner = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
  return 0.5f * z * (1.0f + tanhf(inner));
}

// The activation a plain product's epilogue may apply, by its code: 1 the tanh form of GELU, 2 the square of
// relu (max(z, 0)^2).
__device__ __forceinline__ float lab_act(float z, int code) {
  if (code == 1) return gelu_tanh_f(z);
  const float r = fmaxf(z, 0.f);
  return r * r;
}

// The gate of a gated pair of products.  `act` 1: the tanh form of GELU of g, times u; 0, by the limit: 0, silu(g) *
// u; a positive limit, the capped form with g' = min(g, limit) and u' = clamp(u, -limit, limit): g' * sigmoid(1.702
// g') * (u' + 1).
__device__ __forceinline__ float gate_pair(float g, float u, int act, float limit) {
  if (act == 1) return gelu_tanh_f(g) * u;
  if (limit > 0.f) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
  }
  return g / (1.f + expf(-g)) * u;
}

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a block of up to 1024 threads, same order for every call; `scratch` holds 32 floats.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float t = (lane < nwarps) ? scratch[lane] : 0.f;
  t = warp_sum(t);
  return t;
}

// Two sums over a block at once; `scratch` holds 64 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();
  if (lane == 0) {
    scratch[warp] = a;
    scratch[32 + warp] = b;
  }
  __syncthreads();
  float2 t = lane < nwarps ? make_float2(scratch[lane], scratch[32 + lane]) : make_float2(0.f, 0.f);
  t.x = warp_sum(t.x);
  t.y = warp_sum(t.y);
  return t;
}

// ---- four neighbours at a time (addresses on 16-byte, of bfloat16 8-byte, boundaries) -------
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(q.x << 16), __uint_as_float(q.x & 0xffff0000u), __uint_as_float(q.y << 16),
                     __uint_as_float(q.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
// four entries of `splits` partial products `stride` floats apart, summed in ascending order, eight loads in flight
__device__ __forceinline__ float4 sum_splits4(const float* __restrict__ p, int splits, long long stride, size_t at) {
  if (splits == 1) return load4(p + at);
  float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int s0 = 0; s0 < splits; s0 += 8) {
    float4 v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = s0 + j < splits ? load4(p + (s0 + j) * stride + at) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      t.x += v[j].x;
      t.y += v[j].y;
      t.z += v[j].z;
      t.w += v[j].w;
    }
  }
  return t;
}

#define LAB_LAUNCH_CHECK() return (int)cudaGetLastError()

// ---- programmatic dependent launch --------------------------------------------------------
// Kernels of a step run back to back on one stream, each tiny next to its launch latency.
// Launched with the programmatic-serialization attribute, a kernel may start while its
// predecessor still runs: it signals `pdl_trigger()` at its top (its own successor may be
// scheduled), does whatever does not depend on earlier kernels of the step (barrier set-up,
// prefetch of weights), and calls `pdl_wait()` before it touches anything an earlier kernel
// wrote or may still read.  `pdl_wait()` returns once the predecessor grid has completed and
// its memory is visible; without the launch attribute both are no-ops.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

static int g_lab_pdl = 1;
LAB_EXPORT void lab_set_pdl(int on) { g_lab_pdl = on; }

template <typename... KArgs, typename... Args>
static inline cudaError_t lab_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                     Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = g_lab_pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

// Reads the error word of this library and clears it.  Synchronises the device.
LAB_EXPORT int lab_take_error_word(int* out) {
  int zero = 0;
  cudaError_t e = cudaMemcpyFromSymbol(out, g_lab_error_word, sizeof(int));
  if (e != cudaSuccess) return (int)e;
  return (int)cudaMemcpyToSymbol(g_lab_error_word, &zero, sizeof(int));
}
