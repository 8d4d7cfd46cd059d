// PTX wrappers shared by the kernels that use the 5th-generation tensor cores of sm_100a:
// mbarriers with bounded waits, TMA tile loads, tensor-memory allocation, loads and stores,
// tcgen05.mma issue and commit, operand descriptors, and the host's tensor-map encoding.
#pragma once
#include <cuda.h>

#include "common.cuh"

// ---- mbarriers --------------------------------------------------------------------------
__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_init_fence() { asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory"); }
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
// CLUSTER: the wait also orders against arrivals from the other CTA of a pair.
template <bool CLUSTER = false>
__device__ __forceinline__ bool mbar_try_wait(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  if constexpr (CLUSTER) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(ok)
        : "r"(smem_u32(bar)), "r"(parity)
        : "memory");
  } else {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(ok)
        : "r"(smem_u32(bar)), "r"(parity)
        : "memory");
  }
  return ok != 0;
}
__device__ __forceinline__ uint64_t global_timer_ns() {
  uint64_t t;
  asm volatile("mov.u64 %0, %globaltimer;" : "=l"(t));
  return t;
}
constexpr unsigned long long LAB_WAIT_LIMIT_NS = 2000000000ull;   // two seconds
// Bounded wait: gives up after `limit_ns`, or as soon as another role of the CTA has given up
// (`abort_flag`), and reports it: the error word says that a wait ran out, and the caller lets
// its role drain instead of touching what it waited for.
template <bool CLUSTER = false>
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag,
                                          unsigned long long limit_ns = LAB_WAIT_LIMIT_NS) {
  if (mbar_try_wait<CLUSTER>(bar, parity)) return true;
  const uint64_t t0 = global_timer_ns();
  for (;;) {
    for (int i = 0; i < 256; ++i)
      if (mbar_try_wait<CLUSTER>(bar, parity)) return true;
    if (*abort_flag) return false;
    if (global_timer_ns() - t0 > limit_ns) {
      *abort_flag = 1;
      lab_set_error(LAB_ERR_WAIT_TIMEOUT);
      return false;
    }
  }
}

// ---- TMA ----------------------------------------------------------------------------------
// One tile of a 2-D tensor map into shared memory; the bytes are counted on `bar`.  x is the
// coordinate along the rows (elements; x times the element size must be a multiple of 16 bytes).
__device__ __forceinline__ void tma_load_2d(uint32_t smem_dst, const CUtensorMap* map, uint64_t* bar, int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];" ::"r"(
          smem_dst),
      "l"(map), "r"(smem_u32(bar)), "r"(x), "r"(y)
      : "memory");
}
__device__ __forceinline__ void tma_load_2d(void* smem_dst, const CUtensorMap* map, uint64_t* bar, int x, int y) {
  tma_load_2d(smem_u32(smem_dst), map, bar, x, y);
}
// Generic-proxy writes to shared memory become visible to the tensor cores and to TMA.
__device__ __forceinline__ void proxy_fence() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

// ---- tensor memory ------------------------------------------------------------------------
__device__ __forceinline__ void tmem_alloc(uint32_t* smem_result, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(smem_result)),
               "r"(ncols)
               : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }

__device__ __forceinline__ void tmem_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// 16 consecutive accumulator columns of this thread's lane, waited for.
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, float* v) {
  uint32_t r[16];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, "
      "[%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr));
  tmem_wait();
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}
// 32 consecutive accumulator columns of this thread's lane; the registers are valid after tmem_wait().
__device__ __forceinline__ void tmem_ld32_issue(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
        "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
        "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr));
}
// 32 consecutive columns of this thread's lane are written from r[0..31]; complete after tmem_st_wait().
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
      "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]),
      "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]),
      "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}

// ---- MMA ----------------------------------------------------------------------------------
// The MMA and commit wrappers are called by every lane of a converged warp with the same
// arguments; one elected lane issues the instruction (measured: about half the issue time of a
// loop that a single lane walks alone).
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "@e tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}" ::"r"(smem_u32(bar))
      : "memory");
}
// D[tmem] (+)= A[smem] * B[smem]^T, bf16 inputs, 32-bit accumulate.
__device__ __forceinline__ void umma_bf16(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc,
                                          uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "@e tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}" ::"r"(tmem_d),
      "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(0u)
      : "memory");
}
// The same with the A operand in tensor memory: lane = row, a 32-bit column holds two consecutive
// bfloat16 elements of K (16 elements of K = 8 columns from a_tmem on).
__device__ __forceinline__ void umma_bf16_tmem_a(uint32_t tmem_d, uint32_t a_tmem, uint64_t desc_b, uint32_t idesc,
                                                 uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "@e tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, {%5, %5, %5, %5}, p;\n\t}" ::"r"(tmem_d),
      "r"(a_tmem), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(0u)
      : "memory");
}
// Shared-memory matrix descriptor of a 128-byte-swizzled tile whose rows are 128 bytes: 8-row groups
// lie 1024 bytes apart (stride byte offset), the leading offset is one 16-byte unit.  The same
// descriptor serves a K-major operand (rows = M or N; 16 elements of K are 32 bytes along the row)
// and an N-major operand (rows = K; a row holds 64 elements of N).
__device__ __forceinline__ uint64_t smem_desc_sw128(uint32_t addr) {
  uint64_t d = 0;
  d |= (uint64_t)((addr & 0x3FFFF) >> 4);  // start address, bits [0, 14)
  d |= (uint64_t)1 << 16;                  // leading byte offset (16 bytes), bits [16, 30)
  d |= (uint64_t)(1024 >> 4) << 32;        // stride byte offset, bits [32, 46)
  d |= (uint64_t)1 << 46;                  // descriptor version of sm_100
  d |= (uint64_t)2 << 61;                  // layout: 128-byte swizzle
  return d;
}
// Instruction descriptor: bf16 x bf16 -> f32, A K-major, M = m (64, 128, or 256 over a pair of CTAs),
// N = n; `b_n_major`: the B operand is N-major instead of K-major.
__host__ __device__ constexpr uint32_t umma_instr_desc(int m, int n, bool b_n_major = false) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((b_n_major ? 1u : 0u) << 16) | ((uint32_t)(n >> 3) << 17) |
         ((uint32_t)(m >> 4) << 24);
}

// ---- small arithmetic ----------------------------------------------------------------------
// silu(g) * u in 32-bit on the accumulators, rounded once by the caller (the reference rounds g, u
// and silu(g) to its storage type first, rust/engine/src/runner/model/qwen2/kernels.rs:1469-1486:
// fewer roundings only come closer to the exact value); exp and the division use the hardware
// approximations (relative error about 2^-21, far below bfloat16's 2^-9).
__device__ __forceinline__ float silu_gate(float g, float u) { return __fdividef(g, 1.f + __expf(-g)) * u; }
// The same with the capped form of the gate (`gate_pair` in common.cuh): `limit` caps g from above and u on both
// sides, the sigmoid reads 1.702 g and u enters as u + 1.
__device__ __forceinline__ float capped_gate(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return __fdividef(g, 1.f + __expf(-1.702f * g)) * (u + 1.f);
}
// The tanh form of GELU of g, times u: 0.5 (1 + tanh(y)) is the sigmoid of 2 y, y = sqrt(2/pi) (g + 0.044715 g^3).
__device__ __forceinline__ float gelu_gate(float g, float u) {
  const float twice = 1.5957691216057308f * fmaf(0.044715f * g * g, g, g);
  return __fdividef(g, 1.f + __expf(-twice)) * u;
}
// By the gate's activation: 1, GELU; 0, SiLU with limit 0 and the capped form with a positive one.
__device__ __forceinline__ float gate_value(float g, float u, int act, float limit) {
  if (act == 1) return gelu_gate(g, u);
  return limit > 0.f ? capped_gate(g, u, limit) : silu_gate(g, u);
}
// 32 accumulator columns of gate (r) and up (ru) to their gated values, every pair multiplied by `scale` first where
// SCALED.  The kind of gate is decided once for all of them.
template <bool SCALED>
__device__ __forceinline__ void gate_columns(float (&v)[32], const uint32_t (&r)[32], const uint32_t (&ru)[32], int act,
                                             float limit, float scale) {
  auto g = [&](int j) { return SCALED ? __uint_as_float(r[j]) * scale : __uint_as_float(r[j]); };
  auto u = [&](int j) { return SCALED ? __uint_as_float(ru[j]) * scale : __uint_as_float(ru[j]); };
  if (act == 0 && !(limit > 0.f)) {
#pragma unroll
    for (int j = 0; j < 32; ++j) v[j] = silu_gate(g(j), u(j));
  } else if (act == 0) {
#pragma unroll
    for (int j = 0; j < 32; ++j) v[j] = capped_gate(g(j), u(j), limit);
  } else {
#pragma unroll
    for (int j = 0; j < 32; ++j) v[j] = gelu_gate(g(j), u(j));
  }
}

// ---- host: tensor maps -----------------------------------------------------------------------
typedef CUresult (*LabEncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                     const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                     CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static inline LabEncodeTiledFn lab_encode_fn() {
  static LabEncodeTiledFn fn = nullptr;
  if (!fn) {
    void* sym = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &q) != cudaSuccess ||
        q != cudaDriverEntryPointSuccess)
      return nullptr;
    fn = (LabEncodeTiledFn)sym;
  }
  return fn;
}

// Map of a row-major bf16 matrix [rows, cols] with row stride ld (elements), 128-byte swizzle;
// box = 64 columns (one swizzled row of 128 bytes) by box_rows rows.  Returns a CUDA error code.
static inline int lab_make_map_bf16(CUtensorMap* map, const void* base, long long rows, long long cols, long long ld,
                                    int box_rows) {
  LabEncodeTiledFn fn = lab_encode_fn();
  if (!fn) return (int)cudaErrorNotSupported;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
  cuuint32_t box[2] = {64u, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : (int)cudaErrorInvalidValue;
}
