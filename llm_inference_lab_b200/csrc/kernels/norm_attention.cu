// Row-wise steps around a softmax attention whose queries and keys are RMS-normed over the whole
// projection (all heads at once) and whose heads' outputs pass a sigmoid gate:
//
//   qk_norm_store   from the fused 32-bit projection [q | k | v | ...] of a step's rows (whole, or as
//                   split-K partial products summed here in ascending order) plus an optional bias:
//                   q <- q / rms(q) * wq, k <- k / rms(k) * wk, each root mean square over the whole
//                   projection of the row; q rounded to T into [tokens, n_q * HD]; k and v rounded into
//                   the row's slot of the paged cache [pages, n_kv, page_size, HD].  A head is stored HD
//                   wide, HD >= max(D, V): the entries beyond a head's own size are zeros, so that heads
//                   whose key and value sizes differ (or are no multiple of the tensor-core tile) run on
//                   the attention kernels built for heads of HD.  A layer that reads another layer's keys
//                   and values has only the q part.  Options: no norms (wq null); a rotation of the first
//                   2 * rot_half entries of every q and k head after the norm, by position * inv_freq[i], either
//                   of entries i and i + rot_half or of neighbours 2i and 2i + 1; and values mixed with those
//                   an earlier layer left of the same rows, v <- (1 - mix) v + mix * v_first (v_first [tokens,
//                   n_kv * V] floats), or left for later layers (v_keep, the same shape, before any rounding).
//   head_gate       out[t, h, i] = attn[t, h, i] * sigmoid(g) * c, g one number per head or per entry,
//                   read from the same projection; the V real entries of each head are packed side by
//                   side and rounded to T for the output projection.
//
// All arithmetic is 32-bit; T says how the weights are stored and how results are rounded.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ float sum_splits(const float* __restrict__ p, int splits, long long stride, size_t at) {
  float total = 0.f;
  for (int s0 = 0; s0 < splits; s0 += 8) {
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = s0 + j < splits ? p[(s0 + j) * stride + at] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) total += v[j];
  }
  return total;
}

struct QkNormParams {
  const float* proj;
  int splits;
  long long split_stride;
  int ld;
  const int* slots;
  int n_q, n_kv, D, V, HD, page_size, num_pages, has_kv, ld_q;
  float eps;
  const int* positions;      // of the rows (rot_half > 0)
  const float* inv_freq;
  int rot_half, rot_pairs;
  float* v_keep;             // or null
  const float* v_first;      // or null
  float v_mix;
};

// entry i of a head whose entries before the norm are `h` (weights w, or null), normed with `inv` and rotated with
// the row's cosines and sines
template <typename T>
__device__ __forceinline__ float normed_rotated(const float* h, const T* w, float inv, int i, const QkNormParams& p,
                                                const float* cs, const float* sn) {
  const float a = w != nullptr ? h[i] * inv * to_f32(w[i]) : h[i];
  if (i >= 2 * p.rot_half) return a;
  const int f = p.rot_pairs ? i >> 1 : (i < p.rot_half ? i : i - p.rot_half);
  const bool low = p.rot_pairs ? !(i & 1) : i < p.rot_half;
  const int mate = p.rot_pairs ? i ^ 1 : (low ? i + p.rot_half : i - p.rot_half);
  const float b = w != nullptr ? h[mate] * inv * to_f32(w[mate]) : h[mate];
  float lo, hi;
  rope_rotate(low ? a : b, low ? b : a, cs[f], sn[f], lo, hi);
  return low ? lo : hi;
}

template <typename T>
__global__ void __launch_bounds__(kThreads) qk_norm_store_kernel(T* __restrict__ q_out, T* __restrict__ cache_k,
                                                                 T* __restrict__ cache_v, const T* __restrict__ bias,
                                                                 const T* __restrict__ wq, const T* __restrict__ wk,
                                                                 QkNormParams p) {
  extern __shared__ float row[];      // [n_q * D + n_kv * (D + V)], cosines [rot_half], sines [rot_half]
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int wq_n = p.n_q * p.D, wk_n = p.has_kv ? p.n_kv * p.D : 0, wv_n = p.has_kv ? p.n_kv * p.V : 0;
  const int total = wq_n + wk_n + wv_n;
  float *cs = row + total, *sn = cs + p.rot_half;
  if (p.rot_half > 0) {
    const float pos = (float)p.positions[t];
    for (int i = threadIdx.x; i < p.rot_half; i += kThreads) sincosf(pos * p.inv_freq[i], &sn[i], &cs[i]);
  }
  float ssq = 0.f, ssk = 0.f;
  for (int i = threadIdx.x; i < total; i += kThreads) {
    float v = sum_splits(p.proj, p.splits, p.split_stride, (size_t)t * p.ld + i);
    if (bias != nullptr) v += to_f32(bias[i]);
    if (i < wq_n) {
      ssq += v * v;
    } else if (i < wq_n + wk_n) {
      ssk += v * v;
    } else {
      const size_t at = (size_t)t * wv_n + i - wq_n - wk_n;
      if (p.v_keep != nullptr) p.v_keep[at] = v;
      if (p.v_first != nullptr) v = (1.f - p.v_mix) * v + p.v_mix * p.v_first[at];
    }
    row[i] = v;
  }
  ssq = block_sum(ssq, scratch);
  const float inv_q = 1.0f / sqrtf(ssq / (float)wq_n + p.eps);
  for (int idx = threadIdx.x; idx < p.n_q * p.HD; idx += kThreads) {
    const int h = idx / p.HD, i = idx - h * p.HD;
    const float v = i < p.D ? normed_rotated(row + h * p.D, wq != nullptr ? wq + h * p.D : nullptr, inv_q, i, p, cs, sn) : 0.f;
    q_out[(size_t)t * p.ld_q + idx] = from_f32<T>(v);
  }
  if (!p.has_kv || cache_k == nullptr) return;
  ssk = block_sum(ssk, scratch);
  const float inv_k = 1.0f / sqrtf(ssk / (float)wk_n + p.eps);
  const int slot = p.slots[t];
  if (slot == -1) return;             // a row of padding: its keys and values go nowhere
  const int page = slot / p.page_size, off = slot - page * p.page_size;
  if (slot < 0 || page >= p.num_pages) {
    if (threadIdx.x == 0) lab_set_error(LAB_ERR_PAGE_RANGE);
    return;
  }
  for (int idx = threadIdx.x; idx < p.n_kv * p.HD; idx += kThreads) {
    const int g = idx / p.HD, i = idx - g * p.HD;
    const size_t dst = (((size_t)page * p.n_kv + g) * p.page_size + off) * p.HD + i;
    const float kv = i < p.D ? normed_rotated(row + wq_n + g * p.D, wk != nullptr ? wk + g * p.D : nullptr, inv_k, i, p,
                                              cs, sn) : 0.f;
    const float vv = i < p.V ? row[wq_n + wk_n + g * p.V + i] : 0.f;
    cache_k[dst] = from_f32<T>(kv);
    cache_v[dst] = from_f32<T>(vv);
  }
}

// the same on four entries i .. i + 3 of a head: all of one half (or whole pairs), the mates likewise side by side
template <typename T>
__device__ __forceinline__ float4 normed_rotated4(const float* h, const T* w, float inv, int i, const QkNormParams& p,
                                                  const float* cs, const float* sn) {
  auto normed = [&](int at) {
    float4 a = load4(h + at);
    if (w != nullptr) {
      const float4 g = load4(w + at);
      a.x = a.x * inv * g.x; a.y = a.y * inv * g.y; a.z = a.z * inv * g.z; a.w = a.w * inv * g.w;
    }
    return a;
  };
  float4 a = normed(i), r;
  if (i >= 2 * p.rot_half) return a;
  if (p.rot_pairs) {
    const int f = i >> 1;
    rope_rotate(a.x, a.y, cs[f], sn[f], r.x, r.y);
    rope_rotate(a.z, a.w, cs[f + 1], sn[f + 1], r.z, r.w);
    return r;
  }
  const bool low = i < p.rot_half;
  const int f = low ? i : i - p.rot_half;
  const float4 b = normed(low ? i + p.rot_half : f), c = load4(cs + f), s = load4(sn + f);
  const float4 lo = low ? a : b, hi = low ? b : a;
  float4 ol, oh;
  rope_rotate(lo.x, hi.x, c.x, s.x, ol.x, oh.x);
  rope_rotate(lo.y, hi.y, c.y, s.y, ol.y, oh.y);
  rope_rotate(lo.z, hi.z, c.z, s.z, ol.z, oh.z);
  rope_rotate(lo.w, hi.w, c.w, s.w, ol.w, oh.w);
  return low ? ol : oh;
}

// qk_norm_store for sizes that are whole groups of four (head sizes, row stride, the rotated half): four entries a
// thread and load, two loads a thread in flight before anything is summed, the angles formed while they arrive, and
// both root mean squares from one block-wide sum.
template <typename T>
__global__ void __launch_bounds__(kThreads) qk_norm_store_vec_kernel(T* __restrict__ q_out, T* __restrict__ cache_k,
                                                                     T* __restrict__ cache_v,
                                                                     const T* __restrict__ bias,
                                                                     const T* __restrict__ wq, const T* __restrict__ wk,
                                                                     QkNormParams p) {
  extern __shared__ __align__(16) float row[];      // as above
  __shared__ float scratch[64];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int wq_n = p.n_q * p.D, wk_n = p.has_kv ? p.n_kv * p.D : 0, wv_n = p.has_kv ? p.n_kv * p.V : 0;
  const int n4 = (wq_n + wk_n + wv_n) / 4;
  float *cs = row + 4 * n4, *sn = cs + p.rot_half;
  const int slot = p.has_kv && cache_k != nullptr ? p.slots[t] : -1;
  float ssq = 0.f, ssk = 0.f;
  bool angles = p.rot_half > 0;
  for (int g0 = threadIdx.x; g0 < n4; g0 += 2 * kThreads) {
    float4 v[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int g = g0 + j * kThreads;
      v[j] = g < n4 ? sum_splits4(p.proj, p.splits, p.split_stride, (size_t)t * p.ld + 4 * g) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (angles) {
      angles = false;
      const float pos = (float)p.positions[t];
      for (int i = threadIdx.x; i < p.rot_half; i += kThreads) sincosf(pos * p.inv_freq[i], &sn[i], &cs[i]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = 4 * (g0 + j * kThreads);
      if (i >= 4 * n4) break;
      float4 a = v[j];
      if (bias != nullptr) {
        const float4 b = load4(bias + i);
        a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
      }
      const float ss = a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
      if (i < wq_n) {
        ssq += ss;
      } else if (i < wq_n + wk_n) {
        ssk += ss;
      } else {
        const size_t at = (size_t)t * wv_n + i - wq_n - wk_n;
        if (p.v_keep != nullptr) store4(p.v_keep + at, a);
        if (p.v_first != nullptr) {
          const float4 f = load4(p.v_first + at);
          const float m = p.v_mix, o = 1.f - p.v_mix;
          a = make_float4(o * a.x + m * f.x, o * a.y + m * f.y, o * a.z + m * f.z, o * a.w + m * f.w);
        }
      }
      store4(row + i, a);
    }
  }
  if (angles) {      // threads without an entry of the row may have an angle to form
    const float pos = (float)p.positions[t];
    for (int i = threadIdx.x; i < p.rot_half; i += kThreads) sincosf(pos * p.inv_freq[i], &sn[i], &cs[i]);
  }
  const float2 ss = block_sum2(ssq, ssk, scratch);
  const float inv_q = 1.0f / sqrtf(ss.x / (float)wq_n + p.eps);
  const int per = p.HD / 4;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int g = threadIdx.x; g < p.n_q * per; g += kThreads) {
    const int h = g / per, i = 4 * (g - h * per);
    store4(q_out + (size_t)t * p.ld_q + 4 * g,
           i < p.D ? normed_rotated4(row + h * p.D, wq != nullptr ? wq + h * p.D : nullptr, inv_q, i, p, cs, sn) : zero);
  }
  if (slot == -1) return;
  const int page = slot / p.page_size, off = slot - page * p.page_size;
  if (slot < 0 || page >= p.num_pages) {
    if (threadIdx.x == 0) lab_set_error(LAB_ERR_PAGE_RANGE);
    return;
  }
  const float inv_k = 1.0f / sqrtf(ss.y / (float)wk_n + p.eps);
  // the last threads first: they are the ones with fewest of q's groups
  for (int g = kThreads - 1 - threadIdx.x; g < 2 * p.n_kv * per; g += kThreads) {
    const bool is_v = g >= p.n_kv * per;
    const int e = is_v ? g - p.n_kv * per : g, h = e / per, i = 4 * (e - h * per);
    T* dst = (is_v ? cache_v : cache_k) + (((size_t)page * p.n_kv + h) * p.page_size + off) * p.HD + i;
    if (is_v) store4(dst, i < p.V ? load4(row + wq_n + wk_n + h * p.V + i) : zero);
    else store4(dst, i < p.D ? normed_rotated4(row + wq_n + h * p.D, wk != nullptr ? wk + h * p.D : nullptr, inv_k, i, p, cs, sn)
                             : zero);
  }
}

template <typename T>
int launch_qk_norm_store(void* q_out, void* cache_k, void* cache_v, const void* bias, const void* wq, const void* wk,
                         const QkNormParams& p, int tokens, size_t smem, cudaStream_t stream) {
  auto on16 = [](const void* a) { return (((uintptr_t)a) & 15) == 0; };
  const bool vec = p.D % 4 == 0 && p.V % 4 == 0 && p.HD % 4 == 0 && p.ld % 4 == 0 && p.split_stride % 4 == 0 &&
                   p.ld_q % 4 == 0 && p.rot_half % (p.rot_pairs ? 2 : 4) == 0 && on16(p.proj) && on16(q_out) && on16(cache_k) &&
                   on16(cache_v) && on16(bias) && on16(wq) && on16(wk) && on16(p.v_keep) && on16(p.v_first);
  auto kernel = vec ? qk_norm_store_vec_kernel<T> : qk_norm_store_kernel<T>;
  if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  lab_launch(kernel, dim3(tokens), dim3(kThreads), smem, stream, (T*)q_out, (T*)cache_k, (T*)cache_v, (const T*)bias,
             (const T*)wq, (const T*)wk, p);
  LAB_LAUNCH_CHECK();
}

template <typename T>
__global__ void __launch_bounds__(kThreads) head_gate_kernel(T* __restrict__ out, int ld_o, const T* __restrict__ attn,
                                                             int ld_a, const float* __restrict__ proj, int splits,
                                                             long long split_stride, int ld, int gate_at,
                                                             int per_head, long long tokens, int n_q, int V, int HD,
                                                             float mult) {
  pdl_trigger();
  pdl_wait();
  const int width = n_q * V;
  const long long n = tokens * width;
  for (long long e = (long long)blockIdx.x * kThreads + threadIdx.x; e < n; e += (long long)gridDim.x * kThreads) {
    const long long t = e / width;
    const int c = (int)(e - t * width), h = c / V, i = c - h * V;
    const float g = sum_splits(proj, splits, split_stride, (size_t)t * ld + gate_at + (per_head ? h : c));
    const float a = to_f32(attn[(size_t)t * ld_a + h * HD + i]);
    out[(size_t)t * ld_o + c] = from_f32<T>(a * mult / (1.0f + expf(-g)));
  }
}

// Two score maps over the same values, combined: a1 - lambda * a2 over its root mean square within the head (V
// entries, eps inside the root), times `mult`, rounded to T and packed for the output projection.  A is how the maps'
// outputs are stored: where lambda is near 1 the difference of two alike maps is small next to their own rounding.  A head's two
// maps lie at heads 2 h and 2 h + 1 of attn (grouped 0) or, with the queries ordered (group, map, head in the group),
// at (2 (h / per) + m) per + h % per (grouped 1, per = heads of a group).  A warp per (row, head).
template <typename T, typename A>
__global__ void __launch_bounds__(kThreads) map_difference_kernel(T* __restrict__ out, const A* __restrict__ attn, int ld_a,
                                                                  int tokens, int H, int V, int HD, int grouped, int per,
                                                                  float lambda, float eps, float mult) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  if (unit >= (long long)tokens * H) return;
  const int t = (int)(unit / H), h = (int)(unit - (long long)t * H);
  const int h1 = grouped ? 2 * (h / per) * per + h % per : 2 * h, h2 = grouped ? h1 + per : h1 + 1;
  const A* a1 = attn + (size_t)t * ld_a + (size_t)h1 * HD;
  const A* a2 = attn + (size_t)t * ld_a + (size_t)h2 * HD;
  constexpr int kPerLane = 8;      // heads of up to 256 entries
  float val[kPerLane], ss = 0.f;
#pragma unroll
  for (int i = 0; i < kPerLane; ++i) {
    const int e = lane + 32 * i;
    val[i] = e < V ? fmaf(-lambda, to_f32(a2[e]), to_f32(a1[e])) : 0.f;
    ss = fmaf(val[i], val[i], ss);
  }
  const float inv = mult / sqrtf(warp_sum(ss) / (float)V + eps);
#pragma unroll
  for (int i = 0; i < kPerLane; ++i) {
    const int e = lane + 32 * i;
    if (e < V) out[((size_t)t * H + h) * V + e] = from_f32<T>(val[i] * inv);
  }
}

int blocks_for(long long n) { return (int)((n + kThreads - 1) / kThreads < 148 * 8 ? (n + kThreads - 1) / kThreads : 148 * 8); }

}  // namespace

// proj: [splits][tokens, ld] floats (splits 1: the whole product); bias over the q, k and v columns or null; wq and wk
// null: no norms.  rot_dims (even, at most D; 0: no rotation) entries of a head turn by positions[t] * inv_freq[i],
// rot_pairs: neighbours, else halves.  v_keep / v_first: see above.
LAB_EXPORT int lab_qk_norm_store(void* q_out, int ld_q, void* cache_k, void* cache_v, const float* proj, int splits,
                                 int ld, const void* bias, const void* wq, const void* wk, const int* slots, int tokens,
                                 int n_q, int n_kv, int D, int V, int HD, int page_size, int num_pages, int has_kv,
                                 float eps, const int* positions, const float* inv_freq, int rot_dims, int rot_pairs,
                                 float* v_keep, const float* v_first, float v_mix, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (HD < D || HD < V || n_q <= 0 || (has_kv && n_kv <= 0)) return (int)cudaErrorInvalidValue;
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > D || (rot_dims > 0 && (positions == nullptr || inv_freq == nullptr)) ||
      (!has_kv && (v_keep != nullptr || v_first != nullptr)) || (has_kv && (wq == nullptr) != (wk == nullptr)))
    return (int)cudaErrorInvalidValue;
  QkNormParams p;
  p.proj = proj; p.splits = splits; p.split_stride = (long long)tokens * ld; p.ld = ld; p.slots = slots;
  p.n_q = n_q; p.n_kv = n_kv; p.D = D; p.V = V; p.HD = HD; p.page_size = page_size; p.num_pages = num_pages;
  p.has_kv = has_kv; p.ld_q = ld_q; p.eps = eps; p.positions = positions; p.inv_freq = inv_freq;
  p.rot_half = rot_dims / 2; p.rot_pairs = rot_pairs; p.v_keep = v_keep; p.v_first = v_first; p.v_mix = v_mix;
  const size_t smem = (size_t)(n_q * D + (has_kv ? n_kv * (D + V) : 0) + rot_dims) * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  if (dtype == LAB_F32) return launch_qk_norm_store<float>(q_out, cache_k, cache_v, bias, wq, wk, p, tokens, smem, stream);
  return launch_qk_norm_store<__nv_bfloat16>(q_out, cache_k, cache_v, bias, wq, wk, p, tokens, smem, stream);
}

// attn: [tokens, ld_a] of T with heads HD wide; the gate's pre-activations start at column gate_at of proj.
LAB_EXPORT int lab_head_gate(void* out, int ld_o, const void* attn, int ld_a, const float* proj, int splits, int ld,
                             int gate_at, int per_head, int tokens, int n_q, int V, int HD, float mult, int dtype,
                             cudaStream_t stream) {
  const long long n = (long long)tokens * n_q * V;
  if (n <= 0) return 0;
  const long long stride = (long long)tokens * ld;
  if (dtype == LAB_F32)
    lab_launch(head_gate_kernel<float>, dim3(blocks_for(n)), dim3(kThreads), 0, stream, (float*)out, ld_o,
               (const float*)attn, ld_a, proj, splits, stride, ld, gate_at, per_head, (long long)tokens, n_q, V, HD, mult);
  else
    lab_launch(head_gate_kernel<__nv_bfloat16>, dim3(blocks_for(n)), dim3(kThreads), 0, stream, (__nv_bfloat16*)out, ld_o,
               (const __nv_bfloat16*)attn, ld_a, proj, splits, stride, ld, gate_at, per_head, (long long)tokens, n_q, V,
               HD, mult);
  LAB_LAUNCH_CHECK();
}

// attn [tokens, ld_a] of T (attn_f32: of floats) with 2 * H heads of HD entries; see map_difference_kernel for their order.
LAB_EXPORT int lab_map_difference(void* out, const void* attn, int ld_a, int tokens, int H, int V, int HD, int grouped,
                                  int per, float lambda, float eps, float mult, int attn_f32, int dtype,
                                  cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (V > 256 || V > HD || H <= 0 || per < 1 || H % per) return (int)cudaErrorInvalidValue;
  const int blocks = (int)(((long long)tokens * H + kThreads / 32 - 1) / (kThreads / 32));
  if (dtype == LAB_F32)
    lab_launch(map_difference_kernel<float, float>, dim3(blocks), dim3(kThreads), 0, stream, (float*)out, (const float*)attn,
               ld_a, tokens, H, V, HD, grouped, per, lambda, eps, mult);
  else if (attn_f32)
    lab_launch(map_difference_kernel<__nv_bfloat16, float>, dim3(blocks), dim3(kThreads), 0, stream, (__nv_bfloat16*)out,
               (const float*)attn, ld_a, tokens, H, V, HD, grouped, per, lambda, eps, mult);
  else
    lab_launch(map_difference_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(blocks), dim3(kThreads), 0, stream, (__nv_bfloat16*)out,
               (const __nv_bfloat16*)attn, ld_a, tokens, H, V, HD, grouped, per, lambda, eps, mult);
  LAB_LAUNCH_CHECK();
}
