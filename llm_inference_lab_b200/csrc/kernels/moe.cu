// Routed feed-forward layers (a mixture of experts): the router's choice, the layout of the chosen
// (token, expert) pairs in rows grouped by expert, and the weighted sum of the experts' results.
//
//   scores  s = softmax(z) over all experts, or sigmoid(z), z the router's logits in 32-bit
//   choice  the `top` largest scores of a token (ties: the smaller index); with a correction, the `top` largest
//           s + correction; with groups (equal runs of neighbouring experts), among the experts of the `keep` groups
//           whose largest choice score is largest
//   weights the chosen scores s over their sum (+ 1e-20), or (renorm 0) the chosen scores as they are; times `scale`
//   out[t]  = sum over the chosen of weight * expert's result  (+ sigmoid(g_t) * shared expert's result); the plain
//             sum of the results where the weights have multiplied the experts' inputs
// The last experts of a router may be identities, without matrices: their result is the input itself.  They take
// part in the choice like the others and have no place in the grouped layout (pos_of -1).
//
// The grouped matrix products between these kernels read rows through `row_src` and pick a tile's matrix
// by `tile_group` (see the product kernels): pair (t, k) lies at row pos_of[t * top + k] of the grouped
// layout, every expert's rows start on a tile border, unused rows are marked -1.  Where a pair lands inside
// its expert's rows depends on timing; no result does: the sum over a token's experts runs in the order of
// its choice.
#include <cfloat>

#include "common.cuh"

namespace {
constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

// One warp per token.  logits [tokens, ld]: the experts' logits at columns [0, E); column `gate_col` (if
// >= 0) holds the logit of the shared expert's gate.  Both kinds of score grow with the logit, so a choice without
// a correction compares logits.
__global__ void __launch_bounds__(kThreads) moe_route_kernel(int* __restrict__ chosen, float* __restrict__ weight,
                                                             float* __restrict__ shared_gate,
                                                             const float* __restrict__ logits, int ld, int tokens,
                                                             int E, int top, int gate_col, int renorm, int sigmoid,
                                                             const float* __restrict__ correction, int groups, int keep,
                                                             float scale) {
  extern __shared__ float keys[];      // [kWarps][E], then [kWarps][groups]
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * kWarps + warp;
  if (t >= tokens) return;
  float* s = keys + (size_t)warp * E;
  const float* z = logits + (size_t)t * ld;
  // A logit that is no number (a row of padding may hold anything) counts as the smallest number, and a taken
  // expert as less than any, so that every choice names an expert that exists.
  float big = -INFINITY;
  for (int e = lane; e < E; e += 32) {
    const float v = z[e];
    s[e] = v >= -FLT_MAX ? fminf(v, FLT_MAX) : -FLT_MAX;
    big = fmaxf(big, v);
  }
  big = warp_max(big);
  float sum = 1.f;
  if (!sigmoid) {
    sum = 0.f;
    for (int e = lane; e < E; e += 32) sum += expf(z[e] - big);
    sum = warp_sum(sum);
  }
  auto score_of = [&](float logit) { return sigmoid ? 1.f / (1.f + expf(-logit)) : expf(logit - big) / sum; };
  if (correction != nullptr) {
    for (int e = lane; e < E; e += 32) {
      const float v = score_of(s[e]) + correction[e];
      s[e] = v >= -FLT_MAX ? v : -FLT_MAX;
    }
  }
  __syncwarp();
  if (groups > 1 && keep < groups) {
    // every group's largest choice score; the best `keep` groups in turn are marked, the others' experts are out
    float* best_of = keys + (size_t)kWarps * E + (size_t)warp * groups;
    const int size = E / groups;
    for (int g = lane; g < groups; g += 32) {
      float m = -INFINITY;
      for (int e = g * size; e < (g + 1) * size; ++e) m = fmaxf(m, s[e]);
      best_of[g] = m;
    }
    __syncwarp();
    for (int k = 0; k < keep; ++k) {
      float best = -INFINITY;
      int at = groups;
      for (int g = lane; g < groups; g += 32)
        if (best_of[g] > best && best_of[g] < INFINITY) { best = best_of[g]; at = g; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int oa = __shfl_xor_sync(0xffffffffu, at, o);
        if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
      }
      if (lane == 0 && at < groups) best_of[at] = INFINITY;      // kept
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (best_of[e / size] != INFINITY) s[e] = -INFINITY;
    __syncwarp();
  }
  float total = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = E;
    for (int e = lane; e < E; e += 32)
      if (s[e] > best) { best = s[e]; at = e; }       // ascending e: the first of equals stays
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
    }
    float score = score_of(correction != nullptr ? z[min(at, E - 1)] : best);
    if (!(score >= 0.f)) score = 0.f;
    total += score;
    if (lane == 0) {
      chosen[(size_t)t * top + k] = min(at, E - 1);
      weight[(size_t)t * top + k] = score;
      if (at < E) s[at] = -INFINITY;      // taken
    }
    __syncwarp();
  }
  __syncwarp();
  if (renorm) {
    const float inv = scale / (total + 1e-20f);
    for (int k = lane; k < top; k += 32) weight[(size_t)t * top + k] *= inv;
  } else if (scale != 1.f) {
    for (int k = lane; k < top; k += 32) weight[(size_t)t * top + k] *= scale;
  }
  if (lane == 0 && shared_gate != nullptr) shared_gate[t] = gate_col >= 0 ? 1.f / (1.f + expf(-z[gate_col])) : 1.f;
}

// One CTA lays the pairs out: counts per expert, every expert's first row on a border of `tile` rows, the
// expert of every tile (-1 beyond the last used tile), and every pair's row.
__global__ void __launch_bounds__(1024) moe_align_kernel(int* __restrict__ row_src, int* __restrict__ tile_group,
                                                         int* __restrict__ pos_of, const int* __restrict__ chosen,
                                                         int pairs, int E, int tile, int rows_cap) {
  extern __shared__ int counts[];        // [E] counts, then [E] first rows, then [E] cursors
  int* start = counts + E;
  int* cursor = start + E;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x;
  for (int e = tid; e < E; e += blockDim.x) counts[e] = cursor[e] = 0;
  for (int i = tid; i < rows_cap; i += blockDim.x) row_src[i] = -1;
  __syncthreads();
  for (int i = tid; i < pairs; i += blockDim.x) {
    const int e = chosen[i];
    if (e >= 0 && e < E) atomicAdd(&counts[e], 1);
  }
  __syncthreads();
  if (tid == 0) {
    int at = 0;
    for (int e = 0; e < E; ++e) {
      start[e] = at;
      const int tiles = (counts[e] + tile - 1) / tile;
      for (int j = 0; j < tiles; ++j) tile_group[at / tile + j] = e;
      at += tiles * tile;
    }
    for (int j = at / tile; j < rows_cap / tile; ++j) tile_group[j] = -1;
  }
  __syncthreads();
  for (int i = tid; i < pairs; i += blockDim.x) {
    const int e = chosen[i];
    if (e < 0 || e >= E) {
      pos_of[i] = -1;
      continue;
    }
    const int at = start[e] + atomicAdd(&cursor[e], 1);
    pos_of[i] = at;
    row_src[at] = i;
  }
}

// rows of the grouped layout as a matrix of their own (for products that cannot gather): out[r] = x[row_src[r] / top],
// zeros where row_src is -1.  grid (rows); 16 bytes a thread where the rows allow it (`vec`).
template <typename T>
__global__ void __launch_bounds__(128) moe_gather_kernel(T* __restrict__ out, const T* __restrict__ x,
                                                         const int* __restrict__ row_src, int top, int width, int ldx,
                                                         int vec) {
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, src = row_src[r];
  T* dst = out + (size_t)r * width;
  const T* row = src < 0 ? nullptr : x + (size_t)(src / top) * ldx;
  if (vec) {
    constexpr int PER = 16 / sizeof(T);
    for (int i = threadIdx.x; i < width / PER; i += 128)
      reinterpret_cast<uint4*>(dst)[i] = row ? reinterpret_cast<const uint4*>(row)[i] : make_uint4(0, 0, 0, 0);
    return;
  }
  for (int i = threadIdx.x; i < width; i += 128) dst[i] = row ? row[i] : from_f32<T>(0.f);
}

// The part of a token's weight that goes to identity experts (indices from `first` on): the same in every thread.
__device__ __forceinline__ float identity_weight(const int* __restrict__ chosen, const float* __restrict__ wt, int top,
                                                 int first) {
  float total = 0.f;
  for (int k = 0; k < top; ++k)
    if (chosen[k] >= first) total += wt != nullptr ? wt[k] : 1.f;
  return total;
}

// out[t] = sum_k weight[t, k] * y[pos_of[t, k]] (+ shared_gate[t] * shared[t]), all 32-bit; weight null: ones.
// With `chosen`, the experts from `identity_from` on give the input h [tokens, width] back.  grid (tokens).
template <typename T>
__global__ void __launch_bounds__(kThreads) moe_combine_kernel(float* __restrict__ out, const float* __restrict__ y,
                                                               const int* __restrict__ pos_of,
                                                               const float* __restrict__ weight,
                                                               const float* __restrict__ shared,
                                                               const float* __restrict__ shared_gate, int top,
                                                               int width, int vec, const int* __restrict__ chosen,
                                                               int identity_from, const T* __restrict__ h) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int* pos = pos_of + (size_t)t * top;
  const float* wt = weight != nullptr ? weight + (size_t)t * top : nullptr;
  const float id_w = chosen != nullptr ? identity_weight(chosen + (size_t)t * top, wt, top, identity_from) : 0.f;
  if (vec) {      // rows of whole groups of four
    const float gs = shared != nullptr ? (shared_gate != nullptr ? shared_gate[t] : 1.f) : 0.f;
    for (int i = 4 * threadIdx.x; i < width; i += 4 * kThreads) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      auto add = [&](float c, float4 v) {
        acc = make_float4(fmaf(c, v.x, acc.x), fmaf(c, v.y, acc.y), fmaf(c, v.z, acc.z), fmaf(c, v.w, acc.w));
      };
#pragma unroll 2
      for (int k = 0; k < top; ++k)
        if (pos[k] >= 0) add(wt != nullptr ? wt[k] : 1.f, load4(y + (size_t)pos[k] * width + i));
      if (shared != nullptr) add(gs, load4(shared + (size_t)t * width + i));
      if (chosen != nullptr) add(id_w, load4(h + (size_t)t * width + i));
      store4(out + (size_t)t * width + i, acc);
    }
    return;
  }
  const float g = shared != nullptr ? (shared_gate != nullptr ? shared_gate[t] : 1.f) : 0.f;
  for (int i = threadIdx.x; i < width; i += kThreads) {
    float acc = 0.f;
    for (int k = 0; k < top; ++k) {
      const int at = pos[k];
      if (at >= 0) acc = fmaf(wt != nullptr ? wt[k] : 1.f, y[(size_t)at * width + i], acc);
    }
    if (shared != nullptr) acc = fmaf(g, shared[(size_t)t * width + i], acc);
    if (chosen != nullptr) acc = fmaf(id_w, to_f32(h[(size_t)t * width + i]), acc);
    out[(size_t)t * width + i] = acc;
  }
}

// The same sum into a 32-bit stream that is normed as a whole, one pass: v = alpha x[t] + the sum, with the identity
// experts' weights on x[t] itself; x[t] = v / rms(v) * w, and (copy not null) the new x[t] rounded to T.  The shared
// expert's result may be split-K partial products, summed in ascending order.  grid (tokens).
template <typename T, bool VEC>
__global__ void __launch_bounds__(1024) moe_combine_norm_kernel(float* __restrict__ x, T* __restrict__ copy,
                                                                const float* __restrict__ y, const int* __restrict__ pos_of,
                                                                const float* __restrict__ weight,
                                                                const int* __restrict__ chosen, int identity_from,
                                                                const float* __restrict__ shared, int shared_splits,
                                                                long long split_stride,
                                                                const float* __restrict__ shared_gate,
                                                                const T* __restrict__ w, int top, int width, float alpha,
                                                                float eps) {
  __shared__ float scratch[32];
  extern __shared__ __align__(16) float row[];      // [width]: the sum; then the token's places and weights [top] each
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const size_t base = (size_t)t * width;
  // the token's choice is read once, side by side: every later load depends on it
  int* pos = reinterpret_cast<int*>(row + (width + 3) / 4 * 4);
  float* wt = reinterpret_cast<float*>(pos + top);
  float id_w = 0.f;
  for (int k = threadIdx.x; k < top; k += blockDim.x) {
    const float c = weight != nullptr ? weight[(size_t)t * top + k] : 1.f;
    pos[k] = pos_of[(size_t)t * top + k];
    wt[k] = c;
    if (chosen[(size_t)t * top + k] >= identity_from) id_w += c;
  }
  const float keep = alpha + block_sum(id_w, scratch);      // (its barriers also publish the places and weights)
  const float gs = shared_gate != nullptr ? shared_gate[t] : 1.f;
  float ss = 0.f;
  if constexpr (VEC) {
    for (int i = 4 * threadIdx.x; i < width; i += 4 * blockDim.x) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      auto add = [&](float c, float4 v) {
        acc = make_float4(fmaf(c, v.x, acc.x), fmaf(c, v.y, acc.y), fmaf(c, v.z, acc.z), fmaf(c, v.w, acc.w));
      };
      const float4 own = load4(x + base + i);
#pragma unroll 4
      for (int k = 0; k < top; ++k)
        if (pos[k] >= 0) add(wt[k], load4(y + (size_t)pos[k] * width + i));
      if (shared != nullptr) add(gs, sum_splits4(shared, shared_splits, split_stride, base + i));
      add(keep, own);
      store4(row + i, acc);
      ss += acc.x * acc.x + acc.y * acc.y + acc.z * acc.z + acc.w * acc.w;
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
      float acc = 0.f;
      for (int k = 0; k < top; ++k)
        if (pos[k] >= 0) acc = fmaf(wt[k], y[(size_t)pos[k] * width + i], acc);
      if (shared != nullptr) {
        float sum = 0.f;
        for (int s = 0; s < shared_splits; ++s) sum += shared[(size_t)s * split_stride + base + i];
        acc = fmaf(gs, sum, acc);
      }
      acc = fmaf(keep, x[base + i], acc);
      row[i] = acc;
      ss += acc * acc;
    }
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)width + eps);
  if constexpr (VEC) {
    for (int i = 4 * threadIdx.x; i < width; i += 4 * blockDim.x) {
      const float4 v = load4(row + i), g = load4(w + i);
      const float4 r = make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
      store4(x + base + i, r);
      if (copy != nullptr) store4(copy + base + i, r);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
      const float r = row[i] * inv * to_f32(w[i]);
      x[base + i] = r;
      if (copy != nullptr) copy[base + i] = from_f32<T>(r);
    }
  }
}

template <typename T>
int launch_combine_norm(float* x, void* copy, const float* y, const int* pos_of, const float* weight, const int* chosen,
                        int identity_from, const float* shared, int shared_splits, const float* shared_gate, const void* w,
                        int tokens, int top, int width, float alpha, float eps, cudaStream_t stream) {
  const size_t smem = ((size_t)(width + 3) / 4 * 4 + 2 * top) * sizeof(float);
  auto on16 = [](const void* p) { return (((uintptr_t)p) & 15) == 0; };
  const bool vec = width % 4 == 0 && on16(x) && on16(copy) && on16(y) && on16(shared) && on16(w);
  auto kernel = vec ? moe_combine_norm_kernel<T, true> : moe_combine_norm_kernel<T, false>;
  const int per = vec ? (width + 3) / 4 : width;
  const int threads = tokens <= 64 || per < kThreads ? (per >= 1024 ? 1024 : (per + 31) / 32 * 32) : kThreads;
  if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  return (int)lab_launch(kernel, dim3(tokens), dim3(threads), smem, stream, x, (T*)copy, y, pos_of, weight, chosen,
                         identity_from, shared, shared_splits, (long long)tokens * width, shared_gate, (const T*)w, top,
                         width, alpha, eps);
}
}  // namespace

// correction: null or [E] floats added to the scores for the choice; groups (a divisor of E; 1: none), keep: see above.
LAB_EXPORT int lab_moe_route(int* chosen, float* weight, float* shared_gate, const float* logits, int ld, int tokens,
                             int E, int top, int gate_col, int renorm, int sigmoid, const float* correction, int groups,
                             int keep, float scale, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const size_t smem = sizeof(float) * kWarps * (E + (groups > 1 ? groups : 0));
  if (E <= 0 || top <= 0 || top > E || smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  if (groups < 1 || E % groups || keep < 1 || keep > groups || top > keep * (E / groups)) return (int)cudaErrorInvalidValue;
  lab_launch(moe_route_kernel, dim3((tokens + kWarps - 1) / kWarps), dim3(kThreads), smem, stream, chosen, weight,
             shared_gate, logits, ld, tokens, E, top, gate_col, renorm, sigmoid, correction, groups, keep, scale);
  LAB_LAUNCH_CHECK();
}

// rows_cap: rows of the grouped layout, a multiple of `tile` and at least pairs + E * (tile - 1) rounded up to it.
LAB_EXPORT int lab_moe_align(int* row_src, int* tile_group, int* pos_of, const int* chosen, int pairs, int E, int tile,
                             int rows_cap, cudaStream_t stream) {
  if (pairs <= 0) return 0;
  if (tile <= 0 || rows_cap % tile || rows_cap < pairs + E * (tile - 1) || (size_t)3 * E * sizeof(int) > 48 * 1024)
    return (int)cudaErrorInvalidValue;
  lab_launch(moe_align_kernel, dim3(1), dim3(1024), sizeof(int) * 3 * E, stream, row_src, tile_group, pos_of, chosen,
             pairs, E, tile, rows_cap);
  LAB_LAUNCH_CHECK();
}

LAB_EXPORT int lab_moe_gather(void* out, const void* x, const int* row_src, int rows, int top, int width, int ldx,
                              int dtype, cudaStream_t stream) {
  if (rows <= 0) return 0;
  const int per = dtype == LAB_F32 ? 4 : 8;
  const int vec = width % per == 0 && ldx % per == 0 && ((((uintptr_t)out) | ((uintptr_t)x)) & 15) == 0;
  if (dtype == LAB_F32)
    lab_launch(moe_gather_kernel<float>, dim3(rows), dim3(128), 0, stream, (float*)out, (const float*)x, row_src, top,
               width, ldx, vec);
  else
    lab_launch(moe_gather_kernel<__nv_bfloat16>, dim3(rows), dim3(128), 0, stream, (__nv_bfloat16*)out,
               (const __nv_bfloat16*)x, row_src, top, width, ldx, vec);
  LAB_LAUNCH_CHECK();
}

LAB_EXPORT int lab_moe_combine(float* out, const float* y, const int* pos_of, const float* weight, const float* shared,
                               const float* shared_gate, int tokens, int top, int width, const int* chosen,
                               int identity_from, const void* h, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const int vec = width % 4 == 0 &&
                  ((((uintptr_t)out) | ((uintptr_t)y) | ((uintptr_t)shared) | ((uintptr_t)h)) & 15) == 0;
  if (dtype == LAB_F32)
    lab_launch(moe_combine_kernel<float>, dim3(tokens), dim3(kThreads), 0, stream, out, y, pos_of, weight, shared,
               shared_gate, top, width, vec, chosen, identity_from, (const float*)h);
  else
    lab_launch(moe_combine_kernel<__nv_bfloat16>, dim3(tokens), dim3(kThreads), 0, stream, out, y, pos_of, weight, shared,
               shared_gate, top, width, vec, chosen, identity_from, (const __nv_bfloat16*)h);
  LAB_LAUNCH_CHECK();
}

// x[t] = norm(alpha x[t] + the weighted sum) * w; see moe_combine_norm_kernel.
LAB_EXPORT int lab_moe_combine_norm(float* x, void* copy, const float* y, const int* pos_of, const float* weight,
                                    const int* chosen, int identity_from, const float* shared, int shared_splits,
                                    const float* shared_gate, const void* w, int tokens, int top, int width, float alpha,
                                    float eps, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width <= 0 || top <= 0 || (size_t)width * sizeof(float) > 160 * 1024) return (int)cudaErrorInvalidValue;
  if (dtype == LAB_F32)
    return launch_combine_norm<float>(x, copy, y, pos_of, weight, chosen, identity_from, shared, shared_splits, shared_gate,
                                      w, tokens, top, width, alpha, eps, stream);
  return launch_combine_norm<__nv_bfloat16>(x, copy, y, pos_of, weight, chosen, identity_from, shared, shared_splits,
                                            shared_gate, w, tokens, top, width, alpha, eps, stream);
}
