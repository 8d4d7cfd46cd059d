// Gated delta rule: a recurrent mixer whose state per head is a matrix S [key channel, value channel] in 32-bit
// floats with a scalar decay, where what the decayed state already holds at a key makes way for the new value:
//
//     S <- g S;    u = beta (v - S^T k);    S <- S + k u^T;    o = S^T q
//
// q and k may be shared by the heads of a group.  Three kernels, all of it 32-bit:
//
//   delta_prepare    from the input projection [q | k | v | ... rates ... decays]: a causal convolution per channel
//                    of q, k, v over the last `taps` inputs (those before a step's first row come from the request's
//                    kept inputs) with SiLU, unit vectors per q and k head, q times a constant, rates sigmoid(b),
//                    decays exp(-exp(A_log) softplus(a + dt_bias)), and the products of a row's q and k with the keys
//                    of its block of four rows.  A row's k, q and products leave as one record in the order the walk
//                    holds them in shared memory, records of a group row after row
//   delta_walk       the recurrence over each request's rows (any number of rows, single tokens included), block of
//                    four rows by block; beside it the request's last taps - 1 inputs replace the kept ones
//   head_norm_gate   every head's output over its own root mean square, a weight all heads share, SiLU(gate)
//
// A block of rows in one go.  Within a block of rows 0..3 let K_i = S^T k_i and Q_i = S^T q_i with the state S before
// the block, G_i the product of the decays up to row i and g_ij that of the decays after row j up to row i.  Then
//
//     u_i = beta_i (v_i - G_i K_i - sum_{j<i} g_ij (k_i . k_j) u_j)
//     o_i = G_i Q_i + sum_{j<=i} g_ij (q_i . k_j) u_j
//     S   <- G_3 S + sum_j g_3j k_j u_j^T
//
// which is the recurrence with its sums regrouped: eight independent products with the old state, a substitution of
// four steps on numbers, one update, instead of four dependent rounds.  Products of decays are formed as products,
// never as quotients, so strong decays lose nothing.  Blocks lie on multiples of four rows of the packed batch and end
// at a request's border; a row that is missing from a block has rate 0 and decay 1.
//
// T says how weights are stored and how the last result is rounded.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;
constexpr int PARTS = 4;        // threads that share one column of the state
constexpr int BLK = 4;          // rows of a block
constexpr int CT = 16;          // rows staged per chunk
constexpr int HELPERS = 64;     // threads that copy chunks ahead and form the blocks' coefficients
constexpr int DOTS = 8;         // q . k_0..3, k . k_0..2 of a row's block, one unused
// coefficients of a block: rates, rates times G, three rows of the substitution, four of the outputs, g_3j, G
// A record: k in PARTS shares of R channels with four floats of padding behind each (zeros beyond the head's
// channels), q likewise, the products.
__host__ __device__ constexpr int share_of(int D) {      // R: the smallest of 4, 8, 16, 32, 64 whose shares hold D channels
  int R = 4;
  while (PARTS * R < D) R *= 2;
  return R;
}
__host__ __device__ constexpr int key_floats(int R) { return PARTS * (R + 4); }
__host__ __device__ constexpr int record_floats(int R) { return 2 * key_floats(R) + DOTS; }
constexpr int C_RATE = 0, C_RG = 4, C_SUB = 8, C_OUT = 20, C_LAST = 36, C_G = 40, COEF = 48;

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit_group() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait_group() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// two 32-bit floats in one 64-bit register, for packed arithmetic
typedef unsigned long long pair_t;
__device__ __forceinline__ pair_t pair_of(float lo, float hi) {
  pair_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ pair_t pair_of(float v) { return pair_of(v, v); }
__device__ __forceinline__ void pair_split(pair_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ float pair_sum(pair_t v) {
  float lo, hi;
  pair_split(v, lo, hi);
  return lo + hi;
}
__device__ __forceinline__ pair_t pair_fma(pair_t a, pair_t b, pair_t c) {
  pair_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ pair_t pair_mul(pair_t a, pair_t b) {
  pair_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// ---- preparation --------------------------------------------------------------------------------
struct PrepareParams {
  const float* proj;     // [tokens, ld]: q at 0 (G * D), k at G * D, v at 2 G D (H * V), rates at b_at, decays at a_at
  int ld, b_at, a_at, taps, H, G, D, V, tokens;
  const float* kept;     // [slots, taps - 1, 2 G D + H V]: a request's last inputs, oldest first
  const int* row_req;
  const int* q_start;
  const int* state_slot;
  int n_slots;
  float q_scale, unit_eps;
  float* rec;            // [G, tokens] records
  int R;
  float* v;              // [tokens, H * V]
  float* decay;          // [H, tokens]
  float* rate;
};

// One warp per (row, unit), the eight warps of a CTA on eight consecutive rows (two blocks) of one unit; neighbouring
// rows read the same inputs.  Units: 0 .. G - 1 the q and k head of a group, then the H value heads, then one for the
// rates and decays of all heads.  A row of padding (state slot -1) leaves as zeros.  TAPS: the number of taps where the
// kernel is built for it (a channel's inputs are then all in flight at once), 0: p.taps.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kThreads) delta_prepare_kernel(const T* __restrict__ taps_w, const T* __restrict__ a_log,
                                                                 const T* __restrict__ dt_bias, PrepareParams p) {
  extern __shared__ float keys[];      // [8][D]: the rows' unit keys (q and k units)
  pdl_trigger();
  pdl_wait();
  constexpr int kPerLane = 8;          // heads of up to 256 key channels
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, unit = blockIdx.y;
  const int t = blockIdx.x * (kThreads / 32) + warp;
  bool live = t < p.tokens;
  const int r = live ? p.row_req[t] : 0, first = live ? p.q_start[r] : 0, slot = live ? p.state_slot[r] : -1;
  const bool padding = slot == -1;
  if (live && !padding && (slot < 0 || slot >= p.n_slots)) {
    if (lane == 0) lab_set_error(LAB_ERR_PAGE_RANGE);
    live = false;
  }
  const int K = TAPS > 0 ? TAPS : p.taps, gd = p.G * p.D, C = 2 * gd + p.H * p.V;
  const float* kept = p.kept + (padding ? 0 : (size_t)slot * (K - 1) * C);
  auto channel = [&](int c) {      // the convolution's output of one channel, through SiLU
    if (padding || !live) return 0.f;
    auto input = [&](int jj) {      // the last tap meets the row itself
      const int src = t - (K - 1) + jj;
      return src >= first ? p.proj[(size_t)src * p.ld + c] : kept[(size_t)((K - 1) + (src - first)) * C + c];
    };
    float acc = 0.f;
    if constexpr (TAPS > 0) {
      float u[TAPS], w[TAPS];
#pragma unroll
      for (int jj = 0; jj < TAPS; ++jj) u[jj] = input(jj), w[jj] = to_f32(taps_w[(size_t)c * TAPS + jj]);
#pragma unroll
      for (int jj = 0; jj < TAPS; ++jj) acc = fmaf(w[jj], u[jj], acc);
    } else {
      for (int jj = 0; jj < K; ++jj) acc = fmaf(to_f32(taps_w[(size_t)c * K + jj]), input(jj), acc);
    }
    return silu_f(acc);
  };
  if (unit < p.G) {
    float qv[kPerLane], kv[kPerLane], qq = 0.f, kk = 0.f;
#pragma unroll
    for (int i = 0; i < kPerLane; ++i) {
      const int e = lane + 32 * i;
      qv[i] = kv[i] = 0.f;
      if (e < p.D) qv[i] = channel(unit * p.D + e), kv[i] = channel(gd + unit * p.D + e);
      qq = fmaf(qv[i], qv[i], qq);
      kk = fmaf(kv[i], kv[i], kk);
    }
    const float q_mult = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), k_mult = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
    const int R = p.R, RS = R + 4, NP = key_floats(R);
    float* rec = p.rec + ((size_t)unit * p.tokens + t) * record_floats(R);
#pragma unroll
    for (int i = 0; i < kPerLane; ++i) {
      const int e = lane + 32 * i;
      if (e >= p.D) break;
      qv[i] *= q_mult, kv[i] *= k_mult;
      keys[warp * p.D + e] = kv[i];
      const int place = e / R * RS + e % R;
      if (live) rec[place] = kv[i], rec[NP + place] = qv[i];
    }
    if (live)
      for (int i = lane; i < NP; i += 32)
        if (i % RS >= R || i / RS * R + i % RS >= p.D) rec[i] = rec[NP + i] = 0.f;
    __syncthreads();
    if (!live) return;
    // products with the keys of the block's rows up to this one, as far as they are the request's own
    const int at = warp % BLK;
    for (int j = 0; j < BLK; ++j) {
      const bool own = j <= at && t - at + j >= first;
      float a = 0.f, b = 0.f;
      if (own) {
        const float* key = keys + (warp - at + j) * p.D;
#pragma unroll
        for (int i = 0; i < kPerLane; ++i) {
          const int e = lane + 32 * i;
          if (e >= p.D) break;
          a = fmaf(qv[i], key[e], a);
          b = fmaf(kv[i], key[e], b);
        }
      }
      a = warp_sum(a);
      b = warp_sum(b);
      if (lane == 0) {
        float* dst = rec + 2 * NP;
        dst[j] = a;
        dst[BLK + j] = j < at ? b : 0.f;
      }
    }
  } else if (!live) {
    return;
  } else if (unit < p.G + p.H) {
    const int at = (unit - p.G) * p.V;
    for (int e = lane; e < p.V; e += 32) p.v[(size_t)t * p.H * p.V + at + e] = channel(2 * gd + at + e);
  } else {
    for (int h = lane; h < p.H; h += 32) {
      const float dt = softplus_f(p.proj[(size_t)t * p.ld + p.a_at + h] + to_f32(dt_bias[h]));
      p.decay[(size_t)h * p.tokens + t] = padding ? 0.f : expf(-expf(to_f32(a_log[h])) * dt);
      p.rate[(size_t)h * p.tokens + t] = padding ? 0.f : sigmoid_f(p.proj[(size_t)t * p.ld + p.b_at + h]);
    }
  }
}

// ---- the walk -----------------------------------------------------------------------------------
struct WalkParams {
  float* out;            // [tokens, H * V]
  const float* rec;      // [G, tokens] records
  const float* v;        // [tokens, H * V]
  const float* decay;    // [H, tokens]
  const float* rate;
  int tokens;
  float* state;          // [slots, H, D, V]
  const int* q_start;
  const int* state_slot;
  int n_slots, H, G, D, V, write;
  int vec;               // rows of v may be copied 16 bytes at a time
  // the inputs a request keeps (null: none)
  const float* proj;
  float* kept;           // [slots, keep, channels]
  int ld, keep, channels;
};

// grid (slices of V, heads, requests).  Walkers (the first PARTS * Vs / NC threads): thread (j, part) keeps rows
// part * R .. part * R + R - 1 of NC neighbouring columns of the state in registers, as pairs of rows for packed
// multiply-adds; keys and queries come from shared memory four rows at a time (the parts' shares lie R + 4 floats
// apart, which spreads their 16-byte loads over the banks).  The four threads of a column share its sums: the keys'
// by two levels of shuffles, the queries' by an exchange that leaves thread p the sums of row p, whose output it
// forms and writes.  Helpers copy chunks of 16 rows two ahead (three buffers, one barrier of the CTA a chunk) and form
// the coefficients of the next chunk's blocks.
template <int R, int NC>
__global__ void __launch_bounds__(256) delta_walk_kernel(WalkParams p, int Vs) {
  extern __shared__ __align__(16) float smem[];
  constexpr int RS = R + 4;                      // floats between two threads' shares of a row's keys
  constexpr int NP = key_floats(R), REC = record_floats(R);
  pdl_trigger();
  const int walkers = PARTS * Vs / NC;
  const int h = blockIdx.y, r = blockIdx.z, g = h / (p.H / p.G);
  const bool helper = (int)threadIdx.x >= walkers;
  const int tid = helper ? threadIdx.x - walkers : threadIdx.x;      // index within the walkers or the helpers
  const int t0 = p.q_start[r], t1 = p.q_start[r + 1];
  const int slot = p.state_slot[r];
  if (t1 <= t0 || slot == -1) {      // nothing to do, or rows of padding (their output is never read)
    pdl_wait();
    return;
  }
  if (slot < 0 || slot >= p.n_slots) {
    if (threadIdx.x == 0) lab_set_error(LAB_ERR_PAGE_RANGE);
    pdl_wait();
    return;
  }
  // a chunk in shared memory: CT records, CT rows of Vs values, CT decays, CT rates, the blocks' coefficients
  const int off_v = CT * REC, off_d = off_v + CT * Vs, off_c = off_d + 2 * CT;
  const int buf_floats = off_c + (CT / BLK) * COEF;
  pdl_wait();

  const int base_row = t0 / BLK * BLK;           // blocks lie on multiples of BLK rows of the batch
  const int n_chunks = (t1 - base_row + CT - 1) / CT;
  const int col0 = blockIdx.x * Vs, v_cols = min(Vs, p.V - col0);
  auto buffer = [&](int chunk) { return smem + (chunk % 3) * buf_floats; };

  // ---- helpers' pieces ----
  auto issue = [&](int chunk) {
    const int row0 = base_row + chunk * CT, lo = max(t0 - row0, 0), cnt = min(CT, t1 - row0) - lo;
    float* base = buffer(chunk);
    const float* rec = p.rec + ((size_t)g * p.tokens + row0 + lo) * REC;
    for (int e = tid; e < cnt * (REC / 4); e += HELPERS) cp_async16(base + lo * REC + 4 * e, rec + 4 * e);
    const float* v0 = p.v + ((size_t)(row0 + lo) * p.H + h) * p.V + col0;
    const size_t ld_v = (size_t)p.H * p.V;
    float* v_to = base + off_v + lo * Vs;
    const int per = HELPERS / CT, tt = tid / per;      // helpers per row of values
    if (tt < cnt) {
      if (p.vec)
        for (int c = tid % per; c < v_cols / 4; c += per) cp_async16(v_to + tt * Vs + 4 * c, v0 + tt * ld_v + 4 * c);
      else
        for (int c = tid % per; c < v_cols; c += per) cp_async4(v_to + tt * Vs + c, v0 + tt * ld_v + c);
    }
    if (tid < 2 * cnt) {
      const int which = tid >= cnt, j = tid - which * cnt;
      cp_async4(base + off_d + which * CT + lo + j, (which ? p.rate : p.decay) + (size_t)h * p.tokens + row0 + lo + j);
    }
    // rows missing from a block of this chunk: zeros, so that what lies there cannot be no number
    const int end = lo + cnt, live_end = (end + BLK - 1) / BLK * BLK;
    for (int row = 0; row < live_end; ++row) {
      if (row >= lo && row < end) continue;
      for (int i = tid; i < REC; i += HELPERS) base[row * REC + i] = 0.f;
      for (int i = tid; i < Vs; i += HELPERS) base[off_v + row * Vs + i] = 0.f;
    }
  };
  // after the copies of `chunk` have landed for every helper: the coefficients of its blocks, a thread per pair of
  // rows of a block
  auto coefficients = [&](int chunk) {
    asm volatile("bar.sync 1, %0;" ::"n"(HELPERS) : "memory");      // the helpers alone
    if (tid >= CT * BLK) return;
    const int row0 = base_row + chunk * CT, blk = tid / (BLK * BLK), i = tid / BLK % BLK, j = tid % BLK;
    float* base = buffer(chunk);
    float* cf = base + off_c + blk * COEF;
    auto valid = [&](int m) { const int row = row0 + blk * BLK + m; return row >= t0 && row < t1; };
    const float* dots = base + (blk * BLK + i) * REC + 2 * NP;
    const bool own = valid(i);
    const float beta = own ? base[off_d + CT + blk * BLK + i] : 0.f;
    float G = 1.f, gij = 1.f, last = 1.f;      // products of the decays up to i, after j up to i, after i
#pragma unroll
    for (int m = 0; m < BLK; ++m) {
      const float d = valid(m) ? base[off_d + blk * BLK + m] : 1.f;
      if (m <= i) G *= d;
      if (m > j && m <= i) gij *= d;
      if (m > i) last *= d;
    }
    cf[C_OUT + BLK * i + j] = own && j <= i ? gij * dots[j] : 0.f;
    if (i > 0) cf[C_SUB + BLK * (i - 1) + j] = own && j < i ? beta * gij * dots[BLK + j] : 0.f;
    if (j == 0) cf[C_RATE + i] = beta, cf[C_RG + i] = beta * G, cf[C_G + i] = G, cf[C_LAST + i] = last;
  };

  const int j0 = tid / PARTS * NC, part = tid % PARTS;      // a walker's first column in the slice, its rows
  pair_t S[NC][R / 2];
  float* st = p.state + ((size_t)slot * p.H + h) * p.D * p.V + col0 + j0;
  auto in_state = [&](int n, int c) { return n < p.D && col0 + j0 + c < p.V; };
  if (helper) {
    issue(0);
    cp_async_commit_group();
    if (n_chunks > 1) issue(1);
    cp_async_commit_group();
    cp_async_wait_group<1>();
    coefficients(0);
  } else {
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      const int n = part * R + 2 * i;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        S[c][i] = pair_of(in_state(n, c) ? st[(size_t)n * p.V + c] : 0.f, in_state(n + 1, c) ? st[(size_t)(n + 1) * p.V + c] : 0.f);
    }
  }
  __syncthreads();

  for (int ch = 0; ch < n_chunks; ++ch) {
    if (helper) {
      if (ch + 2 < n_chunks) issue(ch + 2);      // into the buffer the walkers left at the last barrier
      cp_async_commit_group();
      if (ch + 1 < n_chunks) {
        cp_async_wait_group<1>();                // all but the copies just started: chunk ch + 1 is here
        coefficients(ch + 1);
      } else if (p.keep > 0 && p.write) {
        // meanwhile: the request's last inputs replace the kept ones, channels shared out over the request's CTAs.  A
        // thread walks the kept rows of a channel oldest first: what it overwrites it has already moved.
        float* kept = p.kept + (size_t)slot * p.keep * p.channels;
        const int n = t1 - t0, cta = blockIdx.y * gridDim.x + blockIdx.x, ctas = gridDim.x * gridDim.y;
        for (int c = cta * HELPERS + tid; c < p.channels; c += ctas * HELPERS)
          for (int i = 0; i < p.keep; ++i) {
            const int s = n - p.keep + i;        // the step's row that becomes kept row i
            kept[(size_t)i * p.channels + c] =
                s >= 0 ? p.proj[(size_t)(t0 + s) * p.ld + c] : kept[(size_t)(i + n) * p.channels + c];
          }
      }
    } else {
      const int row0 = base_row + ch * CT;
      const float* base = buffer(ch);
#pragma unroll 1
      for (int blk = 0; blk < CT / BLK; ++blk) {
        const int rows = row0 + blk * BLK;
        if (rows >= t1) break;
        if (rows + BLK <= t0) continue;
        const float* tok = base + blk * BLK * REC;
        const float* cf = base + off_c + blk * COEF;
        pair_t kacc[BLK][NC], qacc[BLK][NC];
#pragma unroll
        for (int i = 0; i < BLK; ++i)
#pragma unroll
          for (int c = 0; c < NC; ++c) kacc[i][c] = qacc[i][c] = pair_of(0.f);
#pragma unroll
        for (int x = 0; x < R / 4; ++x)
#pragma unroll
          for (int i = 0; i < BLK; ++i) {
            const ulonglong2 k4 = reinterpret_cast<const ulonglong2*>(tok + i * REC + part * RS)[x];
            const ulonglong2 q4 = reinterpret_cast<const ulonglong2*>(tok + i * REC + NP + part * RS)[x];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              kacc[i][c] = pair_fma(k4.x, S[c][2 * x], kacc[i][c]);
              qacc[i][c] = pair_fma(q4.x, S[c][2 * x], qacc[i][c]);
              kacc[i][c] = pair_fma(k4.y, S[c][2 * x + 1], kacc[i][c]);
              qacc[i][c] = pair_fma(q4.y, S[c][2 * x + 1], qacc[i][c]);
            }
            if (R > 16) asm volatile("" ::: "memory");      // loads stay near their use: registers
          }
        const float4 rate = load4(cf + C_RATE), rg = load4(cf + C_RG), s1 = load4(cf + C_SUB), s2 = load4(cf + C_SUB + 4),
                     s3 = load4(cf + C_SUB + 8), out_w = load4(cf + C_OUT + BLK * part), last = load4(cf + C_LAST);
        const float g_part = cf[C_G + part], g_all = cf[C_G + BLK - 1];
        float u[BLK][NC], o[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float ks[BLK], qs[BLK];
#pragma unroll
          for (int i = 0; i < BLK; ++i) ks[i] = pair_sum(kacc[i][c]), qs[i] = pair_sum(qacc[i][c]);
#pragma unroll
          for (int i = 0; i < BLK; ++i) ks[i] += __shfl_xor_sync(0xffffffffu, ks[i], 1);
#pragma unroll
          for (int i = 0; i < BLK; ++i) ks[i] += __shfl_xor_sync(0xffffffffu, ks[i], 2);
          // thread p of the column's four is left with row p's sum of the queries
          const bool hi2 = part & 2, hi1 = part & 1;
          const float a0 = (hi2 ? qs[2] : qs[0]) + __shfl_xor_sync(0xffffffffu, hi2 ? qs[0] : qs[2], 2);
          const float a1 = (hi2 ? qs[3] : qs[1]) + __shfl_xor_sync(0xffffffffu, hi2 ? qs[1] : qs[3], 2);
          const float qp = (hi1 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, hi1 ? a0 : a1, 1);
          const float* vc = base + off_v + blk * BLK * Vs + j0 + c;
          u[0][c] = fmaf(rate.x, vc[0], -rg.x * ks[0]);
          u[1][c] = fmaf(-s1.x, u[0][c], fmaf(rate.y, vc[Vs], -rg.y * ks[1]));
          u[2][c] = fmaf(-s2.y, u[1][c], fmaf(-s2.x, u[0][c], fmaf(rate.z, vc[2 * Vs], -rg.z * ks[2])));
          u[3][c] = fmaf(-s3.z, u[2][c], fmaf(-s3.y, u[1][c], fmaf(-s3.x, u[0][c],
                                                                  fmaf(rate.w, vc[3 * Vs], -rg.w * ks[3]))));
          o[c] = fmaf(g_part, qp, fmaf(out_w.x, u[0][c], fmaf(out_w.y, u[1][c], fmaf(out_w.z, u[2][c], out_w.w * u[3][c]))));
        }
        const int row = rows + part;
        if (row >= t0 && row < t1) {
          float* dst = p.out + ((size_t)row * p.H + h) * p.V + col0 + j0;
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (col0 + j0 + c < p.V) dst[c] = o[c];
        }
        pair_t ue[BLK][NC];
        const pair_t ga = pair_of(g_all);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          ue[0][c] = pair_of(last.x * u[0][c]), ue[1][c] = pair_of(last.y * u[1][c]);
          ue[2][c] = pair_of(last.z * u[2][c]), ue[3][c] = pair_of(last.w * u[3][c]);
        }
#pragma unroll
        for (int x = 0; x < R / 4; ++x) {
#pragma unroll
          for (int c = 0; c < NC; ++c) S[c][2 * x] = pair_mul(ga, S[c][2 * x]), S[c][2 * x + 1] = pair_mul(ga, S[c][2 * x + 1]);
#pragma unroll
          for (int i = 0; i < BLK; ++i) {
            const ulonglong2 k4 = reinterpret_cast<const ulonglong2*>(tok + i * REC + part * RS)[x];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              S[c][2 * x] = pair_fma(k4.x, ue[i][c], S[c][2 * x]);
              S[c][2 * x + 1] = pair_fma(k4.y, ue[i][c], S[c][2 * x + 1]);
            }
            if (R > 16) asm volatile("" ::: "memory");
          }
        }
      }
    }
    __syncthreads();
  }
  if (helper) {
    cp_async_wait_group<0>();
  } else if (p.write) {
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      const int n = part * R + 2 * i;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        float lo, hi;
        pair_split(S[c][i], lo, hi);
        if (in_state(n, c)) st[(size_t)n * p.V + c] = lo;
        if (in_state(n + 1, c)) st[(size_t)(n + 1) * p.V + c] = hi;
      }
    }
  }
}

// ---- norm and gate ------------------------------------------------------------------------------
// out[t, h * V + i] = o / rms(o of head h) * w[i] * silu(gate[t, h * V + i]), rounded to T; a warp per (row, head).
// Rows of requests without a state slot (padding) leave as zeros.
template <typename T>
__global__ void __launch_bounds__(kThreads) head_norm_gate_kernel(T* __restrict__ out, const float* __restrict__ o,
                                                                  const float* __restrict__ gate, int ld_g,
                                                                  const T* __restrict__ w, const int* __restrict__ row_req,
                                                                  const int* __restrict__ state_slot, int tokens, int H,
                                                                  int V, float eps) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  if (unit >= (long long)tokens * H) return;
  const int t = (int)(unit / H), h = (int)(unit - (long long)t * H);
  const size_t at = (size_t)t * H * V + (size_t)h * V;
  if (state_slot[row_req[t]] == -1) {
    for (int i = lane; i < V; i += 32) out[at + i] = from_f32<T>(0.f);
    return;
  }
  // up to 128 entries a head wait in registers, outputs, gates and weights all asked for at once
  constexpr int kPerLane = 4;
  const float* g = gate + (size_t)t * ld_g + h * V;
  float y[kPerLane], z[kPerLane], ss = 0.f;
#pragma unroll
  for (int j = 0; j < kPerLane; ++j) {
    const int i = lane + 32 * j;
    y[j] = i < V ? o[at + i] : 0.f;
    z[j] = i < V ? silu_f(g[i]) * to_f32(w[i]) : 0.f;
    ss = fmaf(y[j], y[j], ss);
  }
  for (int i = lane + 32 * kPerLane; i < V; i += 32) ss = fmaf(o[at + i], o[at + i], ss);
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps);
#pragma unroll
  for (int j = 0; j < kPerLane; ++j) {
    const int i = lane + 32 * j;
    if (i < V) out[at + i] = from_f32<T>(y[j] * inv * z[j]);
  }
  for (int i = lane + 32 * kPerLane; i < V; i += 32) out[at + i] = from_f32<T>(o[at + i] * inv * (silu_f(g[i]) * to_f32(w[i])));
}

template <typename T>
void launch_prepare(const PrepareParams& p, dim3 grid, size_t smem, const void* taps_w, const void* a_log, const void* dt_bias,
                    cudaStream_t stream) {
  auto kernel = p.taps == 4 ? delta_prepare_kernel<T, 4> : p.taps == 3 ? delta_prepare_kernel<T, 3> : delta_prepare_kernel<T, 0>;
  lab_launch(kernel, grid, dim3(kThreads), smem, stream, (const T*)taps_w, (const T*)a_log, (const T*)dt_bias, p);
}

template <int R, int NC>
int launch_walk(const WalkParams& p, int requests, int vs, cudaStream_t stream) {
  const size_t smem = (size_t)3 * (CT * (record_floats(R) + vs + 2) + (CT / BLK) * COEF) * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(delta_walk_kernel<R, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  dim3 grid((p.V + vs - 1) / vs, p.H, requests);
  return (int)lab_launch(delta_walk_kernel<R, NC>, grid, dim3(PARTS * vs / NC + HELPERS), smem, stream, p, vs);
}

template <int R>
int launch_walk_cols(const WalkParams& p, int requests, int vs, int cols, cudaStream_t stream) {
  return cols == 2 ? launch_walk<R, 2>(p, requests, vs, stream) : launch_walk<R, 1>(p, requests, vs, stream);
}

}  // namespace

// Floats of a record for heads of D key channels, and of one of its shares of k (R channels and four of padding).
LAB_EXPORT int lab_delta_record_floats(int D) { return record_floats(share_of(D)); }
LAB_EXPORT int lab_delta_record_share(int D) { return share_of(D); }

// proj columns: q 0, k G * D, v 2 * G * D, rates b_at, decays a_at.  rec: [G, tokens] records on 16 bytes; v: [tokens,
// H * V]; decay, rate: [H, tokens].
LAB_EXPORT int lab_delta_prepare(float* rec, float* v, float* decay, float* rate, const float* proj, int ld, int b_at,
                                 int a_at, int taps, int H, int G, int D, int V, const void* taps_w, const void* a_log,
                                 const void* dt_bias, const float* kept, const int* row_req, const int* q_start,
                                 const int* state_slot, int tokens, int n_slots, float q_scale, float unit_eps, int dtype,
                                 cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (taps < 1 || H <= 0 || G <= 0 || H % G || D <= 0 || D > 256 || V <= 0 || G + H + 1 > 65535) return (int)cudaErrorInvalidValue;
  PrepareParams p;
  p.proj = proj; p.ld = ld; p.b_at = b_at; p.a_at = a_at; p.taps = taps; p.H = H; p.G = G; p.D = D; p.V = V;
  p.tokens = tokens; p.kept = kept; p.row_req = row_req; p.q_start = q_start; p.state_slot = state_slot;
  p.n_slots = n_slots; p.q_scale = q_scale; p.unit_eps = unit_eps; p.rec = rec; p.R = share_of(D); p.v = v;
  p.decay = decay; p.rate = rate;
  const dim3 grid((tokens + kThreads / 32 - 1) / (kThreads / 32), G + H + 1);
  const size_t smem = (size_t)(kThreads / 32) * D * sizeof(float);
  if (dtype == LAB_F32) launch_prepare<float>(p, grid, smem, taps_w, a_log, dt_bias, stream);
  else launch_prepare<__nv_bfloat16>(p, grid, smem, taps_w, a_log, dt_bias, stream);
  LAB_LAUNCH_CHECK();
}

// vs: columns of the state a CTA takes (a multiple of 8 * cols, at most 32 * cols); cols: columns a thread takes (1, or
// up to 128 key channels 2).
// kept (with proj, ld, keep, channels): the inputs that replace a request's kept ones; null: none.
LAB_EXPORT int lab_delta_walk(float* out, const float* rec, const float* v, const float* decay, const float* rate,
                              float* state, const int* q_start, const int* state_slot, int tokens, int requests,
                              int n_slots, int H, int G, int D, int V, const float* proj, int ld, float* kept, int keep,
                              int channels, int write, int vs, int cols, cudaStream_t stream) {
  if (requests <= 0 || tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || (cols != 1 && cols != 2) || vs <= 0 || vs % (8 * cols) ||
      PARTS * vs / cols + HELPERS > 256 || (((uintptr_t)rec) & 15))
    return (int)cudaErrorInvalidValue;
  WalkParams p;
  p.out = out; p.rec = rec; p.v = v; p.decay = decay; p.rate = rate; p.tokens = tokens; p.state = state;
  p.q_start = q_start; p.state_slot = state_slot; p.n_slots = n_slots; p.H = H; p.G = G; p.D = D; p.V = V;
  p.write = write; p.proj = proj; p.kept = kept; p.ld = ld; p.keep = kept != nullptr ? keep : 0; p.channels = channels;
  // 16-byte copies: every row of v, and every head's and slice's start in it, on a 16-byte boundary
  p.vec = V % 4 == 0 && (((uintptr_t)v) & 15) == 0;
  switch (share_of(D)) {
    case 4: return launch_walk_cols<4>(p, requests, vs, cols, stream);
    case 8: return launch_walk_cols<8>(p, requests, vs, cols, stream);
    case 16: return launch_walk_cols<16>(p, requests, vs, cols, stream);
    case 32: return launch_walk_cols<32>(p, requests, vs, cols, stream);
    case 64: return D <= 256 && cols == 1 ? launch_walk<64, 1>(p, requests, vs, stream) : (int)cudaErrorInvalidValue;
  }
  return (int)cudaErrorInvalidValue;
}

LAB_EXPORT int lab_head_norm_gate(void* out, const float* o, const float* gate, int ld_g, const void* w,
                                  const int* row_req, const int* state_slot, int tokens, int H, int V, float eps,
                                  int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const long long units = (long long)tokens * H;
  const int blocks = (int)((units + kThreads / 32 - 1) / (kThreads / 32));
  if (dtype == LAB_F32)
    lab_launch(head_norm_gate_kernel<float>, dim3(blocks), dim3(kThreads), 0, stream, (float*)out, o, gate, ld_g,
               (const float*)w, row_req, state_slot, tokens, H, V, eps);
  else
    lab_launch(head_norm_gate_kernel<__nv_bfloat16>, dim3(blocks), dim3(kThreads), 0, stream, (__nv_bfloat16*)out, o, gate,
               ld_g, (const __nv_bfloat16*)w, row_req, state_slot, tokens, H, V, eps);
  LAB_LAUNCH_CHECK();
}
