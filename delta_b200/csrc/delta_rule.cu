// The gated delta rule with one decay per head and key channel.
//
// Per head h, with a state S [dk, dv] in 32 bit that a request carries from token to token and the query/key head
// kv = h / (H / G):
//     q = unit(q_kv) * q_scale,  k = unit(k_kv)          unit(x) = x / sqrt(sum(x^2) + guard)
//     g_i  = exp(-exp(A_log_h) * softplus(a_i + dt_bias_i))          one per key channel i
//     beta = sigmoid(b_h)
//     S <- diag(g) S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q .
// The state is kept with a value column's dk entries side by side: [slot][H][dv][dk].  Everything below is 32-bit FMA
// whatever the type of the inputs.
//
// delta_rows: tokens in turn, a slice of the value columns per block; a column's state lies in the registers of eight
// lanes.  Single tokens (the state streams through registers once) and short portions.
//
// Long portions are cut into chunks of 32 tokens.  With L_t the sum of the log decays of a chunk's tokens 0..t (per
// channel) and S the state before the chunk,
//     u_t = beta_t (v_t - S^T (e^(L_t) k_t) - sum_{s<t} A_ts u_s),     A_ts = sum_i k_t[i] k_s[i] e^(L_t[i] - L_s[i])
//     o_t = S^T (e^(L_t) q_t) + sum_{s<=t} B_ts u_s,                    B_ts = sum_i q_t[i] k_s[i] e^(L_t[i] - L_s[i])
//     S  <- diag(e^(L_last)) S + sum_s (e^(L_last - L_s) k_s) u_s^T .
// u is linear in S, u = U - W S, where U and W solve the same unit lower triangular system for the right-hand sides v_t and
// e^(L_t) k_t.  So
//   1. delta_chunk: every chunk of every head in parallel: A, B, U, W and the scaled queries and keys;
//   2. delta_walk:  along a row, chunk after chunk, a slice of the value columns per block: three small products a chunk.
// No exponent is ever positive.  Sums of log decays are kept as two floats, so that a difference of two of them is as good
// when the sums themselves are large.
#include "common.cuh"
#include "mma_helpers.cuh"

namespace {

__device__ __forceinline__ float softplus_dr(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// ---- tokens in turn --------------------------------------------------------------------------------------------------------
constexpr int ROWS_THREADS = 128;
constexpr int ROWS_TOKENS = 4;                       // tokens whose vectors are prepared at a time
constexpr int LANES = 8;                             // lanes that share a value column
constexpr int ROWS_COLS = ROWS_THREADS / LANES;      // value columns of a block

// grid (rows, H, ceil(dv / ROWS_COLS)).  NI: groups of 32 key channels (the last may be partly empty).
template <typename T, int NI>
__global__ void __launch_bounds__(ROWS_THREADS)
delta_rows_kernel(const T* __restrict__ qkv, int stride, int k_off, int v_off, const T* __restrict__ b, int b_stride,
                  const float* __restrict__ a, int a_stride, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                  float* __restrict__ state, float* __restrict__ out, const int* __restrict__ row_slot,
                  const int* __restrict__ row_q_start, const int* __restrict__ row_q_len, int H, int G, int dk, int dv, float q_scale,
                  float guard, int vec) {
  constexpr int W = NI * 32;
  __shared__ __align__(16) float qs[ROWS_TOKENS][W], ks[ROWS_TOKENS][W], gs[ROWS_TOKENS][W];
  __shared__ float vs[ROWS_TOKENS][ROWS_COLS], bs[ROWS_TOKENS];
  const int row = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * ROWS_COLS;
  const int n_new = row_q_len != nullptr ? row_q_len[row] : 1;
  if (n_new <= 0) return;
  const int t0 = row_q_start[row], kv = h / (H / G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, p = tid & (LANES - 1), col = tid / LANES;
  const bool live = j0 + col < dv;
  float* st = state + (((size_t)row_slot[row] * H + h) * dv + (live ? j0 + col : 0)) * dk;
  float S[NI][4];
#pragma unroll
  for (int m = 0; m < NI; ++m) {
    const int i = 32 * m + 4 * p;
    if (vec) {
      const float4 v = (live && i < dk) ? *reinterpret_cast<const float4*>(st + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[m][0] = v.x; S[m][1] = v.y; S[m][2] = v.z; S[m][3] = v.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) S[m][e] = (live && i + e < dk) ? st[i + e] : 0.f;
    }
  }
  const float rate = expf(A_log[h]);
  for (int c0 = 0; c0 < n_new; c0 += ROWS_TOKENS) {
    const int n = min(ROWS_TOKENS, n_new - c0);
    if (c0 > 0) __syncthreads();
    for (int task = warp; task < 3 * n; task += ROWS_THREADS / 32) {      // one warp per vector of a token: q, k, g
      const int t = task / 3, which = task - 3 * t;
      const size_t tok = (size_t)(t0 + c0 + t);
      if (which < 2) {
        const T* src = qkv + tok * stride + (which ? k_off : 0) + (size_t)kv * dk;
        float x[NI], ss = 0.f;
#pragma unroll
        for (int m = 0; m < NI; ++m) {
          x[m] = lane + 32 * m < dk ? to_f32<T>(src[lane + 32 * m]) : 0.f;
          ss = fmaf(x[m], x[m], ss);
        }
        const float f = (which ? 1.f : q_scale) / sqrtf(warp_sum(ss) + guard);
        float* dst = which ? ks[t] : qs[t];
#pragma unroll
        for (int m = 0; m < NI; ++m) dst[lane + 32 * m] = x[m] * f;
      } else {
        const float* ar = a + tok * a_stride + (size_t)h * dk;
#pragma unroll
        for (int m = 0; m < NI; ++m) {
          const int i = lane + 32 * m;
          gs[t][i] = i < dk ? expf(-rate * softplus_dr(ar[i] + dt_bias[(size_t)h * dk + i])) : 0.f;
        }
      }
    }
    for (int idx = tid; idx < n * ROWS_COLS; idx += ROWS_THREADS) {
      const int t = idx / ROWS_COLS, c = idx - t * ROWS_COLS;
      vs[t][c] = j0 + c < dv ? to_f32<T>(qkv[(size_t)(t0 + c0 + t) * stride + v_off + (size_t)h * dv + j0 + c]) : 0.f;
    }
    if (tid < n) bs[tid] = 1.f / (1.f + expf(-to_f32<T>(b[(size_t)(t0 + c0 + tid) * b_stride + h])));
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      float dot = 0.f;
#pragma unroll
      for (int m = 0; m < NI; ++m) {
        const float4 g = *reinterpret_cast<const float4*>(&gs[t][32 * m + 4 * p]);
        const float4 k = *reinterpret_cast<const float4*>(&ks[t][32 * m + 4 * p]);
        S[m][0] *= g.x; S[m][1] *= g.y; S[m][2] *= g.z; S[m][3] *= g.w;
        dot = fmaf(S[m][0], k.x, dot); dot = fmaf(S[m][1], k.y, dot); dot = fmaf(S[m][2], k.z, dot); dot = fmaf(S[m][3], k.w, dot);
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
      const float u = bs[t] * (vs[t][col] - dot);
      float y = 0.f;
#pragma unroll
      for (int m = 0; m < NI; ++m) {
        const float4 k = *reinterpret_cast<const float4*>(&ks[t][32 * m + 4 * p]);
        const float4 q = *reinterpret_cast<const float4*>(&qs[t][32 * m + 4 * p]);
        S[m][0] = fmaf(k.x, u, S[m][0]); S[m][1] = fmaf(k.y, u, S[m][1]); S[m][2] = fmaf(k.z, u, S[m][2]); S[m][3] = fmaf(k.w, u, S[m][3]);
        y = fmaf(S[m][0], q.x, y); y = fmaf(S[m][1], q.y, y); y = fmaf(S[m][2], q.z, y); y = fmaf(S[m][3], q.w, y);
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (p == 0 && live) out[(size_t)(t0 + c0 + t) * H * dv + (size_t)h * dv + j0 + col] = y;
    }
  }
  if (!live) return;
#pragma unroll
  for (int m = 0; m < NI; ++m) {
    const int i = 32 * m + 4 * p;
    if (vec) {
      if (i < dk) *reinterpret_cast<float4*>(st + i) = make_float4(S[m][0], S[m][1], S[m][2], S[m][3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (i + e < dk) st[i + e] = S[m][e];
    }
  }
}

// ---- chunks ----------------------------------------------------------------------------------------------------------------
constexpr int C = 32;                    // tokens of a chunk
constexpr int CP = C + 4;                // padded row of a chunk-by-chunk matrix
constexpr int PREP_THREADS = 288;        // 36 tiles of 4 x 4 token pairs on and below the diagonal, eight lanes each
constexpr int WALK_THREADS = 256;
constexpr int WALK_COLS = 16;            // value columns of a block
constexpr int SHARES = WALK_THREADS / 32;      // the warps share the channels of the first product
constexpr int WALK_LD = WALK_COLS + 4;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float LEAST_LOG2 = -1000.f;    // 2^-1000 is zero in 32 bit: a token's log decay is no smaller, so that sums stay finite
constexpr size_t SMEM_LIMIT = 220 * 1024;

__host__ __device__ __forceinline__ int pad_k(int dk) { return (dk + 3) & ~3; }
__host__ __device__ __forceinline__ int pad_v(int dv) { return (dv + WALK_COLS - 1) / WALK_COLS * WALK_COLS; }
__host__ __device__ __forceinline__ int prep_ld(int dk) { return ((dk + 7) & ~7) + 2; }      // 2 mod 8: the four tiles of a warp read different banks

// What delta_chunk leaves for delta_walk per (chunk, head), in floats, with rows padded as the walk wants them in shared memory, so that
// it copies one piece as it lies: W and Q (rows of wl), K (rows of kp), B (rows of CP), the decays of the whole chunk; then, per slice of
// the value columns, U (rows of WALK_LD).
struct ChunkLayout {
  int wl, w, q, k, b, d, common, u, size;
  __host__ __device__ ChunkLayout(int dk, int dv) {
    const int kp = pad_k(dk);
    wl = kp + 4;
    w = 0;
    q = w + C * wl;
    k = q + C * wl;
    b = k + C * kp;
    d = b + C * CP;
    common = d + kp;
    u = common;
    size = u + pad_v(dv) / WALK_COLS * C * WALK_LD;
  }
};

size_t prep_smem(int dk) { return (size_t)(4 * C * prep_ld(dk) + 2 * C * CP + C) * sizeof(float); }
size_t walk_stage(int dk) { return (size_t)(2 * C * (pad_k(dk) + 4) + C * pad_k(dk) + C * WALK_LD + C * CP + pad_k(dk)) * sizeof(float); }
size_t walk_smem(int dk, int stages) { return stages * walk_stage(dk) + (size_t)(pad_k(dk) * WALK_LD + SHARES * 2 * C * WALK_LD + C * WALK_LD) * sizeof(float); }

// grid (most chunks of a row, rows * H).
template <typename T>
__global__ void __launch_bounds__(PREP_THREADS, 2)
delta_chunk_kernel(const T* __restrict__ qkv, int stride, int k_off, int v_off, const T* __restrict__ b, int b_stride,
                   const float* __restrict__ a, int a_stride, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                   float* __restrict__ work, const int* __restrict__ row_q_start, const int* __restrict__ row_q_len,
                   const int* __restrict__ chunk_base, int H, int G, int dk, int dv, float q_scale, float guard, int vec) {
  extern __shared__ __align__(16) float sm[];
  const int row = blockIdx.y / H, h = blockIdx.y % H, c0 = blockIdx.x * C, n_new = row_q_len[row];
  if (c0 >= n_new) return;
  const int n = min(C, n_new - c0), t0 = row_q_start[row] + c0, kv = h / (H / G);
  const int ld = prep_ld(dk), kp = pad_k(dk), vp = pad_v(dv);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* At = sm;                    // [C][CP]: At[s][t] = A_ts for s < t, else 0
  float* B = At + C * CP;            // [C][CP]: B[t][s] for s <= t, else 0
  float* beta = B + C * CP;          // [C], 0 behind the chunk's end
  float* Q = beta + C;               // [C][ld]
  float* K = Q + C * ld;             // [C][ld], 0 behind the end
  float* Lh = K + C * ld;            // [C][ld]: the sums of log2 decays, high part
  float* Ll = Lh + C * ld;           // [C][ld]: low part
  const ChunkLayout at(dk, dv);
  float* ws = work + ((size_t)(chunk_base[row] + blockIdx.x) * H + h) * at.size;
  const float rate = expf(A_log[h]) * LOG2E;
  if (vec) {      // sizes and addresses allow sixteen-byte loads (eight bfloat16 or float entries at a time)
    const int per = dk / 8;
    for (int idx = tid; idx < 2 * C * per; idx += PREP_THREADS) {
      const int r = idx / per, i = (idx - r * per) * 8, t = r & (C - 1);
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (t < n) load8<T>(qkv + (size_t)(t0 + t) * stride + (r < C ? 0 : k_off) + (size_t)kv * dk + i, x);
#pragma unroll
      for (int e = 0; e < 8; e += 2) *reinterpret_cast<float2*>(Q + r * ld + i + e) = make_float2(x[e], x[e + 1]);      // K's rows follow Q's
    }
    for (int idx = tid; idx < C * per; idx += PREP_THREADS) {
      const int t = idx / per, i = (idx - t * per) * 8;
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, bias[8];
      if (t < n) {
        load8<float>(a + (size_t)(t0 + t) * a_stride + (size_t)h * dk + i, x);
        load8<float>(dt_bias + (size_t)h * dk + i, bias);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = fmaxf(-rate * softplus_dr(x[e] + bias[e]), LEAST_LOG2);
      }
#pragma unroll
      for (int e = 0; e < 8; e += 2) *reinterpret_cast<float2*>(Lh + t * ld + i + e) = make_float2(x[e], x[e + 1]);
    }
  } else {
    for (int idx = tid; idx < 2 * C * dk; idx += PREP_THREADS) {
      const int r = idx / dk, i = idx - r * dk, t = r & (C - 1);
      Q[r * ld + i] = t < n ? to_f32<T>(qkv[(size_t)(t0 + t) * stride + (r < C ? 0 : k_off) + (size_t)kv * dk + i]) : 0.f;
    }
    for (int idx = tid; idx < C * dk; idx += PREP_THREADS) {
      const int t = idx / dk, i = idx - t * dk;
      float l = 0.f;
      if (t < n) l = fmaxf(-rate * softplus_dr(a[(size_t)(t0 + t) * a_stride + (size_t)h * dk + i] + dt_bias[(size_t)h * dk + i]), LEAST_LOG2);
      Lh[t * ld + i] = l;
    }
  }
  if (tid < C) beta[tid] = tid < n ? 1.f / (1.f + expf(-to_f32<T>(b[(size_t)(t0 + tid) * b_stride + h]))) : 0.f;
  __syncthreads();
  for (int r = warp; r < 2 * C; r += PREP_THREADS / 32) {      // unit vectors
    float ss = 0.f;
    for (int i = lane; i < dk; i += 32) ss = fmaf(Q[r * ld + i], Q[r * ld + i], ss);
    const float f = (r < C ? q_scale : 1.f) / sqrtf(warp_sum(ss) + guard);
    for (int i = lane; i < dk; i += 32) Q[r * ld + i] *= f;
  }
  for (int i = tid; i < dk; i += PREP_THREADS) {
    double sum = 0.0;
#pragma unroll 4
    for (int t = 0; t < C; ++t) {
      sum += (double)Lh[t * ld + i];
      const float hi = (float)sum;
      Lh[t * ld + i] = hi;
      Ll[t * ld + i] = (float)(sum - (double)hi);
    }
  }
  __syncthreads();
  {      // A and B: a tile of 4 x 4 pairs (t, s) per eight lanes, which share the channels
    const int tile = tid >> 3, part = tid & 7;
    int ti = 0;
    while ((ti + 1) * (ti + 2) / 2 <= tile) ++ti;
    const int tj = tile - ti * (ti + 1) / 2;
    float acc[32];      // [0, 16): A, [16, 32): B
#pragma unroll
    for (int x = 0; x < 32; ++x) acc[x] = 0.f;
    for (int i = part; i < dk; i += 8) {
      float kt[4], qt[4], ht[4], lt[4], kk[4], hs[4], ls[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int rt = (4 * ti + x) * ld + i, rs = (4 * tj + x) * ld + i;
        kt[x] = K[rt]; qt[x] = Q[rt]; ht[x] = Lh[rt]; lt[x] = Ll[rt];
        kk[x] = K[rs]; hs[x] = Lh[rs]; ls[x] = Ll[rs];
      }
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) {
          // above the diagonal the exponent would be positive: those pairs are dropped below
          const float w = exp2f(fminf((ht[x] - hs[y]) + (lt[x] - ls[y]), 0.f)) * kk[y];
          acc[4 * x + y] = fmaf(kt[x], w, acc[4 * x + y]);
          acc[16 + 4 * x + y] = fmaf(qt[x], w, acc[16 + 4 * x + y]);
        }
    }
    // the eight lanes' sums: each step halves what a lane keeps, so lane `part` ends with four of the 32
#pragma unroll
    for (int half = 16, bit = 4; bit > 0; half >>= 1, bit >>= 1) {
      const bool upper = (part & bit) != 0;
#pragma unroll
      for (int x = 0; x < 16; ++x)
        if (x < half) {
          const float send = upper ? acc[x] : acc[x + half], keep = upper ? acc[x + half] : acc[x];
          acc[x] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
        }
    }
#pragma unroll
    for (int y = 0; y < 4; ++y) {
      const int x = part & 3, t = 4 * ti + x, s = 4 * tj + y;
      if (part < 4) At[s * CP + t] = s < t ? acc[y] : 0.f;
      else B[t * CP + s] = s <= t ? acc[y] : 0.f;
      if (ti != tj && part >= 4) B[(4 * tj + x) * CP + 4 * ti + y] = 0.f;      // the mirrored tile lies above the diagonal
    }
  }
  __syncthreads();
  for (int idx = tid; idx < C * C; idx += PREP_THREADS) ws[at.b + (idx >> 5) * CP + (idx & 31)] = B[(idx >> 5) * CP + (idx & 31)];
  for (int idx = tid; idx < C * kp; idx += PREP_THREADS) {
    const int t = idx / kp, i = idx - t * kp;
    float q = 0.f, k = 0.f;
    if (i < dk) {
      const int r = t * ld + i, last = (C - 1) * ld + i;
      q = Q[r] * exp2f(Lh[r] + Ll[r]);
      k = K[r] * exp2f((Lh[last] - Lh[r]) + (Ll[last] - Ll[r]));
    }
    ws[at.q + t * at.wl + i] = q;
    ws[at.k + idx] = k;
  }
  for (int i = tid; i < kp; i += PREP_THREADS) ws[at.d + i] = i < dk ? exp2f(Lh[(C - 1) * ld + i] + Ll[(C - 1) * ld + i]) : 0.f;
  // the triangular system, a thread per column of the right-hand side: U from the values, W from the decayed keys
  for (int c = tid; c < vp + kp; c += PREP_THREADS) {
    float r[C];
    const int i = c - vp;
    if (c < vp) {
      const T* src = qkv + (size_t)t0 * stride + v_off + (size_t)h * dv + c;
#pragma unroll
      for (int t = 0; t < C; ++t) r[t] = (t < n && c < dv) ? to_f32<T>(src[(size_t)t * stride]) : 0.f;
    } else {
#pragma unroll
      for (int t = 0; t < C; ++t) r[t] = i < dk ? K[t * ld + i] * exp2f(Lh[t * ld + i] + Ll[t * ld + i]) : 0.f;
    }
#pragma unroll
    for (int s = 0; s < C; ++s) {
      const float x = beta[s] * r[s];
      r[s] = x;
#pragma unroll
      for (int t4 = (s + 1) / 4; t4 < C / 4; ++t4) {
        const float4 w = *reinterpret_cast<const float4*>(At + s * CP + 4 * t4);      // 0 for t <= s
        if (4 * t4 + 0 > s) r[4 * t4 + 0] = fmaf(-w.x, x, r[4 * t4 + 0]);
        if (4 * t4 + 1 > s) r[4 * t4 + 1] = fmaf(-w.y, x, r[4 * t4 + 1]);
        if (4 * t4 + 2 > s) r[4 * t4 + 2] = fmaf(-w.z, x, r[4 * t4 + 2]);
        if (4 * t4 + 3 > s) r[4 * t4 + 3] = fmaf(-w.w, x, r[4 * t4 + 3]);
      }
    }
    float* dst = c < vp ? ws + at.u + (c / WALK_COLS) * C * WALK_LD + c % WALK_COLS : ws + at.w + i;
    const int step = c < vp ? WALK_LD : at.wl;
#pragma unroll
    for (int t = 0; t < C; ++t) dst[(size_t)t * step] = r[t];
  }
}

// grid (slices of the value columns, rows * H).  STAGES 2: the next chunk's matrices are fetched during this chunk's products.
template <int STAGES>
__global__ void __launch_bounds__(WALK_THREADS)
delta_walk_kernel(const float* __restrict__ work, float* __restrict__ state, float* __restrict__ out, const int* __restrict__ row_slot,
                  const int* __restrict__ row_q_start, const int* __restrict__ row_q_len, const int* __restrict__ chunk_base, int H,
                  int dk, int dv) {
  extern __shared__ __align__(16) float sm[];
  const int row = blockIdx.y / H, h = blockIdx.y % H, j0 = blockIdx.x * WALK_COLS, n_new = row_q_len[row];
  if (n_new <= 0) return;
  const ChunkLayout at(dk, dv);
  const int kp = pad_k(dk), wl = at.wl, tid = threadIdx.x;
  const int jn = min(WALK_COLS, dv - j0);
  const int stage_floats = at.common + C * WALK_LD;
  float* stages = sm;
  float* S = sm + STAGES * stage_floats;             // [kp][WALK_LD]
  float* part = S + kp * WALK_LD;                    // [SHARES][2 C][WALK_LD]: the shares of the first product
  float* O = part + SHARES * 2 * C * WALK_LD;        // [C][WALK_LD]
  const int chunks = (n_new + C - 1) / C;
  const float* ws0 = work + ((size_t)chunk_base[row] * H + h) * at.size;
  auto fetch = [&](int c) {
    const float* ws = ws0 + (size_t)c * H * at.size;
    float* X = stages + (STAGES == 2 ? (c & 1) : 0) * stage_floats;
    for (int idx = tid; idx < at.common / 4; idx += WALK_THREADS) cp_async_16(smem_u32(X + idx * 4), ws + idx * 4, true);
    const float* u = ws + at.u + (size_t)blockIdx.x * C * WALK_LD;
    for (int idx = tid; idx < C * WALK_LD / 4; idx += WALK_THREADS) cp_async_16(smem_u32(X + at.common + idx * 4), u + idx * 4, true);
    cp_async_commit();
  };
  fetch(0);
  float* st = state + (((size_t)row_slot[row] * H + h) * dv + j0) * dk;
  for (int idx = tid; idx < kp * WALK_COLS; idx += WALK_THREADS) {
    const int j = idx / kp, i = idx - j * kp;
    S[i * WALK_LD + j] = (i < dk && j < jn) ? st[(size_t)j * dk + i] : 0.f;
  }
  const int share = tid >> 5, ti = (tid & 31) >> 2, tj = tid & 3;
  for (int c = 0; c < chunks; ++c) {
    if (STAGES == 2 && c + 1 < chunks) {
      fetch(c + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    float* X = stages + (STAGES == 2 ? (c & 1) : 0) * stage_floats;
    const float *Kd = X + at.k, *B = X + at.b, *D = X + at.d;
    float* U = X + at.common;
    {      // [W ; Q] S: a thread takes the rows ti + 8 q and four columns; the warps share the channels
      float acc[8][4] = {};
      for (int i4 = share; i4 < kp / 4; i4 += SHARES) {
        float4 s[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) s[q] = *reinterpret_cast<const float4*>(S + (4 * i4 + q) * WALK_LD + 4 * tj);
#pragma unroll
        for (int q = 0; q < 8; ++q) {
          const float4 x = *reinterpret_cast<const float4*>(X + (ti + 8 * q) * wl + 4 * i4);
          const float xv[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            acc[q][0] = fmaf(xv[e], s[e].x, acc[q][0]);
            acc[q][1] = fmaf(xv[e], s[e].y, acc[q][1]);
            acc[q][2] = fmaf(xv[e], s[e].z, acc[q][2]);
            acc[q][3] = fmaf(xv[e], s[e].w, acc[q][3]);
          }
        }
      }
#pragma unroll
      for (int q = 0; q < 8; ++q)
        *reinterpret_cast<float4*>(part + ((size_t)share * 2 * C + ti + 8 * q) * WALK_LD + 4 * tj) = make_float4(acc[q][0], acc[q][1], acc[q][2], acc[q][3]);
    }
    __syncthreads();
    {
      const int t = tid >> 2, j = (tid & 3) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int q = 0; q < SHARES; ++q) {
        const float4 w = *reinterpret_cast<const float4*>(part + ((size_t)q * 2 * C + t) * WALK_LD + j);
        v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
      }
      if (t < C) {
        float4* u = reinterpret_cast<float4*>(U + t * WALK_LD + j);
        const float4 o = *u;
        *u = make_float4(o.x - v.x, o.y - v.y, o.z - v.z, o.w - v.w);
      } else {
        *reinterpret_cast<float4*>(O + (t - C) * WALK_LD + j) = v;
      }
    }
    __syncthreads();
    if (tid < WALK_THREADS / 2) {      // half of the warps: the state behind the chunk
      for (int tile = tid; tile < kp; tile += WALK_THREADS / 2) {
        const int i = (tile >> 2) * 4, j = (tile & 3) * 4;
        float acc[4][4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float4 s = *reinterpret_cast<const float4*>(S + (i + x) * WALK_LD + j);
          const float d = D[i + x];
          acc[x][0] = d * s.x; acc[x][1] = d * s.y; acc[x][2] = d * s.z; acc[x][3] = d * s.w;
        }
#pragma unroll 8
        for (int s = 0; s < C; ++s) {
          const float4 k = *reinterpret_cast<const float4*>(Kd + s * kp + i);
          const float4 u = *reinterpret_cast<const float4*>(U + s * WALK_LD + j);
          const float kx[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            acc[x][0] = fmaf(kx[x], u.x, acc[x][0]);
            acc[x][1] = fmaf(kx[x], u.y, acc[x][1]);
            acc[x][2] = fmaf(kx[x], u.z, acc[x][2]);
            acc[x][3] = fmaf(kx[x], u.w, acc[x][3]);
          }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) *reinterpret_cast<float4*>(S + (i + x) * WALK_LD + j) = make_float4(acc[x][0], acc[x][1], acc[x][2], acc[x][3]);
      }
    } else {      // the other half: the chunk's outputs
      const int idx = tid - WALK_THREADS / 2, t = idx >> 2, j = (idx & 3) * 4;
      float4 o = *reinterpret_cast<const float4*>(O + t * WALK_LD + j);
#pragma unroll 4
      for (int s4 = 0; s4 < C / 4; ++s4) {
        const float4 w = *reinterpret_cast<const float4*>(B + t * CP + 4 * s4);
        const float wv[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 u = *reinterpret_cast<const float4*>(U + (4 * s4 + e) * WALK_LD + j);
          o.x = fmaf(wv[e], u.x, o.x); o.y = fmaf(wv[e], u.y, o.y); o.z = fmaf(wv[e], u.z, o.z); o.w = fmaf(wv[e], u.w, o.w);
        }
      }
      if (c * C + t < n_new) {
        float* dst = out + (size_t)(row_q_start[row] + c * C + t) * H * dv + (size_t)h * dv + j0 + j;
        const float ov[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (j + e < jn) dst[e] = ov[e];
      }
    }
    __syncthreads();
    if (STAGES == 1 && c + 1 < chunks) fetch(c + 1);
  }
  for (int idx = tid; idx < dk * jn; idx += WALK_THREADS) {
    const int j = idx / dk, i = idx - j * dk;
    st[(size_t)j * dk + i] = S[i * WALK_LD + j];
  }
}

int check_sizes(const char* who, int rows, int H, int G, int dk, int dv) {
  DK_REQUIRE(rows > 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0, "%s: bad sizes rows=%d H=%d G=%d dk=%d dv=%d", who, rows, H, G, dk, dv);
  DK_REQUIRE((long long)rows * H <= 65535, "%s: %d rows of %d heads are above the grid's limit", who, rows, H);
  return 0;
}
}  // namespace

extern "C" int dk_delta_rule_max_key() { return 512; }

// Tokens in turn.  row_q_len null: every row brings one token.
extern "C" int dk_delta_rule(const void* qkv, int stride, int k_off, int v_off, const void* b, int b_stride, const float* a, int a_stride,
                             const float* A_log, const float* dt_bias, float* state, float* out, const int* row_slot,
                             const int* row_q_start, const int* row_q_len, int rows, int H, int G, int dk, int dv, float q_scale,
                             float guard, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  if (int e = check_sizes("delta_rule", rows, H, G, dk, dv)) return e;
  DK_REQUIRE(dk <= 512, "delta_rule: keys of %d entries are above the 512 this kernel keeps in registers", dk);
  DK_REQUIRE(dtype == DK_F32 || dtype == DK_BF16, "delta_rule: unknown dtype %d", dtype);
  const dim3 grid(rows, H, (dv + ROWS_COLS - 1) / ROWS_COLS);
  const int vec = dk % 4 == 0 && ((uintptr_t)state % 16) == 0;
#define LAUNCH(T, NI)                                                                                                             \
  delta_rows_kernel<T, NI><<<grid, ROWS_THREADS, 0, stream>>>((const T*)qkv, stride, k_off, v_off, (const T*)b, b_stride, a, a_stride, \
                                                              A_log, dt_bias, state, out, row_slot, row_q_start, row_q_len, H, G, dk, \
                                                              dv, q_scale, guard, vec)
#define PICK(T)                       \
  do {                                \
    if (dk <= 32) LAUNCH(T, 1);       \
    else if (dk <= 64) LAUNCH(T, 2);  \
    else if (dk <= 128) LAUNCH(T, 4); \
    else if (dk <= 256) LAUNCH(T, 8); \
    else LAUNCH(T, 16);               \
  } while (0)
  if (dtype == DK_F32) PICK(float);
  else PICK(__nv_bfloat16);
#undef PICK
#undef LAUNCH
  return dk_check_launch("delta_rule");
}

extern "C" int dk_delta_rule_chunk() { return C; }

extern "C" int dk_delta_rule_chunked_supported(int dk, int dv) {
  return dk > 0 && dv > 0 && prep_smem(dk) <= SMEM_LIMIT && walk_smem(dk, 1) <= SMEM_LIMIT;
}

// Floats of working memory per (chunk, head).
extern "C" int dk_delta_rule_chunk_floats(int dk, int dv) { return ChunkLayout(dk, dv).size; }

// Long portions.  `chunk_base` [rows]: the number of chunks of all rows before this one; `max_chunks`: the most chunks of a row;
// `work` holds (all chunks) x H x dk_delta_rule_chunk_floats floats.
extern "C" int dk_delta_rule_chunked(const void* qkv, int stride, int k_off, int v_off, const void* b, int b_stride, const float* a,
                                     int a_stride, const float* A_log, const float* dt_bias, float* state, float* out, float* work,
                                     const int* row_slot, const int* row_q_start, const int* row_q_len, const int* chunk_base, int rows,
                                     int max_chunks, int H, int G, int dk, int dv, float q_scale, float guard, int dtype,
                                     cudaStream_t stream) {
  if (rows == 0 || max_chunks == 0) return 0;
  if (int e = check_sizes("delta_rule_chunked", rows, H, G, dk, dv)) return e;
  DK_REQUIRE(max_chunks > 0 && dk_delta_rule_chunked_supported(dk, dv), "delta_rule_chunked: heads of %d x %d do not fit the shared memory", dk, dv);
  DK_REQUIRE(dtype == DK_F32 || dtype == DK_BF16, "delta_rule_chunked: unknown dtype %d", dtype);
  DK_REQUIRE(((uintptr_t)work % 16) == 0, "delta_rule_chunked: the working memory is not 16-byte aligned");
  static bool granted[DK_MAX_DEVICES] = {false};
  const int dev = dk_current_device();
  if (!granted[dev]) {
    if (cudaFuncSetAttribute(delta_chunk_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT) != cudaSuccess ||
        cudaFuncSetAttribute(delta_chunk_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT) != cudaSuccess ||
        cudaFuncSetAttribute(delta_walk_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT) != cudaSuccess ||
        cudaFuncSetAttribute(delta_walk_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT) != cudaSuccess) {
      cudaGetLastError();
      DK_REQUIRE(false, "delta_rule_chunked: %zu bytes of shared memory were not granted", SMEM_LIMIT);
    }
    granted[dev] = true;
  }
  const dim3 grid(max_chunks, rows * H);
  const int vec = dk % 8 == 0 && stride % 8 == 0 && k_off % 8 == 0 && a_stride % 4 == 0 && ((uintptr_t)qkv % 16) == 0 && ((uintptr_t)a % 16) == 0 &&
                  ((uintptr_t)dt_bias % 16) == 0;
  if (dtype == DK_F32)
    delta_chunk_kernel<float><<<grid, PREP_THREADS, prep_smem(dk), stream>>>((const float*)qkv, stride, k_off, v_off, (const float*)b, b_stride, a, a_stride,
                                                                             A_log, dt_bias, work, row_q_start, row_q_len, chunk_base, H, G, dk, dv, q_scale, guard, vec);
  else
    delta_chunk_kernel<__nv_bfloat16><<<grid, PREP_THREADS, prep_smem(dk), stream>>>((const __nv_bfloat16*)qkv, stride, k_off, v_off, (const __nv_bfloat16*)b,
                                                                                     b_stride, a, a_stride, A_log, dt_bias, work, row_q_start, row_q_len,
                                                                                     chunk_base, H, G, dk, dv, q_scale, guard, vec);
  if (int e = dk_check_launch("delta_rule_chunked")) return e;
  const dim3 walk((dv + WALK_COLS - 1) / WALK_COLS, rows * H);
  if (walk_smem(dk, 2) <= SMEM_LIMIT)
    delta_walk_kernel<2><<<walk, WALK_THREADS, walk_smem(dk, 2), stream>>>(work, state, out, row_slot, row_q_start, row_q_len, chunk_base, H, dk, dv);
  else
    delta_walk_kernel<1><<<walk, WALK_THREADS, walk_smem(dk, 1), stream>>>(work, state, out, row_slot, row_q_start, row_q_len, chunk_base, H, dk, dv);
  return dk_check_launch("delta_rule_chunked");
}
