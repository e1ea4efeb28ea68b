// The state-space recurrence with one scalar decay per head ("SSD", the Mamba-2 kind).
//
// Per head h of P channels, with a state S [N, P] in 32 bit that a request carries from token to token and the group
// g = h / (H / G) whose maps B, C [N] it reads:
//     dt = softplus(dtraw_h + dt_bias_h)
//     S <- exp(-exp(A_log_h) dt) S + dt B x^T ,      y = S^T C + D_h x .
// The state is kept with a channel's N entries side by side: [slot][H][P][N].  Everything below is 32-bit FMA whatever the
// type of the inputs.
//
// ssd_rows: tokens in turn, a slice of the channels per block; a channel's state lies in the registers of eight lanes.
// Single tokens (the state streams through registers once) and short portions.
//
// Long portions are cut into chunks of 32 tokens.  With L_t the sum of the log decays of a chunk's tokens 0..t and S the
// state before the chunk,
//     y_t = e^(L_t) S^T C_t + sum_{s<=t} (C_t . B_s) e^(L_t - L_s) dt_s x_s + D x_t
//     S  <- e^(L_last) S + sum_s e^(L_last - L_s) dt_s B_s x_s^T .
//   1. ssd_chunk: every chunk in parallel: the products C_t . B_s of a group, and dt and L of its heads;
//   2. ssd_walk:  along a row, chunk after chunk, a slice of the channels of a head per block; S stays in shared memory.
// No exponent is ever positive.  Sums of log decays are kept as two floats.
#include "common.cuh"
#include "mma_helpers.cuh"

namespace {

__device__ __forceinline__ float softplus_ss(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// ---- tokens in turn --------------------------------------------------------------------------------------------------------
constexpr int ROWS_THREADS = 128;
constexpr int ROWS_TOKENS = 4;
constexpr int LANES = 8;
constexpr int ROWS_COLS = ROWS_THREADS / LANES;

// grid (rows, H, ceil(P / ROWS_COLS)).  NI: groups of 32 state entries (the last may be partly empty).
template <typename T, int NI>
__global__ void __launch_bounds__(ROWS_THREADS)
ssd_rows_kernel(const T* __restrict__ xbc, int stride, const T* __restrict__ dtraw, int dt_stride, const float* __restrict__ A_log,
                const float* __restrict__ dt_bias, const float* __restrict__ D, float* __restrict__ state, float* __restrict__ out,
                const int* __restrict__ row_slot, const int* __restrict__ row_q_start, const int* __restrict__ row_q_len, int H, int G,
                int N, int P, int vec) {
  constexpr int W = NI * 32;
  __shared__ __align__(16) float Bs[ROWS_TOKENS][W], Cs[ROWS_TOKENS][W];
  __shared__ float xs[ROWS_TOKENS][ROWS_COLS], dts[ROWS_TOKENS];
  const int row = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * ROWS_COLS;
  const int n_new = row_q_len != nullptr ? row_q_len[row] : 1;
  if (n_new <= 0) return;
  const int t0 = row_q_start[row], g = h / (H / G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, p = tid & (LANES - 1), col = tid / LANES;
  const bool live = j0 + col < P;
  float* st = state + (((size_t)row_slot[row] * H + h) * P + (live ? j0 + col : 0)) * N;
  float S[NI][4];
#pragma unroll
  for (int m = 0; m < NI; ++m) {
    const int i = 32 * m + 4 * p;
    if (vec) {
      const float4 v = (live && i < N) ? *reinterpret_cast<const float4*>(st + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[m][0] = v.x; S[m][1] = v.y; S[m][2] = v.z; S[m][3] = v.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) S[m][e] = (live && i + e < N) ? st[i + e] : 0.f;
    }
  }
  const float rate = expf(A_log[h]), Dh = D[h];
  for (int c0 = 0; c0 < n_new; c0 += ROWS_TOKENS) {
    const int n = min(ROWS_TOKENS, n_new - c0);
    if (c0 > 0) __syncthreads();
    for (int task = warp; task < 2 * n; task += ROWS_THREADS / 32) {
      const int t = task >> 1, which = task & 1;
      const T* src = xbc + (size_t)(t0 + c0 + t) * stride + (size_t)H * P + (size_t)(which ? G + g : g) * N;
      float* dst = which ? Cs[t] : Bs[t];
#pragma unroll
      for (int m = 0; m < NI; ++m) dst[lane + 32 * m] = lane + 32 * m < N ? to_f32<T>(src[lane + 32 * m]) : 0.f;
    }
    for (int idx = tid; idx < n * ROWS_COLS; idx += ROWS_THREADS) {
      const int t = idx / ROWS_COLS, c = idx - t * ROWS_COLS;
      xs[t][c] = j0 + c < P ? to_f32<T>(xbc[(size_t)(t0 + c0 + t) * stride + (size_t)h * P + j0 + c]) : 0.f;
    }
    if (tid < n) dts[tid] = softplus_ss(to_f32<T>(dtraw[(size_t)(t0 + c0 + tid) * dt_stride + h]) + dt_bias[h]);
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float dt = dts[t], x = xs[t][col], decay = expf(-rate * dt), u = dt * x;
      float y = 0.f;
#pragma unroll
      for (int m = 0; m < NI; ++m) {
        const float4 b = *reinterpret_cast<const float4*>(&Bs[t][32 * m + 4 * p]);
        const float4 c = *reinterpret_cast<const float4*>(&Cs[t][32 * m + 4 * p]);
        S[m][0] = fmaf(decay, S[m][0], b.x * u); S[m][1] = fmaf(decay, S[m][1], b.y * u);
        S[m][2] = fmaf(decay, S[m][2], b.z * u); S[m][3] = fmaf(decay, S[m][3], b.w * u);
        y = fmaf(S[m][0], c.x, y); y = fmaf(S[m][1], c.y, y); y = fmaf(S[m][2], c.z, y); y = fmaf(S[m][3], c.w, y);
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (p == 0 && live) out[(size_t)(t0 + c0 + t) * H * P + (size_t)h * P + j0 + col] = fmaf(Dh, x, y);
    }
  }
  if (!live) return;
#pragma unroll
  for (int m = 0; m < NI; ++m) {
    const int i = 32 * m + 4 * p;
    if (vec) {
      if (i < N) *reinterpret_cast<float4*>(st + i) = make_float4(S[m][0], S[m][1], S[m][2], S[m][3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (i + e < N) st[i + e] = S[m][e];
    }
  }
}

// ---- chunks ----------------------------------------------------------------------------------------------------------------
constexpr int TC = 32;                   // tokens of a chunk: one lane of a warp per token when the decays are prepared
constexpr int TCP = TC + 4;
constexpr int CHUNK_THREADS = 128;
constexpr int WALK_THREADS = 256;       // eight threads for each of a chunk's tokens when they are fetched
constexpr float LOG2E = 1.4426950408889634f;
constexpr float LEAST_LOG2 = -1000.f;    // 2^-1000 is zero in 32 bit: a token's log decay is no smaller, so that sums stay finite
constexpr size_t SMEM_LIMIT = 220 * 1024;
constexpr int HEAD_FLOATS = 3 * TC;      // per (chunk, head): dt, and the sums of log2 decays as two floats
constexpr int GROUP_FLOATS = TC * TC;    // per (chunk, group): C_t . B_s

__host__ __device__ __forceinline__ int pad4(int n) { return (n + 3) & ~3; }

size_t chunk_smem(int N) { return (size_t)(2 * TC * (pad4(N) + 4)) * sizeof(float); }

// grid (most chunks of a row, rows * G).  work: GROUP_FLOATS for all (chunk, group), then HEAD_FLOATS for all (chunk, head).
template <typename T>
__global__ void __launch_bounds__(CHUNK_THREADS)
ssd_chunk_kernel(const T* __restrict__ xbc, int stride, const T* __restrict__ dtraw, int dt_stride, const float* __restrict__ A_log,
                 const float* __restrict__ dt_bias, float* __restrict__ scores, float* __restrict__ heads, const int* __restrict__ row_q_start,
                 const int* __restrict__ row_q_len, const int* __restrict__ chunk_base, int H, int G, int N, int P) {
  extern __shared__ __align__(16) float sm[];
  const int row = blockIdx.y / G, g = blockIdx.y % G, c0 = blockIdx.x * TC, n_new = row_q_len[row];
  if (c0 >= n_new) return;
  const int n = min(TC, n_new - c0), t0 = row_q_start[row] + c0, ld = pad4(N) + 4, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t chunk = (size_t)chunk_base[row] + blockIdx.x;
  float* Cs = sm;                 // [TC][ld]
  float* Bs = Cs + TC * ld;       // [TC][ld]
  for (int idx = tid; idx < 2 * TC * ld; idx += CHUNK_THREADS) {
    const int r = idx / ld, i = idx - r * ld, t = r & (TC - 1);
    const bool isB = r >= TC;
    sm[idx] = (t < n && i < N) ? to_f32<T>(xbc[(size_t)(t0 + t) * stride + (size_t)H * P + (size_t)(isB ? g : G + g) * N + i]) : 0.f;
  }
  for (int h = g * (H / G) + warp; h < (g + 1) * (H / G); h += CHUNK_THREADS / 32) {
    float dt = 0.f;
    double L = 0.0;
    if (lane < n) {
      dt = softplus_ss(to_f32<T>(dtraw[(size_t)(t0 + lane) * dt_stride + h]) + dt_bias[h]);
      L = (double)fmaxf(-expf(A_log[h]) * LOG2E * dt, LEAST_LOG2);
    }
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const double up = __shfl_up_sync(0xffffffffu, L, d);
      if (lane >= d) L += up;
    }
    float* hs = heads + (chunk * H + h) * HEAD_FLOATS;
    const float hi = (float)L;
    hs[lane] = dt;
    hs[TC + lane] = hi;
    hs[2 * TC + lane] = (float)(L - (double)hi);
  }
  __syncthreads();
  float* out = scores + (chunk * G + g) * GROUP_FLOATS;
  const int tt = tid >> 4, ss = tid & 15;      // rows tt + 8 q (q < 4), columns ss and ss + 16
  float acc[4][2] = {};
  for (int i = 0; i < pad4(N); i += 4) {
    float4 b[2], c[4];
#pragma unroll
    for (int y = 0; y < 2; ++y) b[y] = *reinterpret_cast<const float4*>(Bs + (ss + 16 * y) * ld + i);
#pragma unroll
    for (int q = 0; q < 4; ++q) c[q] = *reinterpret_cast<const float4*>(Cs + (tt + 8 * q) * ld + i);
#pragma unroll
    for (int q = 0; q < 4; ++q)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        acc[q][y] = fmaf(c[q].x, b[y].x, acc[q][y]);
        acc[q][y] = fmaf(c[q].y, b[y].y, acc[q][y]);
        acc[q][y] = fmaf(c[q].z, b[y].z, acc[q][y]);
        acc[q][y] = fmaf(c[q].w, b[y].w, acc[q][y]);
      }
  }
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int t = tt + 8 * q, s = ss + 16 * y;
      out[t * TC + s] = s <= t ? acc[q][y] : 0.f;
    }
}

// Bytes of one fetched chunk (C, B and x as they lie in memory, the group's products, the head's dt and sums), and of the whole
// of the walk's shared memory.
template <typename T, int PS>
__host__ __device__ constexpr size_t raw_bytes(int N) {
  return (size_t)(2 * TC * N + TC * PS) * sizeof(T) + (size_t)(GROUP_FLOATS + HEAD_FLOATS) * sizeof(float);
}
__host__ __device__ constexpr int walk_rows(int PS) { return PS / 4; }      // rows of a thread's tile in the walk's first product
template <typename T, int PS>
size_t walk_smem(int N) {
  const int Np = pad4(N), ld = PS + 4, shares = WALK_THREADS / (TC / walk_rows(PS) * (PS / 4));
  return 2 * raw_bytes<T, PS>((N + 7) & ~7) +
         (size_t)(TC * (Np + 4) + TC * Np + TC * ld + TC * TCP + 2 * TC + Np * ld + shares * TC * ld) * sizeof(float);
}

// grid (slices of the channels, rows * H).  VEC: sizes and addresses allow 16-byte copies, and the next chunk is fetched while
// this one is worked on.
template <typename T, int PS, bool VEC>
__global__ void __launch_bounds__(WALK_THREADS)
ssd_walk_kernel(const T* __restrict__ xbc, int stride, const float* __restrict__ scores, const float* __restrict__ heads,
                const float* __restrict__ D, float* __restrict__ state, float* __restrict__ out, const int* __restrict__ row_slot,
                const int* __restrict__ row_q_start, const int* __restrict__ row_q_len, const int* __restrict__ chunk_base, int H, int G,
                int N, int P) {
  constexpr int LD = PS + 4, JT = PS / 4, RT = walk_rows(PS), TI = TC / RT, SHARE_THREADS = TI * JT, SHARES = WALK_THREADS / SHARE_THREADS;
  constexpr int VN = 16 / (int)sizeof(T);      // entries of a 16-byte piece
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int row = blockIdx.y / H, h = blockIdx.y % H, j0 = blockIdx.x * PS, n_new = row_q_len[row];
  if (n_new <= 0) return;
  const int g = h / (H / G), Np = pad4(N), cl = Np + 4, jn = min(PS, P - j0), tid = threadIdx.x, q0 = row_q_start[row];
  const size_t raw = raw_bytes<T, PS>((N + 7) & ~7);
  float* Cs = reinterpret_cast<float*>(smem_raw + 2 * raw);      // [TC][cl]
  float* Bs = Cs + TC * cl;                                      // [TC][Np]: times e^(L_last - L_s) dt_s
  float* X = Bs + TC * Np;                                       // [TC][LD]
  float* M = X + TC * LD;                                        // [TC][TCP]: (C_t . B_s) e^(L_t - L_s) dt_s
  float* wo = M + TC * TCP;                                      // [TC]: e^(L_t)
  float* wi = wo + TC;                                           // [TC]: e^(L_last - L_s) dt_s
  float* S = wi + TC;                                            // [Np][LD]
  float* part = S + Np * LD;                                     // [SHARES][TC][LD]
  const int chunks = (n_new + TC - 1) / TC;
  const size_t first = chunk_base[row];
  auto piece = [&](int c) { return reinterpret_cast<T*>(smem_raw + (size_t)(c & 1) * raw); };      // C | B | x, then floats
  auto fetch = [&](int c) {
    const int n = min(TC, n_new - c * TC);
    T* rc = piece(c);
    T* rx = rc + 2 * TC * N;
    float* fl = reinterpret_cast<float*>(rx + TC * PS);
    if (VEC) {
      {      // eight threads a token
        const int t = tid >> 3;
        const T* src = xbc + (size_t)(q0 + c * TC + (t < n ? t : 0)) * stride + (size_t)H * P;
        for (int i = (tid & 7) * VN; i < N; i += 8 * VN) {
          cp_async_16(smem_u32(rc + t * N + i), src + (size_t)(G + g) * N + i, t < n);
          cp_async_16(smem_u32(rc + (TC + t) * N + i), src + (size_t)g * N + i, t < n);
        }
      }
      for (int idx = tid; idx < TC * (PS / VN); idx += WALK_THREADS) {
        const int t = idx / (PS / VN), j = (idx - t * (PS / VN)) * VN;
        const bool ok = t < n && j < jn;
        cp_async_16(smem_u32(rx + t * PS + j), xbc + (size_t)(q0 + c * TC + (t < n ? t : 0)) * stride + (size_t)h * P + (ok ? j0 + j : 0), ok);
      }
      const float* sc = scores + ((first + c) * G + g) * GROUP_FLOATS;
      const float* hs = heads + ((first + c) * H + h) * HEAD_FLOATS;
      for (int idx = tid; idx < GROUP_FLOATS / 4; idx += WALK_THREADS) cp_async_16(smem_u32(fl + idx * 4), sc + idx * 4, true);
      for (int idx = tid; idx < HEAD_FLOATS / 4; idx += WALK_THREADS) cp_async_16(smem_u32(fl + GROUP_FLOATS + idx * 4), hs + idx * 4, true);
      cp_async_commit();
    }
  };
  if (VEC) fetch(0);
  float* st = state + (((size_t)row_slot[row] * H + h) * P + j0) * N;
  for (int idx = tid; idx < Np * PS; idx += WALK_THREADS) {
    const int j = idx / Np, i = idx - j * Np;
    S[i * LD + j] = (i < N && j < jn) ? st[(size_t)j * N + i] : 0.f;
  }
  const float Dh = D[h];
  const int share = tid / SHARE_THREADS, r = tid % SHARE_THREADS, ti = r / JT, tj = r % JT;
  for (int c = 0; c < chunks; ++c) {
    const int n = min(TC, n_new - c * TC);
    const float *fs, *hs;
    if (VEC) {
      if (c + 1 < chunks) {
        fetch(c + 1);
        cp_async_wait<1>();
      } else {
        cp_async_wait<0>();
      }
      fs = reinterpret_cast<const float*>(piece(c) + 2 * TC * N + TC * PS);
      hs = fs + GROUP_FLOATS;
    } else {
      fs = scores + ((first + c) * G + g) * GROUP_FLOATS;
      hs = heads + ((first + c) * H + h) * HEAD_FLOATS;
    }
    __syncthreads();
    const float last_h = hs[2 * TC - 1], last_l = hs[3 * TC - 1];      // behind a short chunk's end the sums stay the same
    if (VEC) {
      const T* rc = piece(c);
      const T* rx = rc + 2 * TC * N;
      const int t = tid >> 3;      // eight threads a token
      const float w = exp2f((last_h - hs[TC + t]) + (last_l - hs[2 * TC + t])) * hs[t];
      for (int i = (tid & 7) * 4; i < N; i += 32) {
        const T* pc = rc + t * N + i;
        const T* pb = pc + TC * N;
        *reinterpret_cast<float4*>(Cs + t * cl + i) = make_float4(to_f32<T>(pc[0]), to_f32<T>(pc[1]), to_f32<T>(pc[2]), to_f32<T>(pc[3]));
        *reinterpret_cast<float4*>(Bs + t * Np + i) =
            make_float4(to_f32<T>(pb[0]) * w, to_f32<T>(pb[1]) * w, to_f32<T>(pb[2]) * w, to_f32<T>(pb[3]) * w);
      }
      for (int idx = tid; idx < TC * PS; idx += WALK_THREADS) X[(idx / PS) * LD + idx % PS] = to_f32<T>(rx[idx]);
    } else {
      const T* base = xbc + (size_t)(q0 + c * TC) * stride;
      for (int idx = tid; idx < TC * Np; idx += WALK_THREADS) {
        const int t = idx / Np, i = idx - t * Np;
        const float w = exp2f((last_h - hs[TC + t]) + (last_l - hs[2 * TC + t])) * hs[t];
        const bool ok = t < n && i < N;
        const T* p = base + (size_t)t * stride + (size_t)H * P + i;
        Cs[t * cl + i] = ok ? to_f32<T>(p[(size_t)(G + g) * N]) : 0.f;
        Bs[idx] = ok ? to_f32<T>(p[(size_t)g * N]) * w : 0.f;
      }
      for (int idx = tid; idx < TC * PS; idx += WALK_THREADS) {
        const int t = idx / PS, j = idx - t * PS;
        X[t * LD + j] = (t < n && j < jn) ? to_f32<T>(base[(size_t)t * stride + (size_t)h * P + j0 + j]) : 0.f;
      }
    }
    for (int idx = tid; idx < TC * TC; idx += WALK_THREADS) {
      const int t = idx / TC, s = idx % TC;
      M[t * TCP + s] = s <= t ? fs[idx] * exp2f((hs[TC + t] - hs[TC + s]) + (hs[2 * TC + t] - hs[2 * TC + s])) * hs[s] : 0.f;
    }
    if (tid < TC) wo[tid] = exp2f(hs[TC + tid] + hs[2 * TC + tid]);
    const float keep = exp2f(last_h + last_l);
    __syncthreads();
    {      // C S: a thread takes the rows ti + TI q and four columns; the state entries are shared out over groups of threads
      float acc[RT][4] = {};
      for (int i4 = share; i4 < Np / 4; i4 += SHARES) {
        float4 s[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) s[q] = *reinterpret_cast<const float4*>(S + (4 * i4 + q) * LD + 4 * tj);
#pragma unroll
        for (int q = 0; q < RT; ++q) {
          const float4 x = *reinterpret_cast<const float4*>(Cs + (ti + TI * q) * cl + 4 * i4);
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
      for (int q = 0; q < RT; ++q)
        *reinterpret_cast<float4*>(part + ((size_t)share * TC + ti + TI * q) * LD + 4 * tj) = make_float4(acc[q][0], acc[q][1], acc[q][2], acc[q][3]);
    }
    __syncthreads();
    for (int idx = tid; idx < TC * JT; idx += WALK_THREADS) {      // the chunk's outputs
      const int t = idx / JT, j = (idx % JT) * 4;
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int q = 0; q < SHARES; ++q) {
        const float4 v = *reinterpret_cast<const float4*>(part + ((size_t)q * TC + t) * LD + j);
        o.x += v.x; o.y += v.y; o.z += v.z; o.w += v.w;
      }
      const float w = wo[t];
      const float4 xt = *reinterpret_cast<const float4*>(X + t * LD + j);
      o.x = fmaf(Dh, xt.x, o.x * w); o.y = fmaf(Dh, xt.y, o.y * w); o.z = fmaf(Dh, xt.z, o.z * w); o.w = fmaf(Dh, xt.w, o.w * w);
#pragma unroll 4
      for (int s4 = 0; s4 < TC / 4; ++s4) {
        const float4 m = *reinterpret_cast<const float4*>(M + t * TCP + 4 * s4);
        const float mv[4] = {m.x, m.y, m.z, m.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 x = *reinterpret_cast<const float4*>(X + (4 * s4 + e) * LD + j);
          o.x = fmaf(mv[e], x.x, o.x); o.y = fmaf(mv[e], x.y, o.y); o.z = fmaf(mv[e], x.z, o.z); o.w = fmaf(mv[e], x.w, o.w);
        }
      }
      if (t < n) {
        float* dst = out + (size_t)(q0 + c * TC + t) * H * P + (size_t)h * P + j0 + j;
        const float ov[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (j + e < jn) dst[e] = ov[e];
      }
    }
    for (int tile = tid; tile < Np / 4 * JT; tile += WALK_THREADS) {      // the state behind the chunk
      const int i = (tile / JT) * 4, j = (tile % JT) * 4;
      float acc[4][4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float4 s = *reinterpret_cast<const float4*>(S + (i + x) * LD + j);
        acc[x][0] = keep * s.x; acc[x][1] = keep * s.y; acc[x][2] = keep * s.z; acc[x][3] = keep * s.w;
      }
#pragma unroll 8
      for (int s = 0; s < TC; ++s) {
        const float4 b = *reinterpret_cast<const float4*>(Bs + s * Np + i);
        const float4 x = *reinterpret_cast<const float4*>(X + s * LD + j);
        const float bx[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int y = 0; y < 4; ++y) {
          acc[y][0] = fmaf(bx[y], x.x, acc[y][0]);
          acc[y][1] = fmaf(bx[y], x.y, acc[y][1]);
          acc[y][2] = fmaf(bx[y], x.z, acc[y][2]);
          acc[y][3] = fmaf(bx[y], x.w, acc[y][3]);
        }
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) *reinterpret_cast<float4*>(S + (i + x) * LD + j) = make_float4(acc[x][0], acc[x][1], acc[x][2], acc[x][3]);
    }
    // the next round's first barrier keeps its writes to Cs .. wo behind these reads
    __syncthreads();
  }
  for (int idx = tid; idx < N * jn; idx += WALK_THREADS) {
    const int j = idx / N, i = idx - j * N;
    st[(size_t)j * N + i] = S[i * LD + j];
  }
}

int check_sizes(const char* who, int rows, int H, int G, int N, int P) {
  DK_REQUIRE(rows > 0 && H > 0 && G > 0 && H % G == 0 && N > 0 && P > 0, "%s: bad sizes rows=%d H=%d G=%d N=%d P=%d", who, rows, H, G, N, P);
  DK_REQUIRE((long long)rows * H <= 65535, "%s: %d rows of %d heads are above the grid's limit", who, rows, H);
  return 0;
}
}  // namespace

extern "C" int dk_state_space_max_state() { return 512; }

// Tokens in turn.  xbc [T, stride]: x (H P) | B (G N) | C (G N).  row_q_len null: every row brings one token.
extern "C" int dk_state_space(const void* xbc, int stride, const void* dtraw, int dt_stride, const float* A_log, const float* dt_bias,
                              const float* D, float* state, float* out, const int* row_slot, const int* row_q_start, const int* row_q_len,
                              int rows, int H, int G, int N, int P, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  if (int e = check_sizes("state_space", rows, H, G, N, P)) return e;
  DK_REQUIRE(N <= 512, "state_space: %d state entries a channel are above the 512 this kernel keeps in registers", N);
  DK_REQUIRE(stride >= H * P + 2 * G * N, "state_space: rows of %d elements do not hold x, B and C", stride);
  DK_REQUIRE(dtype == DK_F32 || dtype == DK_BF16, "state_space: unknown dtype %d", dtype);
  const dim3 grid(rows, H, (P + ROWS_COLS - 1) / ROWS_COLS);
  const int vec = N % 4 == 0 && ((uintptr_t)state % 16) == 0;
#define LAUNCH(T, NI)                                                                                                            \
  ssd_rows_kernel<T, NI><<<grid, ROWS_THREADS, 0, stream>>>((const T*)xbc, stride, (const T*)dtraw, dt_stride, A_log, dt_bias, D, state, \
                                                            out, row_slot, row_q_start, row_q_len, H, G, N, P, vec)
#define PICK(T)                      \
  do {                               \
    if (N <= 32) LAUNCH(T, 1);       \
    else if (N <= 64) LAUNCH(T, 2);  \
    else if (N <= 128) LAUNCH(T, 4); \
    else if (N <= 256) LAUNCH(T, 8); \
    else LAUNCH(T, 16);              \
  } while (0)
  if (dtype == DK_F32) PICK(float);
  else PICK(__nv_bfloat16);
#undef PICK
#undef LAUNCH
  return dk_check_launch("state_space");
}

extern "C" int dk_state_space_chunk() { return TC; }

extern "C" int dk_state_space_chunked_supported(int N, int P, int dtype) {
  return N > 0 && P > 0 && chunk_smem(N) <= SMEM_LIMIT && (dtype == DK_F32 ? walk_smem<float, 16>(N) : walk_smem<__nv_bfloat16, 16>(N)) <= SMEM_LIMIT;
}

// Floats of working memory per chunk.
extern "C" int dk_state_space_chunk_floats(int H, int G) { return G * GROUP_FLOATS + H * HEAD_FLOATS; }

// Long portions.  `chunk_base` [rows]: the number of chunks of all rows before this one; `total_chunks`: of all rows;
// `max_chunks`: the most chunks of a row; `work`: total_chunks x dk_state_space_chunk_floats floats.
extern "C" int dk_state_space_chunked(const void* xbc, int stride, const void* dtraw, int dt_stride, const float* A_log,
                                      const float* dt_bias, const float* D, float* state, float* out, float* work, const int* row_slot,
                                      const int* row_q_start, const int* row_q_len, const int* chunk_base, int rows, int total_chunks,
                                      int max_chunks, int H, int G, int N, int P, int dtype, cudaStream_t stream) {
  if (rows == 0 || max_chunks == 0) return 0;
  if (int e = check_sizes("state_space_chunked", rows, H, G, N, P)) return e;
  DK_REQUIRE(max_chunks > 0 && total_chunks >= max_chunks && dk_state_space_chunked_supported(N, P, dtype),
             "state_space_chunked: heads of %d x %d do not fit the shared memory", N, P);
  DK_REQUIRE(stride >= H * P + 2 * G * N, "state_space_chunked: rows of %d elements do not hold x, B and C", stride);
  DK_REQUIRE(dtype == DK_F32 || dtype == DK_BF16, "state_space_chunked: unknown dtype %d", dtype);
  DK_REQUIRE(((uintptr_t)work % 16) == 0, "state_space_chunked: the working memory is not 16-byte aligned");
  float* scores = work;
  float* heads = work + (size_t)total_chunks * G * GROUP_FLOATS;
  const dim3 cgrid(max_chunks, rows * G);
  static bool granted[DK_MAX_DEVICES] = {false};
  const int dev = dk_current_device();
  bool ok = true;
#define GRANT(...) ok = ok && cudaFuncSetAttribute(__VA_ARGS__, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT) == cudaSuccess
  if (!granted[dev]) {
    GRANT(ssd_chunk_kernel<float>);
    GRANT(ssd_chunk_kernel<__nv_bfloat16>);
    GRANT((ssd_walk_kernel<float, 16, true>));
    GRANT((ssd_walk_kernel<float, 16, false>));
    GRANT((ssd_walk_kernel<float, 32, true>));
    GRANT((ssd_walk_kernel<float, 32, false>));
    GRANT((ssd_walk_kernel<__nv_bfloat16, 16, true>));
    GRANT((ssd_walk_kernel<__nv_bfloat16, 16, false>));
    GRANT((ssd_walk_kernel<__nv_bfloat16, 32, true>));
    GRANT((ssd_walk_kernel<__nv_bfloat16, 32, false>));
    if (!ok) {
      cudaGetLastError();
      DK_REQUIRE(false, "state_space_chunked: %zu bytes of shared memory were not granted", SMEM_LIMIT);
    }
    granted[dev] = true;
  }
#undef GRANT
  const int es = dtype == DK_F32 ? 4 : 2, vn = 16 / es;
  // 16-byte copies: rows, heads and maps begin on such a boundary
  const bool vec = stride % vn == 0 && N % vn == 0 && P % vn == 0 && ((uintptr_t)xbc % 16) == 0 && N % 4 == 0;
  // two slices of 32 channels do less in all than four of 16, which fill the device when there are few heads
  const bool wide = P > 16 && (long long)rows * H * ((P + 31) / 32) * 3 >= 2LL * dk_sm_count() &&
                    (dtype == DK_F32 ? walk_smem<float, 32>(N) : walk_smem<__nv_bfloat16, 32>(N)) <= SMEM_LIMIT;
#define WALK(T, PS, V)                                                                                                             \
  ssd_walk_kernel<T, PS, V><<<dim3((P + PS - 1) / PS, rows * H), WALK_THREADS, walk_smem<T, PS>(N), stream>>>(                     \
      (const T*)xbc, stride, scores, heads, D, state, out, row_slot, row_q_start, row_q_len, chunk_base, H, G, N, P)
#define BOTH(T)                                                                                                                   \
  do {                                                                                                                            \
    ssd_chunk_kernel<T><<<cgrid, CHUNK_THREADS, chunk_smem(N), stream>>>((const T*)xbc, stride, (const T*)dtraw, dt_stride, A_log, \
                                                                         dt_bias, scores, heads, row_q_start, row_q_len, chunk_base, H, \
                                                                         G, N, P);                                                 \
    if (wide && vec) WALK(T, 32, true);                                                                                           \
    else if (wide) WALK(T, 32, false);                                                                                            \
    else if (vec) WALK(T, 16, true);                                                                                              \
    else WALK(T, 16, false);                                                                                                      \
  } while (0)
  if (dtype == DK_F32) BOTH(float);
  else BOTH(__nv_bfloat16);
#undef BOTH
#undef WALK
  return dk_check_launch("state_space_chunked");
}
