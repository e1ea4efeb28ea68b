// Between the first product of an attention layer and the attention kernel, for designs whose queries, keys and values go through a
// short causal convolution: one pass from the projected rows src[t] = [q (H*dk) | k (KV*dk) | v (KV*dv)] to finished queries and
// cache rows.  Per channel c, with `taps` weights w[j][c] and zeros before a request's first token:
//
//   u(t)   = sum_j w[j][c] * src(t - (taps - 1) + j)[c]          (taps == 0: u = src)
//   q, k:    x = u / sqrt(mean over the head of u^2 + eps) * norm[i]     (no norm weight: x = u), then rotary positions on the first
//            rot_dims entries; q goes to q_out, k to the token's cache row
//   v:       value mixing with a matrix `first` [T, KV*dv] shared by a group of layers: the group's first layer stores its v there
//            (mix_mode 1), the later ones take (1 - lambda) v + lambda first (mix_mode 2); then the cache row
//
// Everything between the projected rows and the one rounding of the result is 32 bit.  A request's last taps - 1 projected rows are
// its state, conv_state [slot][taps-1][C] (C = (H+KV)*dk + KV*dv); steps in which every row brings one token move it on in the same
// kernel, other steps in a launch behind it.
#include "common.cuh"

extern "C" int dk_conv_state(const void* xin, int in_stride, float* conv_state, const int* row_slot, const int* row_q_start,
                             const int* row_q_len, int rows, int C, int taps, int dtype, cudaStream_t stream);

namespace {
constexpr int WARPS = 4;          // units of a block
constexpr int TILE = 8;           // tokens a warp takes in turn on prompt portions (inputs stay in registers between them)
constexpr int VEC_TILE = 4;       // and side by side in the form for heads of 64 or 128
constexpr int MAX_TAPS = 16;

struct RowsConv {
  const void* src;
  const float* w;            // [taps][C]
  float* conv_state;
  void* q_out;               // [T, H*dk]
  void* cache;               // [num_pages, KV, ps, row_width] or null
  void* first;               // [T, KV*dv]
  const int *tok_pos, *tok_row, *row_slot, *row_q_start, *block_table;
  const float *table, *q_norm, *k_norm;
  int* err;
  int src_stride, T, H, KV, dk, dv, taps, C, ps, row_width, k_off, v_off, max_pages, num_pages;
  int table_positions, rot_dims, interleaved, mix_mode, single;
  float eps, lambda;
};

// Where a unit (a query head, a key head or a value head) reads and what it is.
struct Unit {
  int kind;      // 0 query, 1 key, 2 value
  int head, c0, D;
};
__device__ __forceinline__ Unit unit_of(const RowsConv& p, int u) {
  Unit r;
  if (u < p.H + p.KV) {
    r.kind = u < p.H ? 0 : 1;
    r.head = u < p.H ? u : u - p.H;
    r.c0 = u * p.dk;
    r.D = p.dk;
  } else {
    r.kind = 2;
    r.head = u - p.H - p.KV;
    r.c0 = (p.H + p.KV) * p.dk + r.head * p.dv;
    r.D = p.dv;
  }
  return r;
}

// The token's cache row of a key-value head (null: nothing is appended, or its page is bad and was reported).
template <typename T>
__device__ __forceinline__ T* cache_row(const RowsConv& p, int t, int pos, int row, int head, int lane) {
  if (p.cache == nullptr) return nullptr;
  const int lp = pos / p.ps;
  const int page = lp < p.max_pages ? p.block_table[(size_t)row * p.max_pages + lp] : -1;
  if (page < 0 || page >= p.num_pages) {
    if (lane == 0) dk_report(p.err, DK_DEV_BAD_PAGE, t, lp, page);
    return nullptr;
  }
  return reinterpret_cast<T*>(p.cache) + (((size_t)page * p.KV + head) * p.ps + pos % p.ps) * p.row_width;
}

__device__ __forceinline__ bool good_position(const RowsConv& p, int t, int pos, int lane) {
  if (pos >= 0 && (p.table == nullptr || pos < p.table_positions)) return true;
  if (lane == 0) dk_report(p.err, DK_DEV_BAD_POSITION, t, pos, p.table_positions);
  return false;
}

// Entry i of a head behind the rotation, from the whole head in shared memory; cs: the position's cos and sin.
__device__ __forceinline__ float rotated(const RowsConv& p, const float* x, const float* cs, int i) {
  const float v = x[i];
  if (cs == nullptr || i >= p.rot_dims) return v;
  const int half = p.rot_dims / 2;
  int j, other;
  bool front;
  if (p.interleaved) {
    j = i >> 1;
    front = !(i & 1);
    other = i ^ 1;
  } else {
    front = i < half;
    j = front ? i : i - half;
    other = front ? i + half : i - half;
  }
  const float c = cs[2 * j], s = cs[2 * j + 1];
  return front ? v * c - x[other] * s : v * c + x[other] * s;
}

// Any size: one warp a (unit, token), the entries of a head in turn through shared memory.
template <typename T>
__global__ void __launch_bounds__(WARPS * 32) rows_conv_kernel(const RowsConv p) {
  extern __shared__ float sm[];      // [WARPS][max(dk, dv)]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int u = blockIdx.y * WARPS + warp, t = blockIdx.x;
  if (u >= p.H + 2 * p.KV) return;
  const Unit un = unit_of(p, u);
  float* x = sm + (size_t)warp * max(p.dk, p.dv);
  const int row = p.tok_row[t], pos = p.tok_pos[t];
  const int q0 = p.row_q_start[row];
  const T* src = reinterpret_cast<const T*>(p.src) + un.c0;
  float* st = p.taps > 1 ? p.conv_state + (size_t)p.row_slot[row] * (p.taps - 1) * p.C + un.c0 : nullptr;
  float ss = 0.f;
  for (int i = lane; i < un.D; i += 32) {
    float acc;
    if (p.taps == 0) {
      acc = to_f32<T>(src[(size_t)t * p.src_stride + i]);
    } else {
      acc = 0.f;
      for (int j = 0; j < p.taps; ++j) {
        const int k = t - q0 - (p.taps - 1) + j;      // index among the row's tokens of this step; negative: before it
        const float v = k >= 0 ? to_f32<T>(src[(size_t)(q0 + k) * p.src_stride + i]) : st[(size_t)(p.taps - 1 + k) * p.C + i];
        acc = fmaf(p.w[(size_t)j * p.C + un.c0 + i], v, acc);
      }
      if (p.single && p.taps > 1) {
        for (int j = 0; j + 1 < p.taps - 1; ++j) st[(size_t)j * p.C + i] = st[(size_t)(j + 1) * p.C + i];
        st[(size_t)(p.taps - 2) * p.C + i] = to_f32<T>(src[(size_t)t * p.src_stride + i]);
      }
    }
    x[i] = acc;
    ss += acc * acc;
  }
  if (!good_position(p, t, pos, lane)) return;
  T* crow = un.kind == 0 ? nullptr : cache_row<T>(p, t, pos, row, un.head, lane);
  if (un.kind == 2) {
    T* first = p.mix_mode ? reinterpret_cast<T*>(p.first) + ((size_t)t * p.KV + un.head) * p.dv : nullptr;
    for (int i = lane; i < un.D; i += 32) {
      float v = x[i];
      if (p.mix_mode == 1) first[i] = from_f32<T>(v);
      if (p.mix_mode == 2) v = (1.f - p.lambda) * v + p.lambda * to_f32<T>(first[i]);
      if (crow != nullptr) crow[p.v_off + i] = from_f32<T>(v);
    }
    return;
  }
  const float* nw = un.kind == 0 ? p.q_norm : p.k_norm;
  if (nw != nullptr) {
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)un.D + p.eps);
    for (int i = lane; i < un.D; i += 32) x[i] = x[i] * inv * nw[i];
  }
  __syncwarp();
  const float* cs = p.table != nullptr ? p.table + (size_t)pos * p.rot_dims : nullptr;
  T* out = un.kind == 0 ? reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.H + un.head) * p.dk : (crow != nullptr ? crow + p.k_off : nullptr);
  if (out == nullptr) return;
  for (int i = lane; i < un.D; i += 32) out[i] = from_f32<T>(rotated(p, x, cs, i));
}

template <typename T>
__device__ __forceinline__ float2 load2(const T* p);
template <>
__device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <>
__device__ __forceinline__ float2 load2<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
template <typename T>
__device__ __forceinline__ void store2(T* p, float2 v);
template <>
__device__ __forceinline__ void store2<float>(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
template <>
__device__ __forceinline__ void store2<__nv_bfloat16>(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }

// 2 to 4 taps and even sizes of up to 64 NP entries a head: a lane holds the entry pairs 2 lane + 64 j of its unit, with the window of
// inputs in registers, over `tile` tokens that follow one another.
template <typename T, int TAPS, int NP>
__global__ void __launch_bounds__(WARPS * 32) rows_conv_pairs_kernel(const RowsConv p, int tile) {
  extern __shared__ float sm[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int u = blockIdx.y * WARPS + warp;
  if (u >= p.H + 2 * p.KV) return;
  const Unit un = unit_of(p, u);
  float* x = sm + (size_t)warp * max(p.dk, p.dv);
  const int t_from = blockIdx.x * tile, t_to = min(t_from + tile, p.T);
  const T* src = reinterpret_cast<const T*>(p.src) + un.c0;
  const float* nw = un.kind == 0 ? p.q_norm : (un.kind == 1 ? p.k_norm : nullptr);
  float2 wv[TAPS][NP], win[TAPS - 1][NP], nv[NP];
  bool live[NP];
#pragma unroll
  for (int n = 0; n < NP; ++n) {
    const int i = 2 * lane + 64 * n;
    live[n] = i < un.D;
    nv[n] = make_float2(1.f, 1.f);
    if (live[n] && nw != nullptr) nv[n] = load2<float>(nw + i);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wv[j][n] = live[n] ? load2<float>(p.w + (size_t)j * p.C + un.c0 + i) : make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) win[j][n] = make_float2(0.f, 0.f);
  }
  int row = -1, page_of = -1;
  float* st = nullptr;
  T* page_base = nullptr;
  for (int t = t_from; t < t_to; ++t) {
    const int r = p.tok_row[t], pos = p.tok_pos[t];
    if (r != row) {      // the first token of the tile, or of a row: the inputs before it
      row = r;
      page_of = -1;
      const int q0 = p.row_q_start[row];
      st = p.conv_state + (size_t)p.row_slot[row] * (TAPS - 1) * p.C + un.c0;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int k = t - q0 - (TAPS - 1) + j;
#pragma unroll
        for (int n = 0; n < NP; ++n) {
          const int i = 2 * lane + 64 * n;
          if (live[n]) win[j][n] = k >= 0 ? load2<T>(src + (size_t)(q0 + k) * p.src_stride + i) : load2<float>(st + (size_t)(TAPS - 1 + k) * p.C + i);
        }
      }
    }
    float2 a[NP];
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NP; ++n) {
      const int i = 2 * lane + 64 * n;
      const float2 now = live[n] ? load2<T>(src + (size_t)t * p.src_stride + i) : make_float2(0.f, 0.f);
      a[n] = make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        a[n].x = fmaf(wv[j][n].x, win[j][n].x, a[n].x);
        a[n].y = fmaf(wv[j][n].y, win[j][n].y, a[n].y);
      }
      a[n].x = fmaf(wv[TAPS - 1][n].x, now.x, a[n].x);
      a[n].y = fmaf(wv[TAPS - 1][n].y, now.y, a[n].y);
      ss += a[n].x * a[n].x + a[n].y * a[n].y;
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j) win[j][n] = win[j + 1][n];
      win[TAPS - 2][n] = now;
      if (p.single && live[n]) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) store2<float>(st + (size_t)j * p.C + i, win[j][n]);
      }
    }
    if (!good_position(p, t, pos, lane)) continue;
    T* crow = nullptr;
    if (un.kind != 0 && p.cache != nullptr) {
      if (pos / p.ps != page_of) {      // the page is looked up once per page
        page_of = pos / p.ps;
        T* at = cache_row<T>(p, t, pos, row, un.head, lane);
        page_base = at != nullptr ? at - (size_t)(pos % p.ps) * p.row_width : nullptr;
      }
      if (page_base != nullptr) crow = page_base + (size_t)(pos % p.ps) * p.row_width;
    }
    if (un.kind == 2) {
      T* first = p.mix_mode ? reinterpret_cast<T*>(p.first) + ((size_t)t * p.KV + un.head) * p.dv : nullptr;
#pragma unroll
      for (int n = 0; n < NP; ++n) {
        const int i = 2 * lane + 64 * n;
        if (!live[n]) continue;
        float2 v = a[n];
        if (p.mix_mode == 1) store2<T>(first + i, v);
        if (p.mix_mode == 2) {
          const float2 f = load2<T>(first + i);
          v.x = (1.f - p.lambda) * v.x + p.lambda * f.x;
          v.y = (1.f - p.lambda) * v.y + p.lambda * f.y;
        }
        if (crow != nullptr) store2<T>(crow + p.v_off + i, v);
      }
      continue;
    }
    const float inv = nw != nullptr ? 1.f / sqrtf(warp_sum(ss) / (float)un.D + p.eps) : 1.f;
    const float* cs = p.table != nullptr ? p.table + (size_t)pos * p.rot_dims : nullptr;
#pragma unroll
    for (int n = 0; n < NP; ++n) {
      a[n].x *= inv * nv[n].x;
      a[n].y *= inv * nv[n].y;
      if (cs != nullptr && live[n]) *reinterpret_cast<float2*>(x + 2 * lane + 64 * n) = a[n];
    }
    T* out = un.kind == 0 ? reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.H + un.head) * p.dk : (crow != nullptr ? crow + p.k_off : nullptr);
    if (cs != nullptr) {
      __syncwarp();
#pragma unroll
      for (int n = 0; n < NP; ++n) {
        const int i = 2 * lane + 64 * n;
        if (live[n]) a[n] = make_float2(rotated(p, x, cs, i), rotated(p, x, cs, i + 1));
      }
      __syncwarp();
    }
    if (out != nullptr) {
#pragma unroll
      for (int n = 0; n < NP; ++n)
        if (live[n]) store2<T>(out + 2 * lane + 64 * n, a[n]);
    }
  }
}

// bfloat16, 2 to 4 taps, heads of 32 VEC entries: a lane holds VEC entries that follow one another, and a warp takes TILE tokens of a row
// with every load under way before the first sum is needed; the rotation's partner entries come from another lane.  The inputs
// of earlier steps are bfloat16 values kept in 32 bit, so they are packed again without a loss.
template <int VEC>
struct Raw {
  uint32_t r[VEC / 2];
};
template <int VEC>
__device__ __forceinline__ Raw<VEC> load_raw(const __nv_bfloat16* p) {
  Raw<VEC> v;
  if constexpr (VEC == 2) v.r[0] = *reinterpret_cast<const uint32_t*>(p);
  else {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    v.r[0] = a.x;
    v.r[1] = a.y;
  }
  return v;
}
template <int VEC>
__device__ __forceinline__ void store_raw(__nv_bfloat16* p, const float (&v)[VEC]) {
  uint32_t r[VEC / 2];
#pragma unroll
  for (int e = 0; e < VEC / 2; ++e) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
    r[e] = *reinterpret_cast<const uint32_t*>(&h);
  }
  if constexpr (VEC == 2) *reinterpret_cast<uint32_t*>(p) = r[0];
  else *reinterpret_cast<uint2*>(p) = make_uint2(r[0], r[1]);
}
template <int VEC>
__device__ __forceinline__ void load_floats(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 2) {
    const float2 a = *reinterpret_cast<const float2*>(p);
    v[0] = a.x; v[1] = a.y;
  } else {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  }
}
template <int VEC>
__device__ __forceinline__ void unpack(const Raw<VEC>& raw, float (&v)[VEC]) {
#pragma unroll
  for (int e = 0; e < VEC / 2; ++e) {
    v[2 * e] = __uint_as_float(raw.r[e] << 16);
    v[2 * e + 1] = __uint_as_float(raw.r[e] & 0xffff0000u);
  }
}

// The n <= TILE tokens from t0 on, all of batch row `row`.
template <int TAPS, int VEC, int TILE>
__device__ __forceinline__ void conv_tile(const RowsConv& p, const Unit& un, int t0, int n, int row, int lane) {
  using bf16 = __nv_bfloat16;
  const int i = lane * VEC;
  const bf16* src = reinterpret_cast<const bf16*>(p.src) + un.c0 + i;
  const int q0 = p.row_q_start[row], pos0 = p.tok_pos[t0];
  float* st = p.conv_state + (size_t)p.row_slot[row] * (TAPS - 1) * p.C + un.c0 + i;
  Raw<VEC> raw[TILE + TAPS - 1];
#pragma unroll
  for (int k = 0; k < TILE; ++k)
    if (k < n) raw[TAPS - 1 + k] = load_raw<VEC>(src + (size_t)(t0 + k) * p.src_stride);
#pragma unroll
  for (int k = 0; k < TAPS - 1; ++k) {
    const int at = t0 - q0 - (TAPS - 1) + k;      // index among the row's tokens of this step; negative: before it
    if (at >= 0) {
      raw[k] = load_raw<VEC>(src + (size_t)(q0 + at) * p.src_stride);
    } else {
      float v[VEC];
      load_floats<VEC>(st + (size_t)(TAPS - 1 + at) * p.C, v);
#pragma unroll
      for (int e = 0; e < VEC / 2; ++e) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
        raw[k].r[e] = *reinterpret_cast<const uint32_t*>(&h);
      }
    }
  }
  float w[TAPS][VEC], nw[VEC];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_floats<VEC>(p.w + (size_t)j * p.C + un.c0 + i, w[j]);
  const float* norm = un.kind == 0 ? p.q_norm : (un.kind == 1 ? p.k_norm : nullptr);
#pragma unroll
  for (int e = 0; e < VEC; ++e) nw[e] = 1.f;
  if (norm != nullptr) load_floats<VEC>(norm + i, nw);
  float a[TILE][VEC], ss[TILE];
#pragma unroll
  for (int k = 0; k < TILE; ++k) {
    ss[k] = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) a[k][e] = 0.f;
    if (k < n) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        float v[VEC];
        unpack<VEC>(raw[k + j], v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) a[k][e] = fmaf(w[j][e], v[e], a[k][e]);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss[k] += a[k][e] * a[k][e];
    }
  }
  if (TILE == 1 && p.single) {      // the last TAPS - 1 inputs, this one included
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      float v[VEC];
      unpack<VEC>(raw[j + 1], v);
#pragma unroll
      for (int e = 0; e < VEC; e += 2) *reinterpret_cast<float2*>(st + (size_t)j * p.C + e) = make_float2(v[e], v[e + 1]);
    }
  }
  if (un.kind == 2) {
#pragma unroll
    for (int k = 0; k < TILE; ++k) {
      if (k >= n || !good_position(p, t0 + k, pos0 + k, lane)) continue;
      bf16* first = p.mix_mode ? reinterpret_cast<bf16*>(p.first) + ((size_t)(t0 + k) * p.KV + un.head) * p.dv + i : nullptr;
      if (p.mix_mode == 1) store_raw<VEC>(first, a[k]);
      if (p.mix_mode == 2) {
        float f[VEC];
        unpack<VEC>(load_raw<VEC>(first), f);
#pragma unroll
        for (int e = 0; e < VEC; ++e) a[k][e] = (1.f - p.lambda) * a[k][e] + p.lambda * f[e];
      }
      bf16* crow = cache_row<bf16>(p, t0 + k, pos0 + k, row, un.head, lane);
      if (crow != nullptr) store_raw<VEC>(crow + p.v_off + i, a[k]);
    }
    return;
  }
  if (norm != nullptr) {
#pragma unroll
    for (int k = 0; k < TILE; ++k) {
      const float inv = rsqrtf(warp_sum(ss[k]) * (1.f / (32 * VEC)) + p.eps);
#pragma unroll
      for (int e = 0; e < VEC; ++e) a[k][e] *= inv * nw[e];
    }
  }
  const int half = p.rot_dims / 2;
  const bool turned = p.table != nullptr && i < p.rot_dims, front = i < half;
  const int partner = turned ? (front ? lane + half / VEC : lane - half / VEC) : lane;
  const int j0 = front ? i : i - half;
#pragma unroll
  for (int k = 0; k < TILE; ++k) {
    if (k >= n) continue;
    const int pos = pos0 + k;
    const bool good = good_position(p, t0 + k, pos, lane);
    if (p.table != nullptr) {
      float o[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) o[e] = __shfl_sync(0xffffffffu, a[k][e], partner);
      if (turned && good) {
        const float* cs = p.table + (size_t)pos * p.rot_dims + 2 * j0;
#pragma unroll
        for (int e = 0; e < VEC; e += 2) {
          const float4 t = *reinterpret_cast<const float4*>(cs + 2 * e);      // cos, sin of two pairs
          a[k][e] = front ? a[k][e] * t.x - o[e] * t.y : a[k][e] * t.x + o[e] * t.y;
          a[k][e + 1] = front ? a[k][e + 1] * t.z - o[e + 1] * t.w : a[k][e + 1] * t.z + o[e + 1] * t.w;
        }
      }
    }
    if (!good) continue;
    if (un.kind == 0) {
      store_raw<VEC>(reinterpret_cast<bf16*>(p.q_out) + ((size_t)(t0 + k) * p.H + un.head) * p.dk + i, a[k]);
    } else {
      bf16* crow = cache_row<bf16>(p, t0 + k, pos, row, un.head, lane);
      if (crow != nullptr) store_raw<VEC>(crow + p.k_off + i, a[k]);
    }
  }
}

template <int TAPS, int VK, int VV, int TILE>
__global__ void __launch_bounds__(WARPS * 32) rows_conv_vec_kernel(const RowsConv p) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int u = blockIdx.y * WARPS + warp;
  if (u >= p.H + 2 * p.KV) return;
  const Unit un = unit_of(p, u);
  const int t0 = blockIdx.x * TILE, n = min(TILE, p.T - t0);
  const int row = p.tok_row[t0];
  if (TILE == 1 || p.tok_row[t0 + n - 1] == row) {
    if (un.kind == 2) conv_tile<TAPS, VV, TILE>(p, un, t0, n, row, lane);
    else conv_tile<TAPS, VK, TILE>(p, un, t0, n, row, lane);
  } else {      // the tile's tokens belong to several rows
    for (int k = 0; k < n; ++k) {
      if (un.kind == 2) conv_tile<TAPS, VV, 1>(p, un, t0 + k, 1, p.tok_row[t0 + k], lane);
      else conv_tile<TAPS, VK, 1>(p, un, t0 + k, 1, p.tok_row[t0 + k], lane);
    }
  }
}

template <int TAPS, int TILE>
void launch_vec(const RowsConv& p, dim3 grid, cudaStream_t stream) {
  if (p.dk == 128 && p.dv == 128) rows_conv_vec_kernel<TAPS, 4, 4, TILE><<<grid, WARPS * 32, 0, stream>>>(p);
  else if (p.dk == 128) rows_conv_vec_kernel<TAPS, 4, 2, TILE><<<grid, WARPS * 32, 0, stream>>>(p);
  else if (p.dv == 128) rows_conv_vec_kernel<TAPS, 2, 4, TILE><<<grid, WARPS * 32, 0, stream>>>(p);
  else rows_conv_vec_kernel<TAPS, 2, 2, TILE><<<grid, WARPS * 32, 0, stream>>>(p);
}
template <int TILE>
void launch_vec_taps(const RowsConv& p, dim3 grid, cudaStream_t stream) {
  if (p.taps == 2) launch_vec<2, TILE>(p, grid, stream);
  else if (p.taps == 3) launch_vec<3, TILE>(p, grid, stream);
  else launch_vec<4, TILE>(p, grid, stream);
}

template <typename T, int TAPS>
void launch_pairs(const RowsConv& p, int np, int tile, dim3 grid, size_t smem, cudaStream_t stream) {
  if (np == 1) rows_conv_pairs_kernel<T, TAPS, 1><<<grid, WARPS * 32, smem, stream>>>(p, tile);
  else if (np == 2) rows_conv_pairs_kernel<T, TAPS, 2><<<grid, WARPS * 32, smem, stream>>>(p, tile);
  else rows_conv_pairs_kernel<T, TAPS, 4><<<grid, WARPS * 32, smem, stream>>>(p, tile);
}
template <typename T>
void launch_taps(const RowsConv& p, int np, int tile, dim3 grid, size_t smem, cudaStream_t stream) {
  if (p.taps == 2) launch_pairs<T, 2>(p, np, tile, grid, smem, stream);
  else if (p.taps == 3) launch_pairs<T, 3>(p, np, tile, grid, smem, stream);
  else launch_pairs<T, 4>(p, np, tile, grid, smem, stream);
}
}  // namespace

extern "C" int dk_rows_conv_append(const void* src, int src_stride, const float* w, int taps, float* conv_state, void* q_out, const int* tok_pos,
                                   const int* tok_row, const int* row_slot, const int* row_q_start, const int* row_q_len, int rows,
                                   const int* block_table, int max_pages, void* cache, int num_pages, const float* table,
                                   int table_positions, int rot_dims, int interleaved, const float* q_norm, const float* k_norm, float eps,
                                   void* first, int mix_mode, float lambda, int T_, int H, int KV, int dk, int dv, int ps, int row_width,
                                   int k_off, int v_off, int single, int dtype, int* err, cudaStream_t stream) {
  if (T_ == 0) return 0;
  const int C = (H + KV) * dk + KV * dv;
  DK_REQUIRE(T_ > 0 && rows > 0 && H > 0 && KV > 0 && dk > 0 && dv > 0 && ps > 0, "rows_conv_append: bad sizes T=%d H=%d KV=%d dk=%d dv=%d ps=%d", T_, H,
             KV, dk, dv, ps);
  DK_REQUIRE(src_stride >= C, "rows_conv_append: rows of %d elements do not hold q, k and v", src_stride);
  DK_REQUIRE(taps >= 0 && taps <= MAX_TAPS, "rows_conv_append: %d taps; this kernel takes up to %d", taps, MAX_TAPS);
  DK_REQUIRE(taps == 0 || w != nullptr, "rows_conv_append: the convolution has no weights");
  DK_REQUIRE(taps < 2 || conv_state != nullptr, "rows_conv_append: the convolution has no state");
  DK_REQUIRE(cache == nullptr || (block_table != nullptr && max_pages > 0 && num_pages > 0), "rows_conv_append: a cache is given without a block table");
  DK_REQUIRE(table == nullptr || (rot_dims > 0 && rot_dims % 2 == 0 && rot_dims <= dk), "rows_conv_append: %d rotated entries do not fit a head of %d", rot_dims, dk);
  DK_REQUIRE(k_off >= 0 && v_off >= 0 && k_off + dk <= row_width && v_off + dv <= row_width, "rows_conv_append: key and value do not fit a row of %d", row_width);
  DK_REQUIRE(mix_mode >= 0 && mix_mode <= 2 && (mix_mode == 0 || first != nullptr), "rows_conv_append: value mixing %d without the group's first values", mix_mode);
  DK_REQUIRE((q_norm == nullptr) == (k_norm == nullptr), "rows_conv_append: queries and keys are normed together");
  DK_REQUIRE(dtype == DK_F32 || dtype == DK_BF16, "rows_conv_append: unknown dtype %d", dtype);
  const int D = dk > dv ? dk : dv;
  const size_t smem = (size_t)WARPS * D * sizeof(float);
  DK_REQUIRE(smem <= 48 * 1024, "rows_conv_append: heads of %d entries do not fit the shared memory", D);
  const int units = H + 2 * KV, unit_blocks = (units + WARPS - 1) / WARPS;
  DK_REQUIRE(unit_blocks <= 65535, "rows_conv_append: too many heads");
  RowsConv p{src, w, conv_state, q_out, cache, first, tok_pos, tok_row, row_slot, row_q_start, block_table, table, q_norm, k_norm, err,
             src_stride, T_, H, KV, dk, dv, taps, C, ps, row_width, k_off, v_off, max_pages, num_pages, table_positions, rot_dims, interleaved,
             mix_mode, single, eps, lambda};
  auto aligned = [](const void* q, size_t to) { return q == nullptr || ((uintptr_t)q % to) == 0; };
  const size_t pair = dtype == DK_F32 ? 8 : 4;
  const bool pairs = taps >= 2 && taps <= 4 && dk % 2 == 0 && dv % 2 == 0 && D <= 256 && src_stride % 2 == 0 && row_width % 2 == 0 && k_off % 2 == 0 &&
                     v_off % 2 == 0 && aligned(src, pair) && aligned(q_out, pair) && aligned(cache, pair) && aligned(first, pair) &&
                     aligned(w, 8) && aligned(conv_state, 8) && aligned(q_norm, 8) && aligned(k_norm, 8);
  const int vk = dk / 32;
  const bool vecs = pairs && dtype == DK_BF16 && (dk == 64 || dk == 128) && (dv == 64 || dv == 128) && src_stride % 4 == 0 && row_width % 4 == 0 &&
                    k_off % 4 == 0 && v_off % 4 == 0 && aligned(src, 8) && aligned(q_out, 8) && aligned(cache, 8) && aligned(first, 8) && aligned(w, 16) &&
                    aligned(conv_state, 16) && aligned(q_norm, 16) && aligned(k_norm, 16) && aligned(table, 16) &&
                    (table == nullptr || (!interleaved && (rot_dims / 2) % vk == 0 && rot_dims % 4 == 0));
  if (vecs) {
    // few tokens: one a warp, so that the step has many warps; many: VEC_TILE side by side, so that most inputs are read once
    const bool many = !single && (long long)T_ * units >= 16LL * VEC_TILE * dk_sm_count();
    if (many) launch_vec_taps<VEC_TILE>(p, dim3((T_ + VEC_TILE - 1) / VEC_TILE, unit_blocks), stream);
    else launch_vec_taps<1>(p, dim3(T_, unit_blocks), stream);
  } else if (pairs) {
    const int np = D <= 64 ? 1 : (D <= 128 ? 2 : 4);
    // few tokens: one a warp, so that the step has many warps; many: TILE in turn, so that the inputs are read once
    const int tile = (long long)T_ * units >= 32LL * TILE * dk_sm_count() ? TILE : 1;
    const dim3 grid((T_ + tile - 1) / tile, unit_blocks);
    if (dtype == DK_F32) launch_taps<float>(p, np, tile, grid, smem, stream);
    else launch_taps<__nv_bfloat16>(p, np, tile, grid, smem, stream);
  } else {
    const dim3 grid(T_, unit_blocks);
    if (dtype == DK_F32) rows_conv_kernel<float><<<grid, WARPS * 32, smem, stream>>>(p);
    else rows_conv_kernel<__nv_bfloat16><<<grid, WARPS * 32, smem, stream>>>(p);
  }
  if (int e = dk_check_launch("rows_conv_append")) return e;
  if (taps > 1 && !single) return dk_conv_state(src, src_stride, conv_state, row_slot, row_q_start, row_q_len, rows, C, taps, dtype, stream);
  return 0;
}
