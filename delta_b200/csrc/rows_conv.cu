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
  if (pairs) {
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
