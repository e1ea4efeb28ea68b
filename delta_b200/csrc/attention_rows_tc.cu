// Paged attention over a cache of rows (row_attention_params.h) on the fifth-generation tensor cores (tcgen05), bfloat16: rows
// that bring several tokens (portions of prompts), causal, optionally a window or chunks, a sink and a gate per head.
//
// The plan is that of attention_prefill_tc.cu: a block owns 128 queries of one head, keys and values come in tiles of 128 cached
// rows, both products run as tcgen05.mma with the accumulators in tensor memory (TMEM), and tiles alternate between two halves of the
// block (softmax warps 4w..4w+3, scores S_w, accumulator O_w) that do not wait for each other and are merged at the end.
// What differs:
//
//   * Key and value of a token lie in one cached row, at offsets and with sizes of their own (multiples of 8, 64 to 128 entries): two
//     tensor maps over the same memory.  Sizes between 64 and 128 take boxes of two times 64 columns whose last ones the TMA
//     fills with zeros.
//   * The softmax weights keep 16 bits of mantissa: P = P_hi + P_lo, both bfloat16, two products per value tile.  P takes the place of
//     the scores it was made from in TMEM (128 columns of float scores are 64 columns of P_hi and 64 of P_lo) and is the A operand
//     from there, so it costs no shared memory and no copy; the scores of the half's next tile wait for the products with P.
//   * Pages of a tile that no query of the block sees (before the window or chunk, given back already, or behind the last token)
//     are replaced by one that is there: their scores are masked, and what is multiplied by the zeros is finite.
//
//   warps 0-7   softmax: thread r of a half owns query r, which is lane r of the TMEM
//   warps 8, 9  producers, one for keys and one for values
//   warp 10     issues the score products, warp 11 the products with the values
//
// Every wait is bounded; when one gives up the block records it, stores nothing more, frees its tensor memory and returns.
#include "common.cuh"
#include "row_attention_params.h"
#include "tcgen05_helpers.cuh"

namespace {
constexpr int QT = 128;            // queries per block (rows of both MMAs)
constexpr int KT = 128;            // keys per tile
constexpr int HALF_THREADS = 128;  // softmax threads of one half
constexpr int PRODUCER_WARP0 = 8, MMA_WARP = 10;   // warp 10 issues the score products, warp 11 the P V products
constexpr int THREADS = (MMA_WARP + 2) * 32;
constexpr int BOX_BYTES = 128 * 128;   // 128 rows of one 128-byte swizzle row each
constexpr float RESCALE_STEP = 8.f;    // in powers of two
constexpr int TMEM_COLS = 512;
constexpr int COL_S = 0, COL_O = 2 * KT;   // S_0, S_1, then O_0, O_1

// DKP, DVP: key and value sizes rounded up to whole boxes of 64 columns.
template <int DKP, int DVP>
struct Layout {
  static constexpr int K_HALVES = DKP / 64, V_HALVES = DVP / 64;
  static constexpr int STAGES = 2;    // two, because a stage is freed by the barrier of the tile two before (see the producers)
  static constexpr int Q_BYTES = K_HALVES * BOX_BYTES;
  static constexpr int K_BYTES = K_HALVES * BOX_BYTES, V_BYTES = V_HALVES * BOX_BYTES;
  static constexpr int OFF_Q = 0;
  static constexpr int OFF_K = OFF_Q + Q_BYTES;
  static constexpr int OFF_V = OFF_K + STAGES * K_BYTES;
  static constexpr int OFF_STAT = OFF_V + STAGES * V_BYTES;            // maximum and sum of each half's queries, for the merge
  static constexpr int TOTAL = OFF_STAT + 2 * QT * 8 + 1024;          // 1024 to start on a swizzle boundary
};

// 2^x by the special-function unit (two units in the last place; results below 2^-126 become 0)
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// One piece of work: 128 queries of one head of one row.  Pieces are numbered with the head fastest, then the rows,
// then the query tiles of each row from its latest (which has the most keys) to its first: from long to short.
struct Piece {
  int row, h, qt, nq, t0, pos0, last_pos, kt_first, n_tiles, first_page, last_page;
  bool valid;
};

__device__ __forceinline__ Piece piece_of(const DkRowAttnParams& p, int index, int row_lo, int n_rows) {
  Piece w;
  w.h = index % p.H;
  w.row = row_lo + (index / p.H) % n_rows;
  const int yy = index / (p.H * n_rows);                // 0: the row's latest query tile, which has the most keys
  const int q_len = p.row_q_len[w.row];
  w.qt = (q_len + QT - 1) / QT - 1 - yy;
  const int q0 = w.qt * QT;
  w.valid = !(p.row_filter == 2 && q_len == 1) && w.qt >= 0;
  w.nq = min(QT, q_len - q0);
  w.t0 = p.row_q_start[w.row] + q0;
  w.pos0 = p.row_pos_start[w.row] + q0;
  w.last_pos = w.pos0 + w.nq - 1;
  const int lo = row_first_key(p, w.pos0);
  w.kt_first = lo / KT;
  w.first_page = lo / p.ps;
  w.n_tiles = w.valid ? w.last_pos / KT - w.kt_first + 1 : 0;
  w.last_page = w.last_pos / p.ps;
  return w;
}

// A block takes several pieces, one after the other.  With as many blocks as SMs
// the barriers, the tensor memory and the descriptors are set up once per SM instead of once per piece, and the next
// piece's queries, first keys and first scores are asked for and computed while the softmax threads still merge and
// write the piece before.  Every barrier is used by the tiles of one parity (tile j of a piece by the barriers of
// class j % 2, as is its stage of K and V), so what a wait needs is the number of tiles of that class the block
// has had so far: `had[c]`, counted alike by every warp.
template <int DKP, int DVP>
__global__ void __launch_bounds__(THREADS, 1) attention_rows_tc_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                       const __grid_constant__ CUtensorMap map_k,
                                                                       const __grid_constant__ CUtensorMap map_k_run,
                                                                       const __grid_constant__ CUtensorMap map_v,
                                                                       const __grid_constant__ CUtensorMap map_v_run,
                                                                       const DkRowAttnParams p, const int n_qt) {
  using L = Layout<DKP, DVP>;
  constexpr int STAGES = L::STAGES;
  static_assert(STAGES == 2, "a stage belongs to the tiles of one parity");

  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  // barriers: q_full, k_full[2], v_full[2], s_full[2], p_full[2], o_done[2], merge, piece_done
  __shared__ __align__(8) unsigned long long bars[1 + 2 + 2 + 2 + 2 + 2 + 1 + 1];
  auto row_stat = [&](int w) { return reinterpret_cast<float2*>(smem + L::OFF_STAT + w * QT * 8); };     // maximum and sum of half w's tiles, per query
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int failed;
  __shared__ int row_range[2];

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ps = p.ps, G = p.H / p.KV;

  const uint32_t bar0 = s2u(&bars[0]);
  const uint32_t q_full = bar0;
  const uint32_t k_full = bar0 + 8, v_full = k_full + 16, s_full = v_full + 16, p_full = s_full + 16, o_done = p_full + 16,
                 merge_bar = o_done + 16, piece_done = merge_bar + 8;
  if (tid == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(k_full + 8 * s, 1);
      mbar_init(v_full + 8 * s, 1);
    }
    for (int w = 0; w < 2; ++w) {
      mbar_init(s_full + 8 * w, 1);
      mbar_init(p_full + 8 * w, HALF_THREADS);
      mbar_init(o_done + 8 * w, 1);
    }
    mbar_init(merge_bar, 2 * HALF_THREADS);
    mbar_init(piece_done, 2 * HALF_THREADS);
    failed = 0;
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    // In a step that also holds single tokens (which the decode kernel takes) only the rows from the first to the
    // last one that brings several tokens are cut into pieces: a block does not have to walk over hundreds of rows
    // that are not its business.
    int lo = p.rows, hi = -1;
    if (p.row_filter == 2) {
      for (int r0 = 0; r0 < p.rows; r0 += 32) {
        const int r = r0 + lane;
        if (r < p.rows && p.row_q_len[r] > 1) {
          lo = min(lo, r);
          hi = max(hi, r);
        }
      }
      lo = __reduce_min_sync(0xffffffffu, lo);
      hi = __reduce_max_sync(0xffffffffu, hi);
    } else {
      lo = 0;
      hi = p.rows - 1;
    }
    if (lane == 0) {
      row_range[0] = lo;
      row_range[1] = hi;
    }
  }
  if (warp == MMA_WARP) tmem_alloc(s2u(&tmem_slot), TMEM_COLS);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const int row_lo = row_range[0], n_rows = max(0, row_range[1] - row_range[0] + 1);
  const int n_pieces = p.H * n_qt * n_rows;
  // The pieces a block takes: in rounds of gridDim.x pieces, forwards in the even rounds and backwards in the odd ones.
  // Pieces are numbered from long to short, so a block that got a long one in one round gets a short one in the next,
  // and all blocks end at about the same time without asking each other anything.
  auto piece_index = [&](int round) {
    const int b = (round & 1) ? (int)gridDim.x - 1 - (int)blockIdx.x : (int)blockIdx.x;
    return round * (int)gridDim.x + b;
  };
  const uint32_t tmem = tmem_slot;
  const uint32_t sm_q = s2u(smem + L::OFF_Q), sm_k = s2u(smem + L::OFF_K), sm_v = s2u(smem + L::OFF_V);
  int had0 = 0, had1 = 0;   // tiles of each parity in the pieces before the current one (scalars: an array indexed by a
                            // value the compiler does not know would live in local memory)
  int n_done = 0;           // pieces before the current one

  // The four warps that fetch and issue need few registers, the eight softmax warps hold a row of 128 scores each:
  // the first warpgroup gives registers back and the other two take them (384 threads x 168 = 128 x 64 + 256 x 216).
  // (Each change of the register count stands inside the branch whose code it is for: after a common point the
  // compiler would have to assume the smaller count for everybody.)
  if (warp >= PRODUCER_WARP0) {
  asm volatile("setmaxnreg.dec.sync.aligned.u32 64;\n");
  if (warp < MMA_WARP) {      // (the three branches of this warpgroup keep their indentation)
    // ----------------------------------------------------------- producers
    // one warp for K and one for V, so that the next K is never held up behind a V whose buffer
    // is still being read
    const int kind = warp - PRODUCER_WARP0;     // 0: K, 1: V
    const int ppt = KT / ps;      // pages per tile, at most 16
    // A stage of K is free when the scores made from it are complete, a stage of V when the product
    // with it is: the producers wait on the same barriers as the softmax threads.
    const uint32_t full = kind ? v_full : k_full, done = kind ? o_done : s_full, sm_dst = kind ? sm_v : sm_k;
    const uint32_t tile_bytes = kind ? L::V_BYTES : L::K_BYTES;
    const int halves = kind ? L::V_HALVES : L::K_HALVES;
    const CUtensorMap* map_page = kind ? &map_v : &map_k;
    const CUtensorMap* map_run = kind ? &map_v_run : &map_k_run;
    int q_asked = 0;
    int asked0 = 0, asked1 = 0;   // tiles of each parity asked for so far
    for (int round = 0; round * (int)gridDim.x < n_pieces && !failed; ++round) {
      const int index = piece_index(round);
      if (index >= n_pieces) continue;
      const Piece w = piece_of(p, index, row_lo, n_rows);
      if (!w.valid) continue;
      const int kvh = w.h / G;
      if (kind == 0) {
        // the queries' buffer is free when every score product of the piece before is complete
        bool ok = true;
        if (n_done > 0) ok = mbar_wait(s_full, (had0 - 1) & 1) && mbar_wait(s_full + 8, (had1 - 1) & 1);
        if (!__all_sync(0xffffffffu, ok && !failed)) { failed = 1; break; }
        if (lane == 0) {
          mbar_expect_tx(q_full, (uint32_t)L::Q_BYTES);
          for (int half = 0; half < L::K_HALVES; ++half)      // (columns behind the head's last one meet zeros of the keys)
            tma_load_2d(sm_q + half * BOX_BYTES, &map_q, w.h * p.q_head_stride + half * 64, w.t0, q_full);   // rows past the last token are zeros
        }
        q_asked = n_done + 1;
      }
      for (int j = 0; j < w.n_tiles; ++j) {
        const int c = j & 1, ord = (c ? had1 : had0) + j / 2;     // the ord-th tile of its parity in this block
        const int lp = (w.kt_first + j) * ppt + lane;
        int page = -1;
        if (lane < ppt && lp >= w.first_page && lp <= w.last_page && lp < p.max_pages) {
          page = p.block_table[(size_t)w.row * p.max_pages + lp];
          if (page < 0 || page >= p.num_pages) {
            dk_report(p.err, DK_DEV_BAD_PAGE, w.row, lp, page);
            page = -1;
          }
        }
        const int first = __shfl_sync(0xffffffffu, page, 0);
        // a tile whose pages follow one another in the pool comes with one request per half of the head
        const bool run = __all_sync(0xffffffffu, lane >= ppt || (page >= 0 && page == first + lane));
        const uint32_t there = __ballot_sync(0xffffffffu, page >= 0);
        const int other = there != 0 ? __shfl_sync(0xffffffffu, page, __ffs(there) - 1) : 0;
        if (page < 0) page = other;
        const int grow = (page * p.KV + kvh) * ps;    // row of the cache seen as [pages * KV * ps, row_width]
        bool ok = true;
        if (ord >= 1) ok = mbar_wait(done + 8 * c, (ord - 1) & 1);
        if (!__all_sync(0xffffffffu, ok && !failed)) { failed = 1; break; }
        if (lane == 0) mbar_expect_tx(full + 8 * c, tile_bytes);
        __syncwarp();
        if (run) {
          if (lane == 0)
            for (int half = 0; half < halves; ++half)
              tma_load_4d(sm_dst + c * tile_bytes + half * BOX_BYTES, map_run, half * 64, 0, kvh, first, full + 8 * c);
        } else if (lane < ppt) {
          for (int half = 0; half < halves; ++half)
            tma_load_2d(sm_dst + c * tile_bytes + half * BOX_BYTES + lane * ps * 128, map_page, half * 64, grow, full + 8 * c);
        }
        if (c) asked1 = ord + 1; else asked0 = ord + 1;
      }
      if (failed) break;
      had0 += (w.n_tiles + 1) / 2;
      had1 += w.n_tiles / 2;
      ++n_done;
    }
    if (failed && lane == 0) {
      // nobody may leave while copies of this block are in flight: wait (bounded) for the last ones asked for
      if (kind == 0 && q_asked > 0) mbar_wait(q_full, (q_asked - 1) & 1);
      if (asked0 > 0) mbar_wait(full, (asked0 - 1) & 1);
      if (asked1 > 0) mbar_wait(full + 8, (asked1 - 1) & 1);
    }
  } else if (warp == MMA_WARP) {
    // ------------------------------------------- MMA issuer of the scores
    // The whole warp runs the loop, so that descriptors and addresses stay warp-uniform; one
    // elected lane issues.  The scores of a tile are computed as soon as its keys have arrived and the products
    // with the P of the tile of the same parity before it, which lies where they go, are complete.
    const bool leader = elect_one();
    const uint32_t idesc_s = instr_desc_bf16(QT, KT, false);
    auto wait_all = [&](uint32_t bar, uint32_t parity) -> bool {     // the same answer in every lane
      return __all_sync(0xffffffffu, mbar_wait(bar, parity));
    };
    const uint64_t da0 = smem_desc_k_major(sm_q);
    bool ok = true;
    for (int round = 0; ok && round * (int)gridDim.x < n_pieces; ++round) {
      const int index = piece_index(round);
      if (index >= n_pieces) continue;
      const Piece w = piece_of(p, index, row_lo, n_rows);
      if (!w.valid) continue;
      ok = wait_all(q_full, n_done & 1);
      for (int j = 0; ok && j < w.n_tiles; ++j) {
        const int c = j & 1, ord = (c ? had1 : had0) + j / 2;
        if (ord >= 1 && !wait_all(o_done + 8 * c, (ord - 1) & 1)) { ok = false; break; }
        if (!wait_all(k_full + 8 * c, ord & 1)) { ok = false; break; }
        tc_fence_after();
        const uint64_t db0 = smem_desc_k_major(sm_k + c * L::K_BYTES);
        if (leader) {
#pragma unroll
          for (int kk = 0; kk < DKP / 16; ++kk) {
            const uint64_t off = (uint64_t)(((kk / 4) * BOX_BYTES + (kk % 4) * 32) >> 4);   // start addresses count 16 bytes
            umma(tmem + COL_S + c * KT, da0 + off, db0 + off, idesc_s, kk > 0 ? 1u : 0u);
          }
          umma_commit(s_full + 8 * c);
        }
        __syncwarp();
      }
      had0 += (w.n_tiles + 1) / 2;
      had1 += w.n_tiles / 2;
      ++n_done;
    }
    if (!ok) failed = 1;
  } else if (warp == MMA_WARP + 1) {
    // ------------------------------------------ MMA issuer of P V
    const bool leader = elect_one();
    const uint32_t idesc_o = instr_desc_bf16(QT, DVP, true);
    auto wait_all = [&](uint32_t bar, uint32_t parity) -> bool {
      return __all_sync(0xffffffffu, mbar_wait(bar, parity));
    };
    bool ok = true;
    for (int round = 0; ok && round * (int)gridDim.x < n_pieces; ++round) {
      const int index = piece_index(round);
      if (index >= n_pieces) continue;
      const Piece w = piece_of(p, index, row_lo, n_rows);
      if (!w.valid) continue;
      for (int j = 0; ok && j < w.n_tiles; ++j) {
        const int c = j & 1, ord = (c ? had1 : had0) + j / 2;
        if (!wait_all(v_full + 8 * c, ord & 1) || !wait_all(p_full + 8 * c, ord & 1)) { ok = false; break; }
        tc_fence_after();
        const uint32_t tp = tmem + COL_S + c * KT;      // P_hi, then P_lo: 8 columns per 16 keys
        const uint64_t dv0 = smem_desc_mn_major(sm_v + c * L::V_BYTES, BOX_BYTES);
        if (leader) {
#pragma unroll
          for (int kk = 0; kk < KT / 16; ++kk) {   // 16 keys further: two groups of 8 rows of V
            const uint64_t dv = dv0 + (uint64_t)(kk * (2048 >> 4));
            umma_a_tmem(tmem + COL_O + c * DVP, tp + kk * 8, dv, idesc_o, (j > 1 || kk > 0) ? 1u : 0u);
            umma_a_tmem(tmem + COL_O + c * DVP, tp + KT / 2 + kk * 8, dv, idesc_o, 1u);
          }
          umma_commit(o_done + 8 * c);
        }
        __syncwarp();
      }
      had0 += (w.n_tiles + 1) / 2;
      had1 += w.n_tiles / 2;
      ++n_done;
    }
    if (!ok) failed = 1;
  }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 216;\n");
    // ------------------------------------------------------------- softmax
    const int w = warp >> 2;                            // which half: its tiles are w, w + 2, ...
    const int r = (warp & 3) * 32 + lane;               // query of this thread = lane of the TMEM
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t t_s = tmem + lane_base + COL_S + w * KT;    // scores of this half
    const uint32_t t_o = tmem + lane_base + COL_O + w * DVP;
    const float sl2 = p.scale * 1.4426950408889634f;
    bool good = true;
    int had_w = 0;            // tiles of this half in the pieces before the current one
#pragma unroll 1
    for (int round = 0; good && round * (int)gridDim.x < n_pieces; ++round) {
      const int index = piece_index(round);
      if (index >= n_pieces) continue;
      const Piece pc = piece_of(p, index, row_lo, n_rows);
      if (!pc.valid) continue;
      const int n_tiles = pc.n_tiles, pos0 = pc.pos0, last_pos = pc.last_pos, kt_first = pc.kt_first, nq = pc.nq, t0 = pc.t0, h = pc.h;
      const int qpos = pos0 + r;
      const int q_first = row_first_key(p, qpos), last_first = row_first_key(p, last_pos);      // the first keys this and the last query see
      float m_used = -INFINITY, l_sum = 0.f;
      int mine = 0;                                       // tiles of this half in this piece so far
      // Before this half lets the P V product overwrite an accumulator, and before it leaves a maximum and sum again, both halves
      // must have finished reading them for the piece before.
      if (n_done > 0) {
        bool ok = mbar_wait(piece_done, (n_done - 1) & 1);
        if (!__all_sync(0xffffffffu, ok && !failed)) { failed = 1; good = false; break; }
      }
      for (int j = w; j < n_tiles; j += 2, ++mine) {
        const int ord = had_w + mine;
        bool ok = mbar_wait(s_full + 8 * w, ord & 1);
        if (!__all_sync(0xffffffffu, ok && !failed)) { failed = 1; good = false; break; }
        tc_fence_after();
        const int kbase = (kt_first + j) * KT;
        const bool edge = (kbase + KT - 1 > pos0) || kbase < last_first;
        // the whole row comes into registers in one round trip
        float v[KT];
#pragma unroll
        for (int c = 0; c < KT / 32; ++c) tmem_ld32_nowait(t_s + c * 32, v + c * 32);
        tmem_wait_ld();
        if (edge) {
          const int hi = qpos - kbase, lo = q_first - kbase;
#pragma unroll
          for (int i = 0; i < KT; ++i)     // key kbase + i is seen by query qpos when it is not later and not before its first one
            if (!(i <= hi && i >= lo)) v[i] = -INFINITY;
        }
        float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};   // four chains instead of one long one
#pragma unroll
        for (int i = 0; i < KT; i += 4) {
          mx4[0] = fmaxf(mx4[0], v[i]);
          mx4[1] = fmaxf(mx4[1], v[i + 1]);
          mx4[2] = fmaxf(mx4[2], v[i + 2]);
          mx4[3] = fmaxf(mx4[3], v[i + 3]);
        }
        const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
        const float m_new = fmaxf(m_used, mx * sl2);
        const bool grow = m_new > m_used + RESCALE_STEP;      // also the first finite maximum of a row
        float factor = 1.f;
        if (grow) {
          factor = m_used == -INFINITY ? 0.f : fast_exp2(m_used - m_new);
          m_used = m_new;
        }
        const float neg_m = m_used == -INFINITY ? 0.f : -m_used;
        if (mine > 0) {
          // P V of this half's tile before is done (these scores could not lie here otherwise): O_w is at rest
          ok = mbar_wait(o_done + 8 * w, (ord - 1) & 1);
          if (!__all_sync(0xffffffffu, ok && !failed)) { failed = 1; good = false; break; }
          if (__any_sync(0xffffffffu, grow)) {
            tc_fence_after();
#pragma unroll 1
            for (int c = 0; c < DVP / 32; ++c) {
              float o[32];
              tmem_ld32_nowait(t_o + c * 32, o);
              tmem_wait_ld();
#pragma unroll
              for (int i = 0; i < 32; ++i) o[i] *= factor;
              tmem_st32(t_o + c * 32, o);
            }
            tmem_wait_st();
            tc_fence_before();
          }
        }
        // exponentials, their sum, and P in two bfloat16 parts over the scores: row r in lane r, two keys a column
        float sum4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int c = 0; c < KT / 32; ++c) {
          uint32_t hi[16], lo[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const float e0 = fast_exp2(fmaf(v[c * 32 + 2 * i], sl2, neg_m)), e1 = fast_exp2(fmaf(v[c * 32 + 2 * i + 1], sl2, neg_m));
            sum4[(2 * i) & 3] += e0;
            sum4[(2 * i + 1) & 3] += e1;
            const __nv_bfloat162 h2 = __floats2bfloat162_rn(e0, e1);
            hi[i] = *reinterpret_cast<const uint32_t*>(&h2);
            lo[i] = pack2(e0 - __low2float(h2), e1 - __high2float(h2));
          }
          tmem_st16(t_s + c * 16, hi);
          tmem_st16(t_s + KT / 2 + c * 16, lo);
        }
        tmem_wait_st();
        tc_fence_before();
        l_sum = l_sum * factor + ((sum4[0] + sum4[1]) + (sum4[2] + sum4[3]));
        mbar_arrive(p_full + 8 * w);
      }
      if (good && mine > 0) {
        bool ok = mbar_wait(o_done + 8 * w, (had_w + mine - 1) & 1);
        if (!__all_sync(0xffffffffu, ok && !failed)) { failed = 1; good = false; }
      }
      // merge of the two halves: each tells the other its maximum and sum, then writes half of the columns
      row_stat(w)[r] = make_float2(m_used, l_sum);
      tc_fence_before();
      mbar_arrive(merge_bar);
      if (good) {
        bool ok = mbar_wait(merge_bar, n_done & 1);
        if (!__all_sync(0xffffffffu, ok && !failed)) { failed = 1; good = false; }
      }
      if (good) {
        tc_fence_after();
        const float2 other = row_stat(w ^ 1)[r];
        const float sink2 = p.sink != nullptr ? p.sink[h] * 1.4426950408889634f : -INFINITY;      // the sink: a key with this logit and no value
        const float m_all = fmaxf(fmaxf(m_used, other.x), sink2);
        const float f_mine = m_used == -INFINITY ? 0.f : fast_exp2(m_used - m_all);
        const float f_other = other.x == -INFINITY ? 0.f : fast_exp2(other.x - m_all);
        float l_all = l_sum * f_mine + other.y * f_other;
        if (p.sink != nullptr) l_all += fast_exp2(sink2 - m_all);
        const float inv = l_all > 0.f ? (r < nq ? row_head_gate<__nv_bfloat16>(p, t0 + r, h) : 1.f) / l_all : 0.f;
        const float f0 = (w == 0 ? f_mine : f_other) * inv, f1 = (w == 0 ? f_other : f_mine) * inv;
        const bool two = n_tiles > 1;                     // O_1 holds nothing when there was one tile
        constexpr int OC = DVP / 64;                      // chunks of 32 columns this thread writes
        __nv_bfloat16* orow = reinterpret_cast<__nv_bfloat16*>(p.out) + ((size_t)(t0 + r) * p.H + h) * p.dv;
#pragma unroll
        for (int c = 0; c < OC; ++c) {
          float o0[32], o1[32];
          const uint32_t col = (uint32_t)(w * (DVP / 2) + c * 32);
          tmem_ld32_nowait(tmem + lane_base + COL_O + col, o0);
          if (two) tmem_ld32_nowait(tmem + lane_base + COL_O + DVP + col, o1);
          tmem_wait_ld();
          if (c == OC - 1) {
            // the accumulators and the other half's maximum and sum are in registers: the next piece may overwrite them
            tc_fence_before();
            mbar_arrive(piece_done);
          }
          if (r < nq) {
#pragma unroll
            for (int i = 0; i < 32; ++i) o0[i] = two ? o0[i] * f0 + o1[i] * f1 : o0[i] * f0;
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              uint4 st;
              st.x = pack2(o0[v * 8], o0[v * 8 + 1]);
              st.y = pack2(o0[v * 8 + 2], o0[v * 8 + 3]);
              st.z = pack2(o0[v * 8 + 4], o0[v * 8 + 5]);
              st.w = pack2(o0[v * 8 + 6], o0[v * 8 + 7]);
              if ((int)col + v * 8 < p.dv) *reinterpret_cast<uint4*>(orow + col + v * 8) = st;      // (value sizes are multiples of 8)
            }
          }
        }
      }
      had_w += (n_tiles + 1 - w) / 2;
      ++n_done;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (failed && tid == 0) dk_report(p.err, DK_DEV_TIMEOUT, (int)blockIdx.x, (int)gridDim.x, n_pieces);
  if (warp == MMA_WARP) tmem_dealloc(tmem, TMEM_COLS);
}

template <int DKP, int DVP>
int launch(const DkRowAttnParams& p, int max_q_len, cudaStream_t stream) {
  using L = Layout<DKP, DVP>;
  CUtensorMap map_q, map_k, map_k_run, map_v, map_v_run;
  const long long rows = (long long)p.num_pages * p.KV * p.ps;
  DK_REQUIRE(rows < (1ll << 31), "attention_rows_tc: the cache of one layer has too many rows for a tensor map coordinate");
  DK_REQUIRE(make_tensor_map_bf16(&map_q, p.q, p.T, (p.H - 1) * p.q_head_stride + p.dk, p.q_stride, QT),
             "attention_rows_tc: cannot encode the tensor map of the queries");
  // the cache as rows, and as [page][head][offset][columns]: a run of pages of one head in one box; once from the key's first
  // column on and once from the value's, each as wide as the key or value
  const unsigned long long strides[3] = {(unsigned long long)p.row_width * 2, (unsigned long long)p.ps * p.row_width * 2,
                                         (unsigned long long)p.KV * p.ps * p.row_width * 2};
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.cache);
  for (int kind = 0; kind < 2; ++kind) {
    const __nv_bfloat16* base = cache + (kind ? p.v_off : p.k_off);
    const int cols = kind ? p.dv : p.dk;
    const unsigned long long dims[4] = {(unsigned long long)cols, (unsigned long long)p.ps, (unsigned long long)p.KV, (unsigned long long)p.num_pages};
    DK_REQUIRE(make_tensor_map_bf16(kind ? &map_v : &map_k, base, rows, cols, p.row_width, p.ps) &&
               make_tensor_map_bf16_4d(kind ? &map_v_run : &map_k_run, base, dims, strides, p.ps, KT / p.ps),
               "attention_rows_tc: cannot encode a tensor map of the cache");
  }
  static bool configured_on[DK_MAX_DEVICES] = {false};
  bool& configured = configured_on[dk_current_device()];
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attention_rows_tc_kernel<DKP, DVP>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) {
      dk_set_error("attention_rows_tc: cannot get %d bytes of shared memory: %s", L::TOTAL, cudaGetErrorString(e));
      return DK_ERR_LAUNCH;
    }
    configured = true;
  }
  const int n_qt = (max_q_len + QT - 1) / QT;
  const long long pieces = (long long)p.H * n_qt * p.rows;
  DK_REQUIRE(pieces < (1ll << 30), "attention_rows_tc: too many pieces of work");
  const int sms = dk_sm_count();
  attention_rows_tc_kernel<DKP, DVP><<<(int)(pieces < sms ? pieces : sms), THREADS, L::TOTAL, stream>>>(map_q, map_k, map_k_run, map_v, map_v_run, p, n_qt);
  return dk_check_launch("attention_rows_tc");
}
}  // namespace

extern "C" int dk_attention_rows_tc_supported(const DkRowAttnParams* pp) {
  const DkRowAttnParams& p = *pp;
  if (p.dtype != DK_BF16 || p.KV <= 0 || p.H % p.KV != 0) return 0;
  if (p.dk % 8 || p.dv % 8 || p.dk < 64 || p.dk > 128 || p.dv < 64 || p.dv > 128) return 0;
  if (p.row_width % 8 || p.k_off % 8 || p.v_off % 8 || p.q_stride % 8 || p.q_head_stride % 8) return 0;
  if (p.ps != 8 && p.ps != 16 && p.ps != 32 && p.ps != 64 && p.ps != 128) return 0;
  if (p.softcap > 0.f || p.dist_bias != nullptr || !(p.scale > 0.f)) return 0;
  if (((uintptr_t)p.q % 16) || ((uintptr_t)p.cache % 16) || ((uintptr_t)p.out % 16)) return 0;
  return 1;
}

// max_q_len: the most tokens any row brings (sizes the grid).
extern "C" int dk_attention_rows_tc(const DkRowAttnParams* pp, int max_q_len, cudaStream_t stream) {
  const DkRowAttnParams& p = *pp;
  if (p.T == 0 || p.rows == 0) return 0;
  DK_REQUIRE(dk_attention_rows_tc_supported(pp), "attention_rows_tc: sizes not taken (bfloat16; key and value sizes multiples of 8 from 64 to 128; "
             "page size 8 to 128 and a power of two; offsets and strides multiples of 8; a positive scale; no shaped scores): dk=%d dv=%d width=%d "
             "ps=%d", p.dk, p.dv, p.row_width, p.ps);
  DK_REQUIRE(max_q_len >= 1, "attention_rows_tc: max_q_len must be positive");
  DK_REQUIRE(p.window >= 0 && p.chunk >= 0, "attention_rows_tc: bad window %d or chunk %d", p.window, p.chunk);
  DK_REQUIRE(p.gate == nullptr || p.gate_stride >= p.H, "attention_rows_tc: rows of %d gates do not hold %d heads", p.gate_stride, p.H);
  DK_REQUIRE(p.row_q_start && p.row_q_len && p.row_pos_start && p.block_table, "attention_rows_tc: row tables are missing");
  DK_REQUIRE((max_q_len + QT - 1) / QT <= 65535 && p.rows <= 65535, "attention_rows_tc: grid too large");
  if (p.dk <= 64) return p.dv <= 64 ? launch<64, 64>(p, max_q_len, stream) : launch<64, 128>(p, max_q_len, stream);
  return p.dv <= 64 ? launch<128, 64>(p, max_q_len, stream) : launch<128, 128>(p, max_q_len, stream);
}
