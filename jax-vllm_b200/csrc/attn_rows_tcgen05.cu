// Paged causal attention of prompt portions on the 5th-generation tensor cores for scores that are products with a token's
// WHOLE cached key row (scores mixed across heads: talk_prepare.cu forms such queries): NC pieces of 128 elements, the key
// heads side by side, under one value head of 128 per group of query heads.  It is the kernel of attn_tcgen05.cu (persistent
// blocks, work items of up to 128 rows = (token, query head) pairs of one group, 128-key tiles, scores, weights and output in
// tensor memory, two softmax threads a row) with another supply of operands, since a tile needs NC tiles of keys for every
// tile of values:
//
//   queries    up to four pieces of an item stay in shared memory (for NC = 2 those of two items); with one item's place
//              (`ONE`) the output leaves through the place of piece 0, and the other pieces' places are free for the next
//              item as soon as the item's last scores are formed.  Pieces beyond the fourth stream with the keys.
//   ring       everything else comes through ONE ring of 32 KB stages in the order in which the tensor cores take it: the
//              pieces of a tile's keys (a streamed piece's queries before its keys), then the values of the tile before.
//              While a tile's softmax runs, the stages hold the keys to come rather than values that wait for their weights.
//              Within a stage the 8-row groups of both 64-element halves alternate, [8 rows, half 0][8 rows, half 1], so that
//              ONE copy (a 5-D box) brings a page's rows of a piece; the operand descriptors step over the other half.
//   warp 0     producer of all of it;  warp 1  issues the products, and clears the value rows past the last key;  warps
//              2..9  softmax
//
// A piece's product S += Q_c K_c^T needs 128 bytes of shared memory a clock for its operands alone; the softmax of the tile
// before runs beside it.  Every wait on a barrier is bounded by a clock deadline and reports to the status word.
//
// Restrictions: bfloat16, pieces and values of 128, two pieces or more, no window, up to 16 query heads a group, page size a
// power of two from 8 to 128.
#include "tcgen05.cuh"

#include <math.h>

namespace {

constexpr int D = 128, ROWS = 128, BN = 128;
constexpr int TILE_BYTES = 128 * 128 * 2;       // a 128 x 128 bfloat16 tile
constexpr int HALF_BYTES = 128 * 128;           // queries: two halves of [128 rows][128 bytes]
constexpr int GROUP_BYTES = 2048;               // ring stages: an 8-row group of both halves
constexpr int SMEM_TILES = 7;
constexpr int THREADS = 320;                    // producer warp, mma warp, 8 softmax warps
constexpr int SOFTMAX_THREADS = 256;
constexpr int TMEM_COLS = 512;                  // S0: [0,128)  S1: [128,256)  O: [256,384)  P0: [384,448)  P1: [448,512)
constexpr int TMEM_O = 256, TMEM_P = 384;
constexpr int MAX_STAGES = 4;
constexpr int MAX_LISTED = 32;                  // rounds whose item a block looks up once, for all roles
constexpr float LOG2E = 1.4426950408889634f;

// By the number of pieces NC (0: five or more): items whose queries have a place, pieces that stay there, ring stages.
template <int NC> struct Plan;
template <> struct Plan<2> { static constexpr int QB = 2, KEPT = 2; };
template <> struct Plan<3> { static constexpr int QB = 1, KEPT = 3; };
template <> struct Plan<4> { static constexpr int QB = 1, KEPT = 4; };
template <> struct Plan<0> { static constexpr int QB = 1, KEPT = 4; };

struct Params {
  __nv_bfloat16* out; int out_stride;
  const int* block_table; int table_width;
  const int* cu_seqlens; const int* start_pos; const int* work;
  int n_work, n_q_heads, n_kv_heads, page_size, num_pages, hpt, tokens_per_tile;
  float scale_log2, out_scale;
  const float* sink;           // [n_q_heads] or null: exp(sink) counts once in the denominator
  int* status;
};

struct Shared {
  // queries: one pair of barriers an item's place; with one place, pair 0 is for piece 0 and pair 1 for the other pieces
  uint64_t q_full[2], q_free[2], full[MAX_STAGES], empty[MAX_STAGES];
  uint64_t s_full[2], p_full[2], o_done[2];
  uint64_t o_free;              // the softmax threads have read an item's output: the next item's may be written
  uint64_t drain;               // used only after a wait ran out
  uint32_t tmem_base;
  int failed;                   // a role gave up on a wait
  int armed_q[2], armed[MAX_STAGES];   // parity of the phase the producer armed last; -1: never
  int4 items[MAX_LISTED];       // the block's first items: entry, first row, first position, (group << 16 | tokens)
  float xch[2][128];            // a row's two softmax threads exchange their maxima (and at the end their sums)
};

struct Item {
  int entry, kv_head, q_first;      // request of the batch, group of query heads, first row of the tile among all tokens
  int tokens_here, pos_first;       // tokens in the tile, position of the first
  int j_hi, n_tiles;                // keys [0, j_hi) are visible to some row; key tiles
  int turn;                         // the tile that the item begins with

  // The j-th tile that the item takes.  Blocks begin at different tiles: starting all at the first one, they would ask the
  // L2 for the same few lines at the same time.
  __device__ __forceinline__ int tile(int j) const { return j + turn < n_tiles ? j + turn : j + turn - n_tiles; }
};

template <int NCT>
__global__ void __launch_bounds__(THREADS, 1) attn_rows_tcgen05_kernel(const __grid_constant__ CUtensorMap q_map,
                                                                       const __grid_constant__ CUtensorMap k_map,
                                                                       const __grid_constant__ CUtensorMap v_map,
                                                                       const __grid_constant__ CUtensorMap out_map,
                                                                       const Params p) {
  constexpr int QB = Plan<NCT>::QB, KEPT = Plan<NCT>::KEPT, STAGES = SMEM_TILES - QB * KEPT;
  constexpr bool ONE = QB == 1;
  static_assert(STAGES >= 3 && STAGES <= MAX_STAGES, "ring");
  const int NC = NCT > 0 ? NCT : p.n_kv_heads;
  pdl_trigger();
  extern __shared__ unsigned char smem_raw[];
  unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  unsigned char* q_s = base;                                   // [places][pieces][2 halves][128 rows][128 B]
  unsigned char* r_s = q_s + QB * KEPT * TILE_BYTES;           // [stages][16 groups][2 halves][8 rows][128 B]
  Shared* sh = reinterpret_cast<Shared*>(base + SMEM_TILES * TILE_BYTES);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int HPT = p.hpt;
  const int n_items = p.n_work * p.n_kv_heads, n_blocks = gridDim.x;

  // The items of this block: in round r the blocks take the items r G .. r G + G - 1 of the list ordered longest first (the
  // work list is in ascending order of a tile's first token, so from its end), in the order of their numbers in even rounds
  // and against it in odd ones.  The groups of one tile of tokens follow one another, so blocks at work together read the
  // same keys.
  auto item_of_round = [&](int r) -> int {
    const int L = r * n_blocks + ((r & 1) ? n_blocks - 1 - (int)blockIdx.x : (int)blockIdx.x);
    return L < n_items ? L : -1;
  };
  const int n_rounds = (n_items + n_blocks - 1) / n_blocks;
  auto look_up = [&](int r) -> int4 {
    const int L = item_of_round(r);
    if (L < 0) return make_int4(0, 0, 0, 0);
    const int w = p.n_work - 1 - L / p.n_kv_heads, kv_head = L % p.n_kv_heads;
    const int entry = p.work[2 * w], q_off = p.work[2 * w + 1];
    const int q_begin = p.cu_seqlens[entry];
    const int tokens = max(0, min(p.tokens_per_tile, p.cu_seqlens[entry + 1] - q_begin - q_off));
    return make_int4(entry, q_begin + q_off, p.start_pos[entry] + q_off, kv_head << 16 | tokens);
  };
  auto load_item = [&](int r) -> Item {
    const int4 v = r < MAX_LISTED ? sh->items[r] : look_up(r);
    Item it;
    it.entry = v.x;
    it.q_first = v.y;
    it.pos_first = v.z;
    it.kv_head = v.w >> 16;
    it.tokens_here = v.w & 0xffff;
    it.j_hi = it.pos_first + it.tokens_here;
    it.n_tiles = it.tokens_here > 0 ? (it.j_hi + BN - 1) / BN : 0;
    it.turn = it.n_tiles > 0 ? blockIdx.x % it.n_tiles : 0;
    return it;
  };
  // the first item with tiles from round r on; r becomes its round
  auto next_item = [&](int& r, Item& out) -> bool {
    for (; r < n_rounds; ++r) {
      out = load_item(r);
      if (out.n_tiles > 0) return true;
    }
    return false;
  };

  if (threadIdx.x == 0) {
    for (int b = 0; b < 2; ++b) {
      mbar_init(&sh->q_full[b], 1); mbar_init(&sh->q_free[b], 1); sh->armed_q[b] = -1;
      mbar_init(&sh->s_full[b], 1); mbar_init(&sh->p_full[b], SOFTMAX_THREADS); mbar_init(&sh->o_done[b], 1);
    }
    for (int s = 0; s < STAGES; ++s) { mbar_init(&sh->full[s], 1); mbar_init(&sh->empty[s], 1); sh->armed[s] = -1; }
    mbar_init(&sh->o_free, SOFTMAX_THREADS);
    mbar_init(&sh->drain, 1);
    sh->failed = 0;
    mbar_fence_init();
  }
  for (int r = threadIdx.x; r < min(n_rounds, MAX_LISTED); r += THREADS) sh->items[r] = look_up(r);
  __syncthreads();
  // the producer starts at once; the others wait until the second warp has its tensor memory
  if (warp >= 1) {
    if (warp == 1) {
      asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(&sh->tmem_base)), "r"(TMEM_COLS) : "memory");
      asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    TC_FENCE_BEFORE();
    asm volatile("bar.sync 6, 288;\n" ::: "memory");
    TC_FENCE_AFTER();
  }
  const uint32_t tmem = warp >= 1 ? sh->tmem_base : 0u;
  const uint32_t tmem_o = tmem + TMEM_O;

  if (warp == 0) {
    // ---------------------------------------------------------------- producer
    pdl_wait();                         // queries, keys and values are the work of the kernels before this one
    const int P = p.page_size, pages_per_tile = BN / P;
    const int q_bytes = 2 * 128 * HPT * p.tokens_per_tile;      // of one piece: two boxes of 64 d x heads x tokens
    bool ok = true;
    // page ids of a tile: lane i reads the i-th (a tile has at most 16 pages); NOT_NEEDED, or what the table says (-1: none)
    constexpr int NOT_NEEDED = -2;
    auto tile_pages = [&](const Item& it, int j) -> int {
      const int pi = it.tile(j) * pages_per_tile + lane;
      if (lane >= pages_per_tile || pi * P >= it.j_hi) return NOT_NEEDED;
      return pi < p.table_width ? p.block_table[(size_t)it.entry * p.table_width + pi] : -1;
    };
    auto load_q = [&](const Item& it, int c, unsigned char* dst, uint64_t* bar) {
      tma_load_3d(dst, &q_map, c * D, it.kv_head * HPT, it.q_first, bar);
      tma_load_3d(dst + HALF_BYTES, &q_map, c * D + 64, it.kv_head * HPT, it.q_first, bar);
    };
    // a stage with the rows that the lanes' pages hold of piece (or value head) c.  The announcement need not come before the
    // copies: the phase cannot complete before lane 0 has arrived.
    int s_at = 0, s_ph = 0;             // the next stage and the parity of its phase
    auto put_rows = [&](const CUtensorMap* map, int c, int pages, int n_pages) {
      ok = __all_sync(0xffffffffu, mbar_wait(&sh->empty[s_at], s_ph ^ 1)) && ok;
      if (ok) {
        uint64_t* bar = &sh->full[s_at];
        if (lane == 0) { sh->armed[s_at] = s_ph; mbar_expect_tx(bar, n_pages * P * 256); }
        if (pages >= 0) tma_load_5d(r_s + s_at * TILE_BYTES + lane * P * 256, map, 0, 0, 2 * c, 0, pages, bar);
      }
      if (++s_at == STAGES) { s_at = 0; s_ph ^= 1; }
    };
    auto put_queries = [&](const Item& it, int n) {             // the pieces that stay (with one place: all but piece 0)
      if (lane == 0 && ok) {
        const int qb = ONE ? 1 : n % QB, ph = (n / QB) & 1, first = ONE ? 1 : 0;
        ok = mbar_wait(&sh->q_free[qb], ph ^ 1);
        if (ok) {
          sh->armed_q[qb] = ph;
          mbar_expect_tx(&sh->q_full[qb], (KEPT - first) * q_bytes);
          for (int c = first; c < KEPT; ++c) load_q(it, c, q_s + ((n % QB) * KEPT + c) * TILE_BYTES, &sh->q_full[qb]);
        }
      }
      ok = __shfl_sync(0xffffffffu, ok, 0);
    };
    auto put_keys = [&](const Item& it, int n, bool first_tile, int pages, int n_pages) {
      for (int cc = 0; cc < NC; ++cc) {
        const int c = cc + 1 == NC ? 0 : cc + 1;                // piece 0 last
        if (ONE && first_tile && c == 0) {                      // the output of the item before has left through this place
          ok = __all_sync(0xffffffffu, mbar_wait(&sh->q_free[0], (n & 1) ^ 1)) && ok;
          if (ok && lane == 0) { sh->armed_q[0] = n & 1; mbar_expect_tx(&sh->q_full[0], q_bytes); load_q(it, 0, q_s, &sh->q_full[0]); }
        }
        if (NCT == 0 && c >= KEPT) {                            // a streamed piece: its queries first
          ok = __all_sync(0xffffffffu, mbar_wait(&sh->empty[s_at], s_ph ^ 1)) && ok;
          if (ok && lane == 0) {
            sh->armed[s_at] = s_ph;
            mbar_expect_tx(&sh->full[s_at], q_bytes);
            load_q(it, c, r_s + s_at * TILE_BYTES, &sh->full[s_at]);
          }
          if (++s_at == STAGES) { s_at = 0; s_ph ^= 1; }
        }
        put_rows(&k_map, c, pages, n_pages);
      }
    };
    // what the table says -> pages to copy from (-1: none), with a report of those that should be there
    auto usable = [&](int said, int& n_pages) -> int {
      const bool there = said >= 0 && said < p.num_pages;
      if (said != NOT_NEEDED && !there) atomicOr(p.status, JV_STATUS_BAD_PAGE);
      n_pages = __popc(__ballot_sync(0xffffffffu, there));
      return there ? said : -1;
    };
    // the tiles of all items as one sequence; a tile's page ids are asked for two tiles before they are used
    struct At { Item it; int r, n, j; bool valid; };
    auto after = [&](const At& x) -> At {
      At y = x;
      if (!x.valid) return y;
      if (++y.j < x.it.n_tiles) return y;
      y.j = 0;
      ++y.n;
      ++y.r;
      y.valid = next_item(y.r, y.it);
      return y;
    };
    At cur;
    cur.r = cur.n = cur.j = 0;
    cur.valid = next_item(cur.r, cur.it);
    At nxt = after(cur);
    int n_pages = 0, n_pages_next = 0;
    int pages = usable(cur.valid ? tile_pages(cur.it, 0) : NOT_NEEDED, n_pages);
    int said_next = nxt.valid ? tile_pages(nxt.it, nxt.j) : NOT_NEEDED;
    if (cur.valid) {
      put_queries(cur.it, 0);
      put_keys(cur.it, 0, true, pages, n_pages);
    }
    while (cur.valid && ok) {
      const At next2 = after(nxt);
      const int said_next2 = next2.valid ? tile_pages(next2.it, next2.j) : NOT_NEEDED;
      const bool values_first = ONE && (!nxt.valid || nxt.n != cur.n);
      const int pages_next = usable(said_next, n_pages_next);
      if (values_first) put_rows(&v_map, cur.it.kv_head, pages, n_pages);
      if (nxt.valid) {
        if (nxt.n != cur.n) put_queries(nxt.it, nxt.n);
        put_keys(nxt.it, nxt.n, nxt.n != cur.n, pages_next, n_pages_next);
      }
      if (!values_first) put_rows(&v_map, cur.it.kv_head, pages, n_pages);
      cur = nxt;
      nxt = next2;
      pages = pages_next;
      n_pages = n_pages_next;
      said_next = said_next2;
    }
    if (!ok && lane == 0) { atomicOr(p.status, JV_STATUS_WAIT_EXPIRED); sh->failed = 1; }
  } else if (warp == 1) {
    // -------------------------------------------------------------- mma issuer
    // The whole warp walks through the tiles; lane 0 takes a tile's stages of keys and issues the products.
    const uint64_t q_desc = desc_k_major(smem_u32(q_s)), rq_desc = desc_k_major(smem_u32(r_s));
    const uint64_t k_desc = desc_k_major(smem_u32(r_s), GROUP_BYTES);
    const uint64_t v_desc = desc_mn_major(smem_u32(r_s), GROUP_BYTES / 2, GROUP_BYTES);
    int s_at = 0, s_ph = 0;             // the next stage and the parity of its phase
    auto next_stage = [&]() { if (++s_at == STAGES) { s_at = 0; s_ph ^= 1; } };
    auto wait = [&](uint64_t* bar, int parity) -> bool { return __all_sync(0xffffffffu, mbar_wait(bar, parity)); };
    auto issue_qk_lane = [&](int n, int j, int n_tiles, int gt) -> bool {   // S[gt % 2] = sum_c Q_c K_c^T
      if (j == 0 && !mbar_wait(&sh->q_full[ONE ? 1 : n % QB], (n / QB) & 1)) return false;
      const uint32_t tmem_s = tmem + (gt & 1) * 128;
      const uint64_t q_item = q_desc + (uint64_t)(((n % QB) * KEPT * TILE_BYTES) >> 4);
#pragma unroll (NCT > 0 ? NCT : 1)
      for (int cc = 0; cc < NC; ++cc) {
        const int c = cc + 1 == NC ? 0 : cc + 1;
        if (ONE && j == 0 && c == 0 && !mbar_wait(&sh->q_full[0], n & 1)) return false;
        uint64_t q0 = q_item + (uint64_t)((c * TILE_BYTES) >> 4);
        int sq = -1;
        if (NCT == 0 && c >= KEPT) {
          sq = s_at;
          if (!mbar_wait(&sh->full[sq], s_ph)) return false;
          next_stage();
          q0 = rq_desc + (uint64_t)((sq * TILE_BYTES) >> 4);
        }
        const int s = s_at;
        if (!mbar_wait(&sh->full[s], s_ph)) return false;
        next_stage();
        TC_FENCE_AFTER();
        const uint64_t k0 = k_desc + (uint64_t)((s * TILE_BYTES) >> 4);
        const uint64_t q1 = q0 + (HALF_BYTES >> 4), k1 = k0 + (GROUP_BYTES / 2 >> 4);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) umma(tmem_s, q0 + 2 * kk, k0 + 2 * kk, IDESC_QK, (cc | kk) != 0);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) umma(tmem_s, q1 + 2 * kk, k1 + 2 * kk, IDESC_QK, 1);
        if (sq >= 0) umma_commit(&sh->empty[sq]);
        umma_commit(&sh->empty[s]);
      }
      if (ONE && j == n_tiles - 1) umma_commit(&sh->q_free[1]);     // the other pieces have been used for the last time
      umma_commit(&sh->s_full[gt & 1]);
      return true;
    };
    auto issue_qk = [&](int n, int j, int n_tiles, int gt) -> bool {
      bool fine = true;
      if (lane == 0) fine = issue_qk_lane(n, j, n_tiles, gt);
      s_at = __shfl_sync(0xffffffffu, s_at, 0);
      s_ph = __shfl_sync(0xffffffffu, s_ph, 0);
      return __all_sync(0xffffffffu, fine);
    };
    bool ok = true;
    int r = 0, n = 0, gt = 0;
    Item it, nx;
    bool have = next_item(r, it);
    if (have) ok = issue_qk(0, 0, it.n_tiles, 0);
    while (have && ok) {
      int rn = r + 1;
      const bool more = next_item(rn, nx);
      for (int j = 0; j < it.n_tiles && ok; ++j, ++gt) {
        const bool last = j + 1 == it.n_tiles, has_next = !last || more;
        // the next scores while this tile's softmax runs; with one place for queries the next item's have to wait until
        // this item's output has left
        auto next_scores = [&]() -> bool {
          return last ? issue_qk(n + 1, 0, nx.n_tiles, gt + 1) : issue_qk(n, j + 1, it.n_tiles, gt + 1);
        };
        const bool later = ONE && last;
        if (has_next && !later) ok = next_scores();
        if (!ok) break;
        const int s = s_at;
        if (!wait(&sh->full[s], s_ph)) { ok = false; break; }
        next_stage();
        const int first = it.j_hi - it.tile(j) * BN;
        if (first < BN) {
          // the keys end within the tile: the value rows past the end become zero (they may hold anything, and their weights
          // are zero)
          for (int i = lane; i < (BN - first) * 16; i += 32) {
            const int key_row = first + i / 16, part = i % 16;    // 16 chunks of 16 bytes per row (both halves)
            *reinterpret_cast<uint4*>(r_s + s * TILE_BYTES + (key_row >> 3) * GROUP_BYTES + (part >> 3) * (GROUP_BYTES / 2) +
                                      (key_row & 7) * 128 + (part & 7) * 16) = make_uint4(0, 0, 0, 0);
          }
          PROXY_FENCE();                                          // visible to the tensor core
          __syncwarp();
        }
        if (!wait(&sh->p_full[gt & 1], (gt >> 1) & 1)) { ok = false; break; }
        // an item's first product overwrites the output of the item before it, which its softmax threads must have read
        if (j == 0 && n > 0 && !wait(&sh->o_free, (n - 1) & 1)) { ok = false; break; }
        if (lane == 0) {
          TC_FENCE_AFTER();
          // O += P V : 8 steps of 16 keys; P from tensor memory (8 columns a step), two 8-row groups down V
          const uint32_t tmem_p = tmem + TMEM_P + (gt & 1) * 64;
          const uint64_t v0 = v_desc + (uint64_t)((s * TILE_BYTES) >> 4);
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            umma_a_tmem(tmem_o, tmem_p + kk * 8, v0 + kk * (2 * GROUP_BYTES / 16), IDESC_PV, (j | kk) != 0);
          umma_commit(&sh->empty[s]);
          umma_commit(&sh->o_done[gt & 1]);
        }
        __syncwarp();
        if (has_next && later) ok = next_scores();
      }
      it = nx;
      r = rn;
      have = more;
      ++n;
    }
    if (!ok && lane == 0) { atomicOr(p.status, JV_STATUS_WAIT_EXPIRED); sh->failed = 1; }
  } else {
    // ----------------------------------------------------------------- softmax
    // Two threads per row: warps 2..5 take the first 64 keys of a tile (and the first 64 columns of O), warps 6..9 the
    // other 64.  A warp reads the 32 TMEM lanes of its number modulo 4.
    const int quad = warp & 3;
    const int half = (warp - 2) >> 2;
    const int row = quad * 32 + lane;                           // this thread's row of the tile
    const int t = row / HPT, hh = row % HPT;
    const uint32_t lane_addr = (uint32_t)(quad * 32) << 16;
    const float sc = p.scale_log2;
    constexpr float LAZY = 8.f;
    bool ok = true;
    int gt = 0, n = 0, r_next = 0;
    Item upcoming;
    bool more = next_item(r_next, upcoming);
    while (more) {
      const Item it = upcoming;
      ++r_next;
      more = next_item(r_next, upcoming);       // asked for while the current item runs
      const bool row_ok = t < it.tokens_here && hh < HPT;
      const int pos = row_ok ? it.pos_first + t : -1;
      const int head = it.kv_head * HPT + hh;
      // m_ref is the reference maximum that the exponentials are taken against.  It follows the true maximum lazily: only
      // when the maximum has grown by more than 2^8 (in the exponent) is O rescaled.
      float m_ref = -INFINITY, l_run = 0.f;
      // A wait that runs out makes `ok` false for the whole warp; the loops then only keep their appointments at the named
      // barriers (so that nobody is left waiting there) and do no further work.
      for (int j = 0; j < it.n_tiles; ++j, ++gt) {
        if (ok) ok = mbar_wait(&sh->s_full[gt & 1], (gt >> 1) & 1);
        ok = __all_sync(0xffffffffu, ok);
        const uint32_t s_addr = tmem + lane_addr + (gt & 1) * 128 + half * 64;
        const int jt = it.tile(j);
        const int key0 = jt * BN + half * 64;                    // first key of this thread's 64
        const bool need_mask = jt * BN + BN > it.j_hi || jt * BN + BN - 1 > it.pos_first;   // block-uniform
        uint32_t sr[2][32];
        float my_max = -INFINITY;
        if (ok) {
          TC_FENCE_AFTER();
          tmem_ld32_issue(s_addr, sr[0]);
          tmem_ld32_issue(s_addr + 32, sr[1]);
          tmem_ld_wait();
          if (need_mask) {
            const int last = min(pos, it.j_hi - 1) - key0;       // the last of this thread's 64 keys that counts
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
              for (int i = 0; i < 32; ++i)
                if (c * 32 + i > last) sr[c][i] = __float_as_uint(-INFINITY);
          }
          float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
          for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 32; i += 2)
              mx[(i >> 1) & 3] = max3(mx[(i >> 1) & 3], __uint_as_float(sr[c][i]), __uint_as_float(sr[c][i + 1]));
          my_max = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
        }
        // the reference moves only if some score of the tile has outgrown it; only then do a row's two threads exchange maxima
        const bool outgrown = ok && my_max != -INFINITY && (m_ref == -INFINITY || (my_max - m_ref) * sc > LAZY);
        float alpha = 1.f;
        if (pair_barrier_or(quad, outgrown)) {
          sh->xch[half][row] = my_max;
          pair_barrier(quad);
          const float m_tile = fmaxf(sh->xch[0][row], sh->xch[1][row]);
          pair_barrier(quad);                                    // both have read before a later tile writes
          if (ok && m_tile != -INFINITY && (m_ref == -INFINITY || (m_tile - m_ref) * sc > LAZY)) {
            alpha = (m_ref == -INFINITY) ? 0.f : fast_exp2((m_ref - m_tile) * sc);
            m_ref = m_tile;
          }
        }
        const float m_scaled = (m_ref == -INFINITY) ? 0.f : m_ref * sc;
        // O is rescaled only if some row of this warp moved its reference; the previous P V must be complete then
        if (ok && j > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
          ok = __all_sync(0xffffffffu, mbar_wait(&sh->o_done[(gt - 1) & 1], ((gt - 1) >> 1) & 1));
          if (ok) {
            TC_FENCE_AFTER();
#pragma unroll 1
            for (int c = 0; c < 2; ++c) {
              float v[32];
              tmem_ld32(tmem_o + lane_addr + half * 64 + c * 32, v);
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] *= alpha;
              tmem_st32(tmem_o + lane_addr + half * 64 + c * 32, v);
            }
          }
        }
        if (!ok) continue;
        // weights: pairs of scores in packed 32-bit arithmetic, as bfloat16 pairs into this thread's 32 columns of P
        {
          const uint64_t scale2 = pack2(sc, sc), neg_m2 = pack2(-m_scaled, -m_scaled);
          uint64_t sum2[2] = {pack2(0.f, 0.f), pack2(0.f, 0.f)};
          uint32_t pw[32];
#pragma unroll
          for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const uint64_t x2 = fma2(pack2(__uint_as_float(sr[c][i]), __uint_as_float(sr[c][i + 1])), scale2, neg_m2);
              float x0, x1;
              unpack2(x2, x0, x1);
              const float p0 = fast_exp2(x0), p1 = fast_exp2(x1);
              sum2[(i >> 1) & 1] = add2(sum2[(i >> 1) & 1], pack2(p0, p1));
              const __nv_bfloat162 h2 = __floats2bfloat162_rn(p0, p1);
              pw[c * 16 + (i >> 1)] = *reinterpret_cast<const uint32_t*>(&h2);
            }
          float sum[4];
          unpack2(sum2[0], sum[0], sum[1]);
          unpack2(sum2[1], sum[2], sum[3]);
          tmem_st32_bits(tmem + lane_addr + TMEM_P + (gt & 1) * 64 + half * 32, pw);
          l_run = l_run * alpha + ((sum[0] + sum[1]) + (sum[2] + sum[3]));
        }
        TC_FENCE_BEFORE();                                       // P is in tensor memory before the arrival
        mbar_arrive(&sh->p_full[gt & 1]);
      }
      // ---- the item's output: O / sum, each thread its 64 columns; the row's sum is the two threads' together
      const int g_last = gt - 1, qb = n % QB;
      sh->xch[half][row] = l_run;
      pair_barrier(quad);
      const float l_row = sh->xch[0][row] + sh->xch[1][row];
      pair_barrier(quad);                                        // both have read before the next item's first tile writes
      const bool got = ok && mbar_wait(&sh->o_done[g_last & 1], (g_last >> 1) & 1);
      float inv = row_ok ? 1.f / l_row : 0.f;
      if (p.sink != nullptr && row_ok && m_ref != -INFINITY) {
        // the sink joins the denominator: the row's sum stands against the reference m_ref * sc (an exponent of two)
        const float sk = p.sink[head] * LOG2E, mr = m_ref * sc, mx = fmaxf(mr, sk);
        const float e = fast_exp2(mr - mx);
        inv = e / (l_row * e + fast_exp2(sk - mx));
      }
      inv *= p.out_scale;
      // A whole tile leaves through shared memory (where the item's piece 0 was: every product with it has completed) and
      // one TMA store per half of the head.
      const bool whole = it.tokens_here == p.tokens_per_tile;
      unsigned char* out_s = q_s + qb * KEPT * TILE_BYTES;
      unsigned char* row_base = out_s + half * HALF_BYTES + row * 128;
      __nv_bfloat16* dst = p.out + (size_t)(it.q_first + t) * p.out_stride + (size_t)head * D + half * 64;
      if (got) {
        TC_FENCE_AFTER();
#pragma unroll 1
        for (int c = 0; c < 2; ++c) {
          float v[32];
          tmem_ld32(tmem_o + lane_addr + half * 64 + c * 32, v);
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            uint4 pk;
            __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&pk);
#pragma unroll
            for (int e = 0; e < 4; ++e) h2[e] = __floats2bfloat162_rn(v[q * 8 + 2 * e] * inv, v[q * 8 + 2 * e + 1] * inv);
            const int chunk = c * 4 + q;                         // 16-byte chunk within the 128-byte row
            if (whole) *reinterpret_cast<uint4*>(row_base + ((chunk ^ (row & 7)) << 4)) = pk;
            else if (row_ok) *reinterpret_cast<uint4*>(dst + c * 32 + q * 8) = pk;
          }
        }
        TC_FENCE_BEFORE();
        mbar_arrive(&sh->o_free);                                // this thread has read its part of the output
      }
      if (whole) {
        PROXY_FENCE();
        asm volatile("bar.sync 5, 256;\n" ::: "memory");
      }
      if (threadIdx.x == 64) {
        if (whole && got) {
          tma_store_3d(&out_map, out_s, 0, it.kv_head * HPT, it.q_first);
          tma_store_3d(&out_map, out_s + HALF_BYTES, 64, it.kv_head * HPT, it.q_first);
          asm volatile("cp.async.bulk.commit_group;\n" ::: "memory");
          asm volatile("cp.async.bulk.wait_group.read 0;\n" ::: "memory");
        }
        mbar_arrive(&sh->q_free[qb]);                            // the place may take the queries of another item
      }
      if (!got) ok = false;
      ++n;
    }
    if (!ok && lane == 0) { atomicOr(p.status, JV_STATUS_WAIT_EXPIRED); sh->failed = 1; }
  }

  TC_FENCE_BEFORE();
  __syncthreads();
  if (sh->failed) {
    // a wait ran out: products already issued may still write tensor memory and copies already asked for still land in this
    // block's shared memory; both get a bounded time to finish before tensor memory is freed and the block ends
    if (warp == 1 && lane == 0) drain_products_after_failure(&sh->drain);
    if (warp == 0 && lane == 0) {
      for (int b = 0; b < 2; ++b)
        if (sh->armed_q[b] >= 0) drain_copies_after_failure(&sh->q_full[b], sh->armed_q[b]);
      for (int s = 0; s < STAGES; ++s)
        if (sh->armed[s] >= 0) drain_copies_after_failure(&sh->full[s], sh->armed[s]);
    }
    __syncthreads();
  }
  if (warp == 1) {
    TC_FENCE_AFTER();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(TMEM_COLS) : "memory");
  }
}

template <int NCT>
int launch(int blocks, cudaStream_t stream, const CUtensorMap& q_map, const CUtensorMap& k_map, const CUtensorMap& v_map,
           const CUtensorMap& out_map, const Params& p) {
  constexpr size_t smem = TILE_BYTES * SMEM_TILES + sizeof(Shared) + 1024;
  static_assert(smem <= 227 * 1024, "shared memory");
  static bool ready[JV_MAX_DEVICES];
  if (!jv_once_per_device(ready, [&] {
        return cudaFuncSetAttribute(attn_rows_tcgen05_kernel<NCT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) == cudaSuccess;
      }))
    return JV_ERR_UNSUPPORTED;
  return jv_launch(attn_rows_tcgen05_kernel<NCT>, dim3(blocks), dim3(THREADS), smem, stream, q_map, k_map, v_map, out_map, p);
}
}  // namespace

// q: [n_tokens, q_stride] bfloat16, head h of a token at column h * n_kv_heads * 128; out: [n_tokens, out_stride], head h at
// h * 128; k_cache/v_cache: [num_pages, page_size, n_kv_heads, 128]; work: [n_work, 2] (entry, first token of the tile), tiles
// of 128 / (n_q_heads / n_kv_heads) tokens, in ascending order of work; sink: [n_q_heads] floats or null.
JV_EXPORT int jv_attn_rows_tcgen05(const void* q, int q_stride, int n_tokens, void* out, int out_stride, const void* k_cache,
                                   const void* v_cache, const int* block_table, int table_width, const int* cu_seqlens,
                                   const int* start_pos, const int* work, int n_work, int n_q_heads, int n_kv_heads,
                                   int page_size, int num_pages, float scale, float out_scale, const float* sink, int* status,
                                   cudaStream_t stream) {
  if (n_work == 0) return JV_OK;
  if (n_kv_heads < 2 || n_q_heads % n_kv_heads || n_q_heads / n_kv_heads > 16 || page_size < 8 || page_size > 128 ||
      (page_size & (page_size - 1)))
    return JV_ERR_UNSUPPORTED;
  if ((q_stride % 8) || (out_stride % 8) || ((uintptr_t)q % 16) || ((uintptr_t)out % 16) || ((uintptr_t)k_cache % 16) ||
      ((uintptr_t)v_cache % 16))
    return JV_ERR_UNSUPPORTED;
  auto fn = encode_fn();
  if (fn == nullptr) return JV_ERR_UNSUPPORTED;
  const int HPT = n_q_heads / n_kv_heads;
  CUtensorMap q_map, k_map, v_map, out_map;
  for (int which = 0; which < 2; ++which) {
    // queries and output: (d, head, token); a box is 64 d x HPT heads x (128 / HPT) tokens = 128 rows, head fastest
    const int d = which ? D : D * n_kv_heads;
    const cuuint64_t dims[3] = {(cuuint64_t)d, (cuuint64_t)n_q_heads, (cuuint64_t)n_tokens};
    const cuuint64_t strides[2] = {(cuuint64_t)d * 2, (cuuint64_t)(which ? out_stride : q_stride) * 2};
    const cuuint32_t box[3] = {64, (cuuint32_t)HPT, (cuuint32_t)(ROWS / HPT)};
    const cuuint32_t es[3] = {1, 1, 1};
    if (fn(which ? &out_map : &q_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, which ? out : const_cast<void*>(q), dims, strides, box, es,
           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
      return JV_ERR_UNSUPPORTED;
  }
  for (int which = 0; which < 2; ++which) {
    // cache: (d within a half, slot within a group of 8, half of a head, group, page); a box is a page's rows of one head
    const cuuint64_t pitch = (cuuint64_t)n_kv_heads * D * 2;
    const cuuint64_t dims[5] = {64, 8, (cuuint64_t)n_kv_heads * 2, (cuuint64_t)page_size / 8, (cuuint64_t)num_pages};
    const cuuint64_t strides[4] = {pitch, 128, 8 * pitch, page_size * pitch};
    const cuuint32_t box[5] = {64, 8, 2, (cuuint32_t)page_size / 8, 1};
    const cuuint32_t es[5] = {1, 1, 1, 1, 1};
    if (fn(which ? &v_map : &k_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 5, const_cast<void*>(which ? v_cache : k_cache), dims,
           strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
      return JV_ERR_UNSUPPORTED;
  }
  Params p;
  p.out = (__nv_bfloat16*)out; p.out_stride = out_stride; p.block_table = block_table; p.table_width = table_width;
  p.cu_seqlens = cu_seqlens; p.start_pos = start_pos; p.work = work; p.n_work = n_work; p.n_q_heads = n_q_heads;
  p.n_kv_heads = n_kv_heads; p.page_size = page_size; p.num_pages = num_pages; p.hpt = HPT; p.tokens_per_tile = ROWS / HPT;
  p.scale_log2 = scale * LOG2E; p.out_scale = out_scale; p.sink = sink; p.status = status;
  // persistent blocks: one per multiprocessor (or per item, if there are fewer)
  static int sm_count[JV_MAX_DEVICES];
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= JV_MAX_DEVICES) return JV_ERR_UNSUPPORTED;
  if (sm_count[dev] == 0 &&
      (cudaDeviceGetAttribute(&sm_count[dev], cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sm_count[dev] <= 0))
    sm_count[dev] = 148;
  const long long items = (long long)n_work * n_kv_heads;
  const int blocks = items < sm_count[dev] ? (int)items : sm_count[dev];
  switch (n_kv_heads) {
    case 2: return launch<2>(blocks, stream, q_map, k_map, v_map, out_map, p);
    case 3: return launch<3>(blocks, stream, q_map, k_map, v_map, out_map, p);
    case 4: return launch<4>(blocks, stream, q_map, k_map, v_map, out_map, p);
    default: return launch<0>(blocks, stream, q_map, k_map, v_map, out_map, p);
  }
}
