// Attention of single tokens whose scores are products with a token's WHOLE cached key row (KD elements, the key heads
// side by side: scores mixed across heads, see talk_prepare.cu), bfloat16, the value heads as in grouped-query attention
// (query head h reads value head h / (H / G)).
//
// Every query head reads every byte of the keys, so a block takes ALL heads of one request over a range of keys (grid:
// request x range) and each cached byte is read once from memory.  Tiles of KT keys come in by bulk copies (one a key row,
// one a value row) into two stages, the next tile's under way while this one is worked on; two blocks share a
// multiprocessor where their stages allow it:
//   scores     S [H, KT] = Q [H, KD] K^T on the tensor cores (mma.sync m16n8k16, 32-bit accumulation): a warp takes 16 heads
//              and a part of KD, keeps its piece of the queries in registers for the whole range, and goes over the keys of
//              the tile; the parts of a score are added up by its reader
//   softmax    running (max, sum) a head in 32-bit, eight lanes a head
//   output     O [H, DV] += P V on the tensor cores, a warp 16 columns of a value head at a time for all query heads that
//              read it (rows of the tile without a head are zero); P is rounded to bfloat16 as in the prompt kernels
// Each range leaves its unnormalised output and (max, sum); a second kernel merges a head's ranges in ascending order and
// lets the sink join the denominator.  Every wait on a barrier is bounded and reports to the status word.
#include "common.cuh"
#include "mbarrier.cuh"
#include <math.h>

namespace {
constexpr int THREADS = 256, WARPS = THREADS / 32;
constexpr int MAX_SPLIT = 256;                  // keys of a range
constexpr int MAX_HEADS = 128;
constexpr float LOG2E = 1.4426950408889634f;

struct Params {
  const __nv_bfloat16* q; int q_stride;
  __nv_bfloat16* out; int out_stride;
  float* part_o; float* part_ml;
  const __nv_bfloat16* k_cache; const __nv_bfloat16* v_cache;
  const int* block_table; int table_width;
  const int* cu_seqlens; const int* start_pos; const int* work;
  int H, G, KD, DV, page_size, num_pages;
  float scale_log2, out_scale;
  const float* sink;           // [H] or null
  int KT;                      // keys of a tile
  int split_size, n_splits;
  int* status;
};

__device__ __forceinline__ void bulk_copy(void* dst, const void* src, int bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t (&r)[2], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

template <int N> struct Int { static constexpr int value = N; };

// Offsets (bytes) of the arrays in dynamic shared memory, for the kernel and its launcher.
struct Layout {
  int k_row, v_row, s_row, p_row;              // elements from row to row
  size_t k, v, s, w, total;                    // s: [k_parts][H16][s_row] floats; w: [H16][p_row] bfloat16
  __host__ __device__ Layout(int H, int G, int KD, int DV, int KT, int k_parts) {
    const int H16 = (H + 15) / 16 * 16;
    k_row = KD + 8; v_row = G * DV + 8; s_row = KT + 4; p_row = KT + 8;
    k = 0;
    v = k + sizeof(__nv_bfloat16) * (size_t)2 * KT * k_row;
    s = v + sizeof(__nv_bfloat16) * (size_t)2 * KT * v_row;
    w = s + sizeof(float) * (size_t)k_parts * H16 * s_row;
    total = w + sizeof(__nv_bfloat16) * (size_t)H16 * p_row;
  }
};

// NP: pieces of 16 output columns a warp keeps; KP: parts of KD that warps share the scores of 16 heads in; KS: steps of 16
// elements of KD a warp keeps of the queries.
template <int NP, int KP, int KS>
__global__ void __launch_bounds__(THREADS, NP * 8 + KS * 4 <= 64 ? 2 : 1) attn_rows_decode_kernel(const Params p) {
  extern __shared__ __align__(128) unsigned char smem[];
  __shared__ long long slots[MAX_SPLIT];        // cache slot of every key of the range (-1: none)
  __shared__ float row_m[MAX_HEADS], row_l[MAX_HEADS], row_alpha[MAX_HEADS];
  __shared__ __align__(8) uint64_t bars[2];
  const int H = p.H, G = p.G, KD = p.KD, DV = p.DV, KT = p.KT, HPT = H / G;
  const Layout L(H, G, KD, DV, KT, KP);
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(smem + L.k);
  __nv_bfloat16* vs = reinterpret_cast<__nv_bfloat16*>(smem + L.v);
  float* ss = reinterpret_cast<float*>(smem + L.s);
  __nv_bfloat16* ps = reinterpret_cast<__nv_bfloat16*>(smem + L.w);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_trigger();
  if (tid == 0) {
    mbar_init(&bars[0], WARPS);
    mbar_init(&bars[1], WARPS);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  pdl_wait();
  const int entry = p.work[2 * blockIdx.x];
  const int pos = p.start_pos[entry];
  const int j_lo = blockIdx.y * p.split_size, j_hi = min(pos + 1, j_lo + p.split_size);
  if (blockIdx.y == 0 && tid == 0 && pos / p.split_size >= p.n_splits) atomicOr(p.status, JV_STATUS_BAD_ROW);
  if (j_lo >= j_hi) return;
  const int token = p.cu_seqlens[entry];
  for (int i = tid; i < j_hi - j_lo; i += THREADS) {
    const int j = j_lo + i, pi = j / p.page_size;
    const int page = pi < p.table_width ? p.block_table[(size_t)entry * p.table_width + pi] : -1;
    long long s = -1;
    if (page < 0 || page >= p.num_pages) atomicOr(p.status, JV_STATUS_BAD_PAGE);
    else s = (long long)page * p.page_size + (j - pi * p.page_size);
    slots[i] = s;
  }
  for (int h = tid; h < MAX_HEADS; h += THREADS) { row_m[h] = -INFINITY; row_l[h] = 0.f; }
  __syncthreads();

  const int n_tiles = (j_hi - j_lo + KT - 1) / KT;
  // Tile t into stage t & 1: a key row and a value row a copy, every warp its share of the rows (issuing a copy takes some
  // sixty clocks).  Rows past the last key are not copied: their scores are masked, and their value rows become zero (they
  // may hold anything, and their weights are zero).
  auto issue = [&](int t) {
    uint64_t* bar = &bars[t & 1];
    const int here = min(KT, j_hi - j_lo - t * KT), k_bytes = KD * 2, v_bytes = G * DV * 2;
    const int n = warp + WARPS * (lane >> 1), at = (t & 1) * KT + n;       // two lanes a row: keys, values
    const bool is_v = lane & 1;
    const long long slot = n < here ? slots[t * KT + n] : -1;
    const int n_k = __popc(__ballot_sync(0xffffffffu, slot >= 0 && !is_v));
    if (lane == 0) mbar_expect_tx(bar, n_k * (k_bytes + v_bytes));
    __syncwarp();                                // the announcement before the copies
    if (slot >= 0) {
      if (is_v) bulk_copy(vs + (size_t)at * L.v_row, p.v_cache + slot * (G * DV), v_bytes, bar);
      else bulk_copy(ks + (size_t)at * L.k_row, p.k_cache + slot * KD, k_bytes, bar);
    } else if (is_v && n < KT) {
      for (int c = 0; c < G * DV / 8; ++c) *reinterpret_cast<uint4*>(vs + (size_t)at * L.v_row + c * 8) = make_uint4(0, 0, 0, 0);
    }
  };
  issue(0);
  if (n_tiles > 1) issue(1);

  // ---- this warp's queries: 16 heads, k steps [k0, k1) of 16 elements, as operand fragments
  const int H16 = (H + 15) / 16 * 16, mt = H16 / 16, k_steps = KD / 16;
  const int m16 = warp % mt, part = warp / mt;
  const bool scores_here = part < KP;
  const int k0 = k_steps * part / KP, k1 = scores_here ? k_steps * (part + 1) / KP : k0;
  uint32_t qa[KS][4];
  {
    const int h0 = m16 * 16 + (lane >> 2), h1 = h0 + 8;
    const __nv_bfloat16* q0 = p.q + (size_t)token * p.q_stride + (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < KS; ++i) {
      const int k = (k0 + i) * 16;
      const bool in = k0 + i < k1;
      qa[i][0] = in && h0 < H ? *reinterpret_cast<const uint32_t*>(q0 + (size_t)h0 * KD + k) : 0u;
      qa[i][1] = in && h1 < H ? *reinterpret_cast<const uint32_t*>(q0 + (size_t)h1 * KD + k) : 0u;
      qa[i][2] = in && h0 < H ? *reinterpret_cast<const uint32_t*>(q0 + (size_t)h0 * KD + k + 8) : 0u;
      qa[i][3] = in && h1 < H ? *reinterpret_cast<const uint32_t*>(q0 + (size_t)h1 * KD + k + 8) : 0u;
    }
  }

  // ---- this warp's columns of the output: pieces warp * NP .. of 16 columns, for up to 16 query heads of a value head
  const int pieces = G * DV / 16, first_piece = warp * NP;
  float acc[NP][2][4];
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][0][e] = acc[i][1][e] = 0.f;
  const int g0 = lane >> 2, g1 = g0 + 8;         // this lane's two rows: query heads of the value head
  const bool in0 = g0 < HPT, in1 = g1 < HPT;
  int head0[NP];                                 // the first query head of a piece's value head (-1: no such piece)
#pragma unroll
  for (int i = 0; i < NP; ++i) head0[i] = first_piece + i < pieces ? (first_piece + i) * 16 / DV * HPT : -1;

  for (int t = 0; t < n_tiles; ++t) {
    const int buf = t & 1;
    // every thread takes the same way out: all saw the tile, or the block stops (status word set)
    if (!__syncthreads_and(mbar_wait(&bars[buf], (t >> 1) & 1))) {
      if (tid == 0) atomicOr(p.status, JV_STATUS_WAIT_EXPIRED);
      mbar_wait(&bars[buf], (t >> 1) & 1);       // once more, bounded, for copies that may still be landing
      if (t + 1 < n_tiles) mbar_wait(&bars[buf ^ 1], ((t + 1) >> 1) & 1);
      return;
    }
    // ---- scores: 8 keys at a time
    if (scores_here) {
      const __nv_bfloat16* kb = ks + (size_t)(buf * KT + (lane & 7)) * L.k_row + k0 * 16 + (lane >> 3) * 8;
      float* dst = ss + ((size_t)part * H16 + m16 * 16 + (lane >> 2)) * L.s_row + (lane & 3) * 2;
      const int n_here = k1 - k0;
      for (int n8 = 0; n8 < KT / 8; ++n8, kb += 8 * L.k_row, dst += 8) {
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < KS; i += 2) {          // two independent sums
          if (i + 1 < n_here) {
            uint32_t b[4];
            ldmatrix_x4(b, kb + i * 16);
            mma_bf16(c0, qa[i], b[0], b[1]);
            mma_bf16(c1, qa[i + 1], b[2], b[3]);
          } else if (i < n_here) {                 // one step is left: the upper lanes' addresses are not used
            uint32_t b[2];
            ldmatrix_x2(b, kb + i * 16 - ((lane & 16) ? 16 : 0));
            mma_bf16(c0, qa[i], b[0], b[1]);
          }
        }
        *reinterpret_cast<float2*>(dst) = make_float2(c0[0] + c1[0], c0[1] + c1[1]);
        *reinterpret_cast<float2*>(dst + 8 * L.s_row) = make_float2(c0[2] + c1[2], c0[3] + c1[3]);
      }
    }
    __syncthreads();
    // ---- softmax: eight lanes a head
    const int here = min(KT, j_hi - j_lo - t * KT);
    for (int h = tid >> 3; h < H16; h += THREADS / 8) {        // whole warps stay together: H16 is a multiple of 4
      const float* row = ss + (size_t)h * L.s_row + (lane & 7);
      __nv_bfloat16* wrow = ps + (size_t)h * L.p_row + (lane & 7);
      auto softmax = [&](auto columns) {
        constexpr int C = decltype(columns)::value;            // keys of a lane
        float v[C];
        float mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < C; ++i) {
          float x[KP];
#pragma unroll
          for (int q = 0; q < KP; ++q) x[q] = row[(size_t)q * H16 * L.s_row + 8 * i];
#pragma unroll
          for (int q = 1; q < KP; ++q) x[0] += x[q];
          v[i] = (lane & 7) + 8 * i < here ? x[0] * p.scale_log2 : -INFINITY;
          mx = fmaxf(mx, v[i]);
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_old = row_m[h], m_new = fmaxf(m_old, mx);        // finite: a tile has at least one key
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < C; ++i) {
          const float e = fast_exp2(v[i] - m_new);
          wrow[8 * i] = __float2bfloat16_rn(e);
          sum += e;
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if ((lane & 7) == 0) {
          const float alpha = fast_exp2(m_old - m_new);                // of -inf: 0
          row_alpha[h] = alpha;
          row_m[h] = m_new;
          row_l[h] = row_l[h] * alpha + sum;
        }
        __syncwarp();
      };
      if (KT == 16) softmax(Int<2>{});
      else if (KT == 32) softmax(Int<4>{});
      else softmax(Int<8>{});
    }
    __syncthreads();
    // ---- output
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      if (head0[i] >= 0) {
        const int h0 = head0[i] + g0, h1 = head0[i] + g1;
        const float al0 = in0 ? row_alpha[h0] : 1.f, al1 = in1 ? row_alpha[h1] : 1.f;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          acc[i][e][0] *= al0; acc[i][e][1] *= al0;
          acc[i][e][2] *= al1; acc[i][e][3] *= al1;
        }
        const __nv_bfloat16* w0 = ps + h0 * L.p_row + (lane & 3) * 2;
        const __nv_bfloat16* w1 = ps + h1 * L.p_row + (lane & 3) * 2;
        const __nv_bfloat16* vb = vs + (buf * KT + ((lane >> 3) & 1) * 8 + (lane & 7)) * L.v_row + (first_piece + i) * 16 + (lane >> 4) * 8;
        for (int k = 0; k < KT; k += 16, vb += 16 * L.v_row) {
          uint32_t a[4], b[4];
          a[0] = in0 ? *reinterpret_cast<const uint32_t*>(w0 + k) : 0u;
          a[1] = in1 ? *reinterpret_cast<const uint32_t*>(w1 + k) : 0u;
          a[2] = in0 ? *reinterpret_cast<const uint32_t*>(w0 + k + 8) : 0u;
          a[3] = in1 ? *reinterpret_cast<const uint32_t*>(w1 + k + 8) : 0u;
          ldmatrix_x4_trans(b, vb);
          mma_bf16(acc[i][0], a, b[0], b[1]);
          mma_bf16(acc[i][1], a, b[2], b[3]);
        }
      }
    }
    __syncthreads();                             // the stage and the weights have been read
    if (t + 2 < n_tiles) {
      asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
      issue(t + 2);
    }
  }
  // ---- what the range leaves
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int piece = first_piece + i;
    if (piece < pieces) {
      const int c = piece * 16 / DV, d = piece * 16 - c * DV + (lane & 3) * 2;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int g = half ? g1 : g0;
        if (g < HPT) {
          float* o = p.part_o + (((size_t)blockIdx.x * H + c * HPT + g) * p.n_splits + blockIdx.y) * DV + d;
          *reinterpret_cast<float2*>(o) = make_float2(acc[i][0][2 * half], acc[i][0][2 * half + 1]);
          *reinterpret_cast<float2*>(o + 8) = make_float2(acc[i][1][2 * half], acc[i][1][2 * half + 1]);
        }
      }
    }
  }
  for (int h = tid; h < H; h += THREADS) {
    const size_t at = ((size_t)blockIdx.x * H + h) * p.n_splits + blockIdx.y;
    p.part_ml[2 * at] = row_m[h];
    p.part_ml[2 * at + 1] = row_l[h];
  }
}

// One block a (request, head): the ranges in ascending order; maxima are exponents of two.
__global__ void __launch_bounds__(128) attn_rows_merge_kernel(const Params p) {
  __shared__ float weight[128];
  pdl_trigger();
  pdl_wait();
  const int entry = p.work[2 * blockIdx.x], h = blockIdx.y, lane = threadIdx.x & 31;
  const int n = min(p.start_pos[entry] / p.split_size, p.n_splits - 1) + 1;
  const size_t base = ((size_t)blockIdx.x * p.H + h) * p.n_splits;
  const float2* ml = reinterpret_cast<const float2*>(p.part_ml) + base;
  // the sink is one more part, with no value: maximum sink, sum 1; every warp forms the maximum and the sum for itself
  const float sk = p.sink != nullptr ? p.sink[h] * LOG2E : -INFINITY;
  float m = sk;
  for (int s = lane; s < n; s += 32) m = fmaxf(m, ml[s].x);
  m = warp_max(m);
  float l = 0.f;
  for (int s = lane; s < n; s += 32) l += exp2f(ml[s].x - m) * ml[s].y;
  l = warp_sum(l) + (p.sink != nullptr ? exp2f(sk - m) : 0.f);
  const float inv = p.out_scale / l;
  const size_t out_at = (size_t)p.cu_seqlens[entry] * p.out_stride + (size_t)h * p.DV;
  for (int d0 = 0; d0 < p.DV; d0 += 128) {
    const int d = d0 + threadIdx.x;
    float o = 0.f;
    for (int s0 = 0; s0 < n; s0 += 128) {
      __syncthreads();
      if (s0 + (int)threadIdx.x < n) weight[threadIdx.x] = exp2f(ml[s0 + threadIdx.x].x - m);
      __syncthreads();
      const int upto = min(128, n - s0);
      if (d < p.DV) {
        const float* src = p.part_o + (base + s0) * p.DV + d;
#pragma unroll 8
        for (int s = 0; s < upto; ++s) o = fmaf(weight[s], src[(size_t)s * p.DV], o);
      }
    }
    if (d < p.DV) p.out[out_at + d] = __float2bfloat16_rn(o * inv);
  }
}

// Parts of KD that the warps of 16 heads share.
int parts_of(int H) {
  const int mt = (H + 15) / 16;
  return mt <= 1 ? 8 : mt <= 2 ? 4 : mt <= 4 ? 2 : 1;
}

// Keys of a tile: as many as let two blocks share a multiprocessor, 64 at most and 16 at least (then one block may need
// most of the shared memory).
int tile_keys(int H, int G, int KD, int DV) {
  for (int kt = 64; kt >= 16; kt /= 2)
    if (Layout(H, G, KD, DV, kt, parts_of(H)).total <= (kt > 16 ? 104 : 200) * 1024) return kt;
  return 0;
}

template <int NP, int KP, int KS>
int launch(const Params& p, int n_work, size_t smem, cudaStream_t stream) {
  auto kern = attn_rows_decode_kernel<NP, KP, KS>;
  static bool ready[JV_MAX_DEVICES];
  if (!jv_once_per_device(ready, [&] {
        return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess;
      }))
    return JV_ERR_UNSUPPORTED;
  const int rc = jv_launch(kern, dim3(n_work, p.n_splits), dim3(THREADS), smem, stream, p);
  if (rc != JV_OK) return rc;
  return jv_launch(attn_rows_merge_kernel, dim3(n_work, p.H), dim3(128), 0, stream, p);
}

template <int NP>
int launch_parts(const Params& p, int n_work, size_t smem, cudaStream_t stream) {
  const int kp = parts_of(p.H), steps = (p.KD / 16 + kp - 1) / kp;
  if (kp == 8) return launch<NP, 8, 8>(p, n_work, smem, stream);
  if (kp == 4) return steps <= 8 ? launch<NP, 4, 8>(p, n_work, smem, stream) : launch<NP, 4, 16>(p, n_work, smem, stream);
  if (kp == 2) return launch<NP, 2, 16>(p, n_work, smem, stream);
  return launch<NP, 1, 16>(p, n_work, smem, stream);
}
}  // namespace

// 1 if the kernel takes these sizes: KD and DV multiples of 16, up to 16 query heads a value head and 128 in all, and what a
// warp keeps in registers: 16 steps of the queries, 8 pieces of 16 columns of the output.
JV_EXPORT int jv_attn_rows_decode_supports(int H, int G, int KD, int DV) {
  if (G < 1 || H < 1 || H % G || H > MAX_HEADS || KD % 16 || KD < 16 || DV % 16 || DV < 16) return 0;
  const int kp = parts_of(H), steps = (KD / 16 + kp - 1) / kp;
  return H / G <= 16 && G * DV <= 1024 && steps <= (kp == 8 ? 8 : 16) && tile_keys(H, G, KD, DV) > 0;
}

// q: rows of q_stride elements, head h of a token at column h*KD; out: rows of out_stride, head h at h*DV; k_cache:
// [num_pages, page_size, KD], v_cache: [num_pages, page_size, G*DV]; work: [n_work, 2] entries of one token; part_o:
// [n_work * H * n_splits * DV] and part_ml: [n_work * H * n_splits * 2] floats of scratch; split_size: keys of a range, up to
// 256; sink: [H] floats or null.
JV_EXPORT int jv_attn_rows_decode(const void* q, int q_stride, void* out, int out_stride, float* part_o, float* part_ml,
                                  const void* k_cache, const void* v_cache, const int* block_table, int table_width,
                                  const int* cu_seqlens, const int* start_pos, const int* work, int n_work, int H, int G,
                                  int KD, int DV, int page_size, int num_pages, float scale, float out_scale,
                                  const float* sink, int split_size, int n_splits, int* status, cudaStream_t stream) {
  if (n_work == 0) return JV_OK;
  if (!jv_attn_rows_decode_supports(H, G, KD, DV) || split_size < 1 || split_size > MAX_SPLIT || n_splits < 1 ||
      n_splits > 65535 || (q_stride % 8) || ((uintptr_t)q % 16) || ((uintptr_t)k_cache % 16) || ((uintptr_t)v_cache % 16))
    return JV_ERR_UNSUPPORTED;
  Params p;
  p.q = (const __nv_bfloat16*)q; p.q_stride = q_stride; p.out = (__nv_bfloat16*)out; p.out_stride = out_stride;
  p.part_o = part_o; p.part_ml = part_ml; p.k_cache = (const __nv_bfloat16*)k_cache; p.v_cache = (const __nv_bfloat16*)v_cache;
  p.block_table = block_table; p.table_width = table_width; p.cu_seqlens = cu_seqlens; p.start_pos = start_pos; p.work = work;
  p.H = H; p.G = G; p.KD = KD; p.DV = DV; p.page_size = page_size; p.num_pages = num_pages; p.scale_log2 = scale * LOG2E;
  p.out_scale = out_scale; p.sink = sink; p.split_size = split_size; p.n_splits = n_splits; p.status = status;
  p.KT = tile_keys(H, G, KD, DV);
  const size_t smem = Layout(H, G, KD, DV, p.KT, parts_of(H)).total;
  const int np = (G * DV / 16 + WARPS - 1) / WARPS;
  return np <= 2 ? launch_parts<2>(p, n_work, smem, stream) : np <= 4 ? launch_parts<4>(p, n_work, smem, stream)
                                                                      : launch_parts<8>(p, n_work, smem, stream);
}
