// Preparation of queries, keys and values for attention whose heads' scores are mixed before the softmax
// ("talking heads"), fused with the write of the new keys and values into the paged cache.
//
// With H query heads on G key heads (head g reads key head g / (H/G)), raw scores r_g(j) = q_g . k_{g/(H/G)}(j) and
// a matrix T [H, H], the score of head h is
//
//   s_h(j) = sum_g T[h, g] r_g(j) = sum_c ( sum_{g on key head c} T[h, g] q_g ) . k_c(j) = Q_h . K(j)
//
// where K(j) is the token's WHOLE cached key row (its G key heads side by side) and Q_h, of the same size G*D, holds at
// key head c the mixture of the query heads that read c.  So the mixing moves from the scores, one per pair of tokens, to
// the queries, one per token: the attention kernels then run H query heads on ONE key head of G*D elements, with values
// as before.  The mixture is formed in 32-bit from queries that have not been rounded, and rounded once.
//
// Per token: query and key heads are rotated by position * freq[j] over their first rot_dim elements (element j with
// j + rot_dim/2, 32-bit) and divided by their root mean square (`normed`; no weight: a rotation keeps the sum of squares,
// so the order of the two does not matter); Q goes to q_out [n, H * G*D], keys to k_cache[page, slot, G, D], values as
// they are to v_cache[page, slot, G, DV].
//
// One block a token (or, for a few tokens, several blocks a token that share its mixed heads; only the first writes the
// cache).  One warp norms and rotates a head; the queries lie in shared memory as floats, and a thread keeps 4 elements of
// the query heads of one key head in registers and forms its elements of every mixed head from them.
#include "common.cuh"

namespace {
constexpr int THREADS = 256;
constexpr int GROUP_REGS = 8;      // query heads of a key head that a thread keeps in registers (more are read again)

struct TalkParams {
  const void* proj; long long row_stride; int q_off, k_off, v_off;
  void* q_out;
  const float* talk;                 // [H, H]
  const int* positions; const int* token_entry; const int* block_table; int table_width;
  const float* freq; int rot_dim;
  int normed; float eps;
  void* k_cache; void* v_cache;
  int n, n_q_heads, n_kv_heads, key_dim, value_dim, page_size, num_pages;
  int parts;                         // blocks per token
  int* status;
};

template <typename T, int V> struct Pack;
template <> struct Pack<float, 1> {
  static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
};
template <> struct Pack<float, 4> {
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Pack<__nv_bfloat16, 1> {
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct Pack<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    uint2 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
    h[0] = __floats2bfloat162_rn(v[0], v[1]);
    h[1] = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = u;
  }
};

// VEC: elements of a mixed head that a thread forms together (4 where the key size allows it).  HPTC: query heads of a key
// head, 4 or 8 (0: any number).  ND: the key size in 32s where a rotation by whole 32s lets a lane hold both elements of its
// pairs in registers, 2 or 4 (0: any size, pairs through shared memory).
template <typename T, int VEC, int HPTC, int ND>
__global__ void __launch_bounds__(THREADS) talk_prepare_kernel(const TalkParams p) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  const int H = p.n_q_heads, G = p.n_kv_heads, D = p.key_dim, HPT = HPTC > 0 ? HPTC : H / G, half = p.rot_dim >> 1;
  float* ts = smem;                                    // [mixed heads of this block][H]
  const int t = blockIdx.x / p.parts, part = blockIdx.x - t * p.parts;
  const int h_lo = (int)((long long)H * part / p.parts), h_hi = (int)((long long)H * (part + 1) / p.parts);
  float* qs = ts + (((h_hi - h_lo) * H + 3) & ~3);     // [H][D]
  float* ks = qs + (((size_t)H * D + 3) & ~(size_t)3);  // ND == 0: [G][D], then the angles' [half] cosines and sines
  float* cs = ks + (size_t)G * D;
  float* sn = cs + half;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int i = tid; i < (h_hi - h_lo) * H; i += THREADS) ts[i] = p.talk[(size_t)h_lo * H + i];   // a weight: before the wait
  pdl_wait();
  const int posi = p.positions[t];
  const T* row = (const T*)p.proj + (size_t)t * p.row_stride;
  const bool writes = p.k_cache != nullptr && part == 0;
  const int n_heads = H + (writes ? G : 0);
  constexpr int WARPS = THREADS / 32;
  // element e of the token's query and key heads, in the order [query heads][key heads]
  auto source = [&](int h) { return row + (h < H ? p.q_off + h * D : p.k_off + (h - H) * D); };
  T raw[ND > 0 ? ND : 1];
  if (ND > 0 && warp < n_heads) {
#pragma unroll
    for (int i = 0; i < ND; ++i) raw[i] = source(warp)[lane + 32 * i];
  }
  size_t slot = 0;
  bool page_ok = false;
  if (writes) {
    const int pi = posi / p.page_size;
    const int page = (posi >= 0 && pi < p.table_width) ? p.block_table[(size_t)p.token_entry[t] * p.table_width + pi] : -1;
    page_ok = page >= 0 && page < p.num_pages;
    if (page_ok) slot = (size_t)page * p.page_size + (posi - pi * p.page_size);
    else if (tid == 0) atomicOr(p.status, JV_STATUS_BAD_PAGE);
  }
  if (ND > 0) {
    // ---- one warp a head, pairs within a lane: element lane + 32 i turns with lane + 32 (i + half / 32)
    const int hi = half >> 5;
    float c[ND > 0 ? ND : 1], s[ND > 0 ? ND : 1];
#pragma unroll
    for (int i = 0; i < ND / 2; ++i)
      if (i < hi) sincosf((float)posi * p.freq[lane + 32 * i], &s[i], &c[i]);
    for (int h = warp; h < n_heads; h += WARPS) {
      float x[ND > 0 ? ND : 1];
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < ND; ++i) { x[i] = to_f32(raw[i]); ss = fmaf(x[i], x[i], ss); }
      if (h + WARPS < n_heads) {                       // the next head's loads fly while this one is worked on
#pragma unroll
        for (int i = 0; i < ND; ++i) raw[i] = source(h + WARPS)[lane + 32 * i];
      }
      if (p.normed) {
        const float inv = rsqrtf(warp_sum(ss) / (float)D + p.eps);
#pragma unroll
        for (int i = 0; i < ND; ++i) x[i] *= inv;
      }
#pragma unroll
      for (int i = 0; i < ND / 2; ++i)
#pragma unroll
        for (int o = 1; o <= ND / 2; ++o)              // the partner's place, i + hi, as a constant
          if (o == hi && i < hi) {
            const float u = x[i], v = x[i + o];
            x[i] = u * c[i] - v * s[i];
            x[i + o] = v * c[i] + u * s[i];
          }
      if (h < H) {
#pragma unroll
        for (int i = 0; i < ND; ++i) qs[(size_t)h * D + lane + 32 * i] = x[i];
      } else if (page_ok) {
        T* kd = (T*)p.k_cache + (slot * G + (h - H)) * D + lane;
#pragma unroll
        for (int i = 0; i < ND; ++i) kd[32 * i] = from_f32<T>(x[i]);
      }
    }
  } else {
    for (int e = tid; e < n_heads * D; e += THREADS) {
      const int h = e / D;
      (h < H ? qs[e] : ks[e - H * D]) = to_f32(source(h)[e - h * D]);
    }
    for (int j = tid; j < half; j += THREADS) sincosf((float)posi * p.freq[j], &sn[j], &cs[j]);
    __syncthreads();
    for (int h = warp; h < n_heads; h += WARPS) {
      float* x = h < H ? qs + (size_t)h * D : ks + (size_t)(h - H) * D;
      float inv = 1.f;
      if (p.normed) {
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) ss = fmaf(x[d], x[d], ss);
        inv = rsqrtf(warp_sum(ss) / (float)D + p.eps);
      }
      T* kd = (h >= H && page_ok) ? (T*)p.k_cache + (slot * G + (h - H)) * D : nullptr;
      for (int j = lane; j < half; j += 32) {
        const float u = x[j] * inv, v = x[j + half] * inv;
        const float a = u * cs[j] - v * sn[j], b = v * cs[j] + u * sn[j];
        x[j] = a; x[j + half] = b;
        if (kd != nullptr) { kd[j] = from_f32<T>(a); kd[j + half] = from_f32<T>(b); }
      }
      for (int d = p.rot_dim + lane; d < D; d += 32) {
        const float u = x[d] * inv;
        x[d] = u;
        if (kd != nullptr) kd[d] = from_f32<T>(u);
      }
    }
  }
  if (page_ok) {                                       // the values of all heads, as they are
    T* dst = (T*)p.v_cache + slot * G * p.value_dim;
    for (int e = tid; e < G * p.value_dim; e += THREADS) dst[e] = row[p.v_off + e];
  }
  __syncthreads();

  // ---- mixed heads: places of the whole key row x sub-ranges of the block's heads, over the threads
  const int GD = G * D, places = GD / VEC;
  const int subs = places >= THREADS ? 1 : THREADS / places;
  for (int i = tid; i < places * subs; i += THREADS) {
    const int sub = i / places, at = (i - sub * places) * VEC;
    const int c = at / D, d = at - c * D;
    const float* q0 = qs + (size_t)c * HPT * D + d;      // query heads of key head c, D apart
    constexpr int REGS = HPTC > 0 ? HPTC : GROUP_REGS;
    float q[REGS][VEC];
#pragma unroll
    for (int g = 0; g < REGS; ++g) {
      if (VEC == 4) {
        const float4 f = g < HPT ? *reinterpret_cast<const float4*>(q0 + (size_t)g * D) : make_float4(0.f, 0.f, 0.f, 0.f);
        q[g][0] = f.x; q[g][VEC > 1 ? 1 : 0] = f.y; q[g][VEC > 2 ? 2 : 0] = f.z; q[g][VEC > 3 ? 3 : 0] = f.w;
      } else {
        q[g][0] = g < HPT ? q0[(size_t)g * D] : 0.f;
      }
    }
    const int n_here = h_hi - h_lo, lo = n_here * sub / subs, hi = n_here * (sub + 1) / subs;
    T* dst = (T*)p.q_out + ((size_t)t * H + h_lo) * GD + at;
#pragma unroll 2
    for (int h = lo; h < hi; ++h) {
      const float* w = ts + h * H + c * HPT;
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      if (HPTC > 0) {
#pragma unroll
        for (int g = 0; g < HPTC; g += 4) {
          const float4 wg = *reinterpret_cast<const float4*>(w + g);
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            acc[e] = fmaf(wg.x, q[g][e], acc[e]);
            acc[e] = fmaf(wg.y, q[g + 1][e], acc[e]);
            acc[e] = fmaf(wg.z, q[g + 2][e], acc[e]);
            acc[e] = fmaf(wg.w, q[g + 3][e], acc[e]);
          }
        }
      } else {
#pragma unroll
        for (int g = 0; g < REGS; ++g)
          if (g < HPT) {
            const float wg = w[g];
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] = fmaf(wg, q[g][e], acc[e]);
          }
        for (int g = REGS; g < HPT; ++g) {
          const float wg = w[g];
#pragma unroll
          for (int e = 0; e < VEC; ++e) acc[e] = fmaf(wg, q0[(size_t)g * D + e], acc[e]);
        }
      }
      Pack<T, VEC>::store(dst + (size_t)h * GD, acc);
    }
  }
}

template <typename T, int VEC, int HPTC, int ND>
int launch(const TalkParams& p, size_t smem, cudaStream_t stream) {
  auto kern = talk_prepare_kernel<T, VEC, HPTC, ND>;
  static bool ready[JV_MAX_DEVICES];
  if (!jv_once_per_device(ready, [&] {
        return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess;
      }))
    return JV_ERR_UNSUPPORTED;
  return jv_launch(kern, dim3((unsigned)(p.n * p.parts)), dim3(THREADS), smem, stream, p);
}
}  // namespace

// proj: [n, row_stride] of `dtype`; q_out: [n, H * G*D] of `dtype`; talk: [H, H] float; freq: [rot_dim/2] float or null
// (rot_dim 0); normed: query and key heads divided by their root mean square (eps inside the root); caches:
// [num_pages, page_size, G, D] and [num_pages, page_size, G, DV] of `dtype`, both null: queries only.
JV_EXPORT int jv_talk_prepare(const void* proj, int dtype, long long row_stride, int q_off, int k_off, int v_off, void* q_out,
                              const float* talk, const int* positions, const int* token_entry, const int* block_table,
                              int table_width, const float* freq, int rot_dim, int normed, float eps, void* k_cache,
                              void* v_cache, int n, int n_q_heads, int n_kv_heads, int key_dim, int value_dim,
                              int page_size, int num_pages, int* status, cudaStream_t stream) {
  if (n == 0) return JV_OK;
  if (n_kv_heads < 1 || n_q_heads % n_kv_heads || rot_dim < 0 || rot_dim > key_dim || (rot_dim & 1) ||
      (rot_dim > 0 && freq == nullptr) || key_dim < 1 || value_dim < 1 || page_size < 1 ||
      (k_cache == nullptr) != (v_cache == nullptr))
    return JV_ERR_UNSUPPORTED;
  TalkParams p;
  p.proj = proj; p.row_stride = row_stride; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.q_out = q_out; p.talk = talk;
  p.positions = positions; p.token_entry = token_entry; p.block_table = block_table; p.table_width = table_width;
  p.freq = freq; p.rot_dim = rot_dim; p.normed = normed ? 1 : 0; p.eps = eps; p.k_cache = k_cache; p.v_cache = v_cache;
  p.n = n; p.n_q_heads = n_q_heads; p.n_kv_heads = n_kv_heads; p.key_dim = key_dim; p.value_dim = value_dim;
  p.page_size = page_size; p.num_pages = num_pages; p.status = status;
  // a few tokens: their mixed heads are shared among blocks (every block prepares the token's queries for itself)
  p.parts = 1;
  while (p.parts < 8 && n * p.parts * 2 <= 148 && n_q_heads / (p.parts * 2) >= 2) p.parts *= 2;
  const size_t head_rows = (n_q_heads + p.parts - 1) / p.parts;
  const size_t up4 = ~(size_t)3;
  const size_t smem = sizeof(float) * (((head_rows * n_q_heads + 3) & up4) + (((size_t)n_q_heads * key_dim + 3) & up4) +
                                       (size_t)n_kv_heads * key_dim + rot_dim);
  if (smem > 200 * 1024) return JV_ERR_UNSUPPORTED;
  const bool vec = key_dim % 4 == 0 && (uintptr_t)q_out % 16 == 0;
  const int hpt = n_q_heads / n_kv_heads;
  const int nd = (vec && rot_dim % 64 == 0) ? (key_dim == 128 ? 4 : key_dim == 64 ? 2 : 0) : 0;
  JV_DISPATCH_DTYPE(dtype, T, {
    if (!vec) return launch<T, 1, 0, 0>(p, smem, stream);
    if (nd == 4) return hpt == 4 ? launch<T, 4, 4, 4>(p, smem, stream) : hpt == 8 ? launch<T, 4, 8, 4>(p, smem, stream)
                                                                                  : launch<T, 4, 0, 4>(p, smem, stream);
    if (nd == 2) return hpt == 4 ? launch<T, 4, 4, 2>(p, smem, stream) : hpt == 8 ? launch<T, 4, 8, 2>(p, smem, stream)
                                                                                  : launch<T, 4, 0, 2>(p, smem, stream);
    return launch<T, 4, 0, 0>(p, smem, stream);
  });
  return JV_ERR_UNSUPPORTED;
}
