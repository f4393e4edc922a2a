// A gated recurrence whose gates read only the current token ("minimal GRU"), element by element over C channels:
//
//   z = sigmoid(zl + zb),  y = yl + yb,  candidate = y + 1/2 where y >= 0, sigmoid(y) elsewhere
//   S <- (1 - z) S + z * candidate,      out = scale * S * silu(g)
//
// zl, yl and g are column ranges of the packed projection; everything from them on is 32-bit, the state is a row of
// floats in the request's state slot.  Since the gates do not read the state, a run of tokens is one affine map of it:
// S -> (1 - D) S + B with 1 - D the product of the (1 - z) and B what the run makes of a zero state.  Every update is
// written as S + z (candidate - S), and D is carried rather than 1 - D: a gate close to zero keeps its relative precision
// over thousands of tokens, which 1 - z rounded to 32-bit does not.  A block takes CB channels of one entry in tiles of
// tokens: every thread reads TPT tokens of one channel (the loads of the next tile fly while this one is computed), forms
// their gates and candidates in registers and the pair (D, B) of its run, the runs of a tile are chained through shared
// memory from the state that the tile before left, and every thread goes through its tokens again from its true start.
// One pass over memory, one launch; the order of the sums differs from token by token by 32-bit rounding only.  A step of
// single tokens is a flat kernel, one thread a channel.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int TPT = 8;            // tokens of a thread per tile
constexpr int THREADS = 1024;

struct GruParams {
  const void* proj; long long stride; int z_off, x_off, g_off;
  const void* z_bias; const void* x_bias;
  void* out; long long out_stride;
  float* state; long long slot_stride;
  const int* cu_seqlens; const int* slots;
  int n_slots, channels;
  float scale;
  int* status;
};

// sigmoid(x) = 1 / (1 + e^-x): of a large negative x the sum is infinite and the result 0, and a small result keeps its
// relative precision.  EXACT (32-bit projections): library exponential and division; else one instruction each for the
// power of two and the reciprocal, whose error is far below the 16-bit rounding of what they are given.
template <bool EXACT> __device__ __forceinline__ float sigmoid_of(float x) {
  if (EXACT) return 1.f / (1.f + expf(-x));
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(x * -1.4426950408889634f));
  asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(r) : "f"(1.f + e));
  return r;
}

// Gate and candidate of one token.
template <bool EXACT>
__device__ __forceinline__ void gru_pair(float zl, float y, float& z, float& c) {
  z = sigmoid_of<EXACT>(zl);
  const float low = sigmoid_of<EXACT>(y);
  c = y >= 0.f ? y + 0.5f : low;
}
__device__ __forceinline__ float blend(float S, float z, float c) { return fmaf(z, c - S, S); }
template <bool EXACT>
__device__ __forceinline__ float silu_of(float g) { return g * sigmoid_of<EXACT>(g); }

// CB channels a block, THREADS / CB runs of TPT tokens a tile.
template <typename T, typename W, int CB>
__global__ void __launch_bounds__(THREADS, 1) gru_scan_kernel(const GruParams p) {
  constexpr int RUNS = THREADS / CB, TILE = RUNS * TPT;
  constexpr bool EXACT = sizeof(T) == 4;
  __shared__ float Ds[RUNS][CB], Bs[RUNS][CB];
  __shared__ float carry[2][CB];
  pdl_trigger();
  const int cl = threadIdx.x % CB, run = threadIdx.x / CB;
  const int c = blockIdx.y * CB + cl;
  const bool live = c < p.channels;
  const float zb = live ? to_f32(((const W*)p.z_bias)[c]) : 0.f, xb = live ? to_f32(((const W*)p.x_bias)[c]) : 0.f;
  pdl_wait();
  const int entry = blockIdx.x;
  const int t0 = p.cu_seqlens[entry], t1 = p.cu_seqlens[entry + 1];
  const int slot = p.slots[entry];
  if (slot < 0 || slot >= p.n_slots) {
    if (threadIdx.x == 0) atomicOr(p.status, JV_STATUS_BAD_ROW);
    return;
  }
  float* S_g = p.state + (size_t)slot * p.slot_stride + c;
  if (run == 0) carry[0][cl] = live ? *S_g : 0.f;
  const T* row = (const T*)p.proj + c;
  T zr[TPT], xr[TPT], gr[TPT];
  auto fetch = [&](int tile0) {
    const int first = tile0 + run * TPT, n_here = live ? t1 - first : 0;
    const T* at = row + (size_t)first * p.stride;
    if (n_here >= TPT) {
#pragma unroll
      for (int i = 0; i < TPT; ++i, at += p.stride) { zr[i] = at[p.z_off]; xr[i] = at[p.x_off]; gr[i] = at[p.g_off]; }
    } else {
#pragma unroll
      for (int i = 0; i < TPT; ++i, at += p.stride) {
        zr[i] = xr[i] = gr[i] = from_f32<T>(0.f);
        if (i < n_here) { zr[i] = at[p.z_off]; xr[i] = at[p.x_off]; gr[i] = at[p.g_off]; }
      }
    }
  };
  fetch(t0);
  int which = 0;
  for (int tile0 = t0; tile0 < t1; tile0 += TILE, which ^= 1) {
    const int first = tile0 + run * TPT, n_here = live ? t1 - first : 0;
    float z[TPT], cand[TPT], g[TPT];
    float D = 0.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < TPT; ++i) {
      gru_pair<EXACT>(to_f32(zr[i]) + zb, to_f32(xr[i]) + xb, z[i], cand[i]);
      g[i] = p.scale * silu_of<EXACT>(to_f32(gr[i]));
      if (i >= n_here) z[i] = 0.f;                         // no token: the state passes
      D = blend(D, z[i], 1.f);
      B = blend(B, z[i], cand[i]);
    }
    if (tile0 + TILE < t1) fetch(tile0 + TILE);
    Ds[run][cl] = D;
    Bs[run][cl] = B;
    __syncthreads();
    float S = carry[which][cl];
#pragma unroll 8
    for (int r = 0; r < run; ++r) S = fmaf(-Ds[r][cl], S, S) + Bs[r][cl];
    if (run == RUNS - 1) carry[which ^ 1][cl] = fmaf(-D, S, S) + B;
    T* out = (T*)p.out + (size_t)first * p.out_stride + c;
    if (n_here >= TPT) {
#pragma unroll
      for (int i = 0; i < TPT; ++i, out += p.out_stride) {
        S = blend(S, z[i], cand[i]);
        *out = from_f32<T>(S * g[i]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < TPT; ++i, out += p.out_stride) {
        S = blend(S, z[i], cand[i]);
        if (i < n_here) *out = from_f32<T>(S * g[i]);
      }
    }
    __syncthreads();                                       // the runs' pairs have been read; the carry is there
  }
  if (run == 0 && live && t1 > t0) *S_g = carry[which][cl];
}

template <typename T, typename W>
__global__ void __launch_bounds__(128) gru_single_kernel(const GruParams p) {
  constexpr bool EXACT = sizeof(T) == 4;
  pdl_trigger();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.channels) return;
  const float zb = to_f32(((const W*)p.z_bias)[c]), xb = to_f32(((const W*)p.x_bias)[c]);
  pdl_wait();
  const int t = p.cu_seqlens[blockIdx.x];
  const int slot = p.slots[blockIdx.x];
  if (slot < 0 || slot >= p.n_slots) {
    if (threadIdx.x == 0) atomicOr(p.status, JV_STATUS_BAD_ROW);
    return;
  }
  const T* row = (const T*)p.proj + (size_t)t * p.stride;
  float* S_g = p.state + (size_t)slot * p.slot_stride + c;
  const float zl = to_f32(row[p.z_off + c]), y = to_f32(row[p.x_off + c]), g = to_f32(row[p.g_off + c]), S0 = *S_g;
  float z, cand;
  gru_pair<EXACT>(zl + zb, y + xb, z, cand);
  const float S = blend(S0, z, cand);
  *S_g = S;
  ((T*)p.out)[(size_t)t * p.out_stride + c] = from_f32<T>(p.scale * S * silu_of<EXACT>(g));
}
}  // namespace

// proj: rows of `stride` elements of `dtype` with the three pre-activations (C columns each) at the given columns;
// z_bias, x_bias: [C] of `w_dtype`; out: rows of `out_stride` elements of `dtype`; state: row of slot 0, rows
// `slot_stride` floats apart.  singles != 0: every entry has exactly one token.
JV_EXPORT int jv_min_gru(const void* proj, int dtype, long long stride, int z_off, int x_off, int g_off, const void* z_bias,
                         const void* x_bias, int w_dtype, void* out, long long out_stride, float* state,
                         long long slot_stride, const int* cu_seqlens, const int* slots, int n_slots, int entries,
                         int channels, float scale, int singles, int* status, cudaStream_t stream) {
  if (entries == 0 || channels == 0) return JV_OK;
  GruParams p;
  p.proj = proj; p.stride = stride; p.z_off = z_off; p.x_off = x_off; p.g_off = g_off; p.z_bias = z_bias; p.x_bias = x_bias;
  p.out = out; p.out_stride = out_stride; p.state = state; p.slot_stride = slot_stride; p.cu_seqlens = cu_seqlens;
  p.slots = slots; p.n_slots = n_slots; p.channels = channels; p.scale = scale; p.status = status;
  JV_DISPATCH_DTYPE(dtype, T, JV_DISPATCH_DTYPE(w_dtype, W, {
    if (singles)
      return jv_launch(gru_single_kernel<T, W>, dim3(entries, (channels + 127) / 128), dim3(128), 0, stream, p);
    // half a warp's worth of channels a block where whole warps would leave multiprocessors without a block
    if ((long long)entries * ((channels + 31) / 32) < 120)
      return jv_launch(gru_scan_kernel<T, W, 16>, dim3(entries, (channels + 15) / 16), dim3(THREADS), 0, stream, p);
    return jv_launch(gru_scan_kernel<T, W, 32>, dim3(entries, (channels + 31) / 32), dim3(THREADS), 0, stream, p);
  }));
  return JV_ERR_UNSUPPORTED;
}
