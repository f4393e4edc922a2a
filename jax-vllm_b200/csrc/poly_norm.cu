// The activation of a feed-forward made of normed powers: for a token's vector z of `width` values and four numbers
//
//   out = a N(z) + b N(z^2) + c N(z^3) + e,      N(y) = y / sqrt(mean(y^2) + eps),  powers element by element
//
// so a row needs its sums of squares, fourth and sixth powers.  One block a row; the row stays in registers between the
// sums and the result where it fits.  z may come as `parts` float tensors `part_stride` elements apart whose sum it is
// (what a product leaves whose k was cut into parts), added in order as they are read.  32-bit arithmetic; the result is
// rounded once.
#include "common.cuh"

namespace {
constexpr int VEC = 4;

template <typename T> __device__ __forceinline__ void load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void load4<float>(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <> __device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 a = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&a);
  const float2 f0 = __bfloat1622float2(h[0]), f1 = __bfloat1622float2(h[1]);
  v[0] = f0.x; v[1] = f0.y; v[2] = f1.x; v[3] = f1.y;
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float (&v)[4]);
template <> __device__ __forceinline__ void store4<float>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[4]) {
  uint2 a;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&a);
  h[0] = __floats2bfloat162_rn(v[0], v[1]);
  h[1] = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = a;
}

// The three sums over the block, one barrier pair for all of them.
__device__ __forceinline__ void block_sum3(float& x, float& y, float& z, float (*scratch)[33]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  x = warp_sum(x); y = warp_sum(y); z = warp_sum(z);
  if (lane == 0) { scratch[0][warp] = x; scratch[1][warp] = y; scratch[2][warp] = z; }
  __syncthreads();
  x = warp_sum(lane < nwarps ? scratch[0][lane] : 0.f);
  y = warp_sum(lane < nwarps ? scratch[1][lane] : 0.f);
  z = warp_sum(lane < nwarps ? scratch[2][lane] : 0.f);
}

struct Coef { float k1, k2, k3, e; };
template <typename W>
__device__ __forceinline__ Coef finish(float s2, float s4, float s6, const W* coef, int width, float eps) {
  const float inv = 1.f / (float)width;
  return Coef{to_f32(coef[0]) / sqrtf(s2 * inv + eps), to_f32(coef[1]) / sqrtf(s4 * inv + eps),
              to_f32(coef[2]) / sqrtf(s6 * inv + eps), to_f32(coef[3])};
}
__device__ __forceinline__ float poly(const Coef& k, float z) { return fmaf(z, fmaf(z, fmaf(z, k.k3, k.k2), k.k1), k.e); }

// Rows of up to blockDim.x * VEC * ITERS values, a multiple of VEC, on aligned addresses.
template <typename TI, typename T, typename W, int ITERS>
__global__ void __launch_bounds__(ITERS > 8 ? 256 : 1024) poly_norm_vec_kernel(const TI* __restrict__ in, long long in_stride, T* __restrict__ out, long long out_stride,
                                     const W* __restrict__ coef, int width, float eps, int parts, size_t part_stride) {
  __shared__ float scratch[3][33];
  pdl_trigger();
  pdl_wait();
  const TI* src = in + (size_t)blockIdx.x * in_stride;
  T* dst = out + (size_t)blockIdx.x * out_stride;
  float v[ITERS][VEC];
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c < width) load4<TI>(src + c, v[it]);
    else
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[it][i] = 0.f;
  }
  for (int s = 1; s < parts; ++s)
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int c = (it * blockDim.x + threadIdx.x) * VEC;
      if (c < width) {
        float w[VEC];
        load4<TI>(src + s * part_stride + c, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[it][i] += w[i];
      }
    }
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
#pragma unroll
  for (int it = 0; it < ITERS; ++it)
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const float q = v[it][i] * v[it][i], q2 = q * q;
      s2 += q;
      s4 += q2;
      s6 = fmaf(q2, q, s6);
    }
  block_sum3(s2, s4, s6, scratch);
  const Coef k = finish(s2, s4, s6, coef, width, eps);
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c < width) {
      float y[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = poly(k, v[it][i]);
      store4<T>(dst + c, y);
    }
  }
}

// Any width and alignment: the row is read twice.
template <typename TI, typename T, typename W>
__global__ void poly_norm_kernel(const TI* __restrict__ in, long long in_stride, T* __restrict__ out, long long out_stride,
                                 const W* __restrict__ coef, int width, float eps, int parts, size_t part_stride) {
  __shared__ float scratch[3][33];
  pdl_trigger();
  pdl_wait();
  const TI* src = in + (size_t)blockIdx.x * in_stride;
  T* dst = out + (size_t)blockIdx.x * out_stride;
  auto at = [&](int c) {
    float v = to_f32(src[c]);
    for (int s = 1; s < parts; ++s) v += to_f32(src[s * part_stride + c]);
    return v;
  };
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = at(c), q = v * v, q2 = q * q;
    s2 += q;
    s4 += q2;
    s6 = fmaf(q2, q, s6);
  }
  block_sum3(s2, s4, s6, scratch);
  const Coef k = finish(s2, s4, s6, coef, width, eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x) dst[c] = from_f32<T>(poly(k, at(c)));
}

template <typename TI, typename T, typename W>
int launch(const void* in, long long in_stride, void* out, long long out_stride, const void* coef, int n, int width, float eps,
           int parts, long long part_stride, cudaStream_t stream) {
  const size_t ai = sizeof(TI) * VEC, ao = sizeof(T) * VEC;
  const bool vec = width % VEC == 0 && in_stride % VEC == 0 && out_stride % VEC == 0 && part_stride % VEC == 0 &&
                   (uintptr_t)in % ai == 0 && (uintptr_t)out % ao == 0;
  const int per = width / VEC;
  // a few rows: as many threads as a row has vectors, up to 1,024; many rows: four vectors a thread where that leaves 128
  // threads at least
  int threads = 1024;
  while (threads > 64 && threads / 2 >= per) threads /= 2;
  if (n > 148)
    while (threads > 128 && (per + threads / 2 - 1) / (threads / 2) <= 4) threads /= 2;
  const int iters = (per + threads - 1) / threads;
#define JV_POLY(I)                                                                                                          \
  if (vec && iters <= I)                                                                                                    \
    return jv_launch(poly_norm_vec_kernel<TI, T, W, I>, dim3(n), dim3(threads), 0, stream, (const TI*)in, in_stride,         \
                     (T*)out, out_stride, (const W*)coef, width, eps, parts, (size_t)part_stride)
  JV_POLY(1); JV_POLY(2); JV_POLY(4); JV_POLY(8);
  if (threads <= 256) { JV_POLY(16); }
#undef JV_POLY
  return jv_launch(poly_norm_kernel<TI, T, W>, dim3(n), dim3(width >= 2048 ? 512 : 128), 0, stream, (const TI*)in, in_stride,
                   (T*)out, out_stride, (const W*)coef, width, eps, parts, (size_t)part_stride);
}
}  // namespace

// in: [n] rows of in_stride elements of in_dtype (parts > 1: float tensors part_stride elements apart); out: rows of
// out_stride elements of out_dtype; coef: the four numbers, of w_dtype.
JV_EXPORT int jv_poly_norm(const void* in, int in_dtype, long long in_stride, int parts, long long part_stride, void* out,
                           int out_dtype, long long out_stride, const void* coef, int w_dtype, float eps, int n, int width,
                           cudaStream_t stream) {
  if (n == 0) return JV_OK;
  if (width < 1 || parts < 1) return JV_ERR_UNSUPPORTED;
  JV_DISPATCH_DTYPE(in_dtype, TI, JV_DISPATCH_DTYPE(out_dtype, TO, JV_DISPATCH_DTYPE(w_dtype, W,
      return (launch<TI, TO, W>(in, in_stride, out, out_stride, coef, n, width, eps, parts, part_stride, stream)))));
  return JV_ERR_UNSUPPORTED;
}
