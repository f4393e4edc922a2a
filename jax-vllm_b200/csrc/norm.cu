// RMSNorm over rows of the 32-bit residual stream, optionally fused with the residual
// sum that precedes it and with a row gather.
//
//   h[r, :] += delta[r, :]           (if delta is given; the sum is kept in 32-bit.  delta may come as
//                                     `parts` tensors `part_stride` elements apart, added in order: the
//                                     sums over the parts of k that a split product leaves)
//   y[i, :]  = h[r, :] * rsqrt(mean(h[r, :]^2) + eps) * weight[:]
//
// with r = rows[i] if `rows` is given, else r = i.  When `rows` is given the sum is
// not written back to h (the gathered rows are the last use of the stream).  Squares,
// mean, rsqrt and the scaling are 32-bit; the result is rounded once, to the output
// type.  With a second weight the same normed row times that weight is written too, to y2 (two branches that read the
// stream through a norm each).
#include "common.cuh"

template <typename TD, typename TW, typename TY>
__global__ void rmsnorm_kernel(float* __restrict__ h, const TD* __restrict__ delta,
                               const int* __restrict__ rows, const TW* __restrict__ weight,
                               TY* __restrict__ y, const TW* __restrict__ weight2, TY* __restrict__ y2, int hidden, float eps,
                               int n_rows_total, int* __restrict__ status, int parts, size_t part_stride) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  int r = i;
  if (rows != nullptr) {
    r = rows[i];
    if (r < 0 || r >= n_rows_total) {
      if (threadIdx.x == 0) atomicOr(status, JV_STATUS_BAD_ROW);
      for (int c = threadIdx.x; c < hidden; c += blockDim.x) y[(size_t)i * hidden + c] = from_f32<TY>(0.f);
      return;
    }
  }
  float* hr = h + (size_t)r * hidden;
  const TD* dr = delta ? delta + (size_t)r * hidden : nullptr;
  const bool write_back = (dr != nullptr) && (rows == nullptr);
  float ss = 0.f;
  auto delta_at = [&](int c) {
    float d = to_f32(dr[c]);
    for (int s = 1; s < parts; ++s) d += to_f32(dr[s * part_stride + c]);
    return d;
  };
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    float v = hr[c];
    if (dr) v += delta_at(c);
    if (write_back) hr[c] = v;
    ss += v * v;
  }
  ss = block_sum(ss, scratch);
  const float inv = rsqrtf(ss / (float)hidden + eps);
  TY* yr = y + (size_t)i * hidden;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    float v = hr[c];                          // this thread's own write, if any
    if (dr && !write_back) v += delta_at(c);
    yr[c] = from_f32<TY>(v * inv * to_f32(weight[c]));
    if (y2 != nullptr) y2[(size_t)i * hidden + c] = from_f32<TY>(v * inv * to_f32(weight2[c]));
  }
}

// The same with the row held in registers and 8 elements per thread and pass (hidden a multiple
// of 8, at most blockDim.x * 8 * RM_ITERS): one read of the stream, no second read for the scaling.
constexpr int RM_ITERS = 4;

template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&a);
#pragma unroll
  for (int k = 0; k < 4; ++k) { const float2 f = __bfloat1622float2(h[k]); v[2 * k] = f.x; v[2 * k + 1] = f.y; }
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 a;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&a);
#pragma unroll
  for (int k = 0; k < 4; ++k) h[k] = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
  *reinterpret_cast<uint4*>(p) = a;
}

// ITERS: passes per thread (1 for rows of up to 640 vectors of 8, else RM_ITERS).  TOGETHER: how many parts of a
// sum ask for their loads at once: 8 for a few rows (a decode step waits for this kernel, and one trip to the L2
// per part is most of its time), 1 for many rows, where registers are better spent on more blocks per
// multiprocessor.
template <typename TD, typename TW, typename TY, int ITERS, int TOGETHER>
__global__ void __launch_bounds__(ITERS == 1 ? 640 : 1024) rmsnorm_vec_kernel(float* __restrict__ h, const TD* __restrict__ delta,
                                   const int* __restrict__ rows, const TW* __restrict__ weight,
                                   TY* __restrict__ y, const TW* __restrict__ weight2, TY* __restrict__ y2, int hidden, float eps,
                                   int n_rows_total, int* __restrict__ status, int parts, size_t part_stride) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  int r = i;
  if (rows != nullptr) {
    r = rows[i];
    if (r < 0 || r >= n_rows_total) {
      if (threadIdx.x == 0) atomicOr(status, JV_STATUS_BAD_ROW);
      for (int c = threadIdx.x; c < hidden; c += blockDim.x) y[(size_t)i * hidden + c] = from_f32<TY>(0.f);
      return;
    }
  }
  float* hr = h + (size_t)r * hidden;
  const TD* dr = delta ? delta + (size_t)r * hidden : nullptr;
  const bool write_back = (dr != nullptr) && (rows == nullptr);
  float v[ITERS][8];
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * 8;
    if (c < hidden) {
      load8<float>(hr + c, v[it]);
      if (dr) {
        // the parts of a sum (eight at most ask for their loads together, then add in the order of the parts)
        float d[8];
        load8<TD>(dr + c, d);
        float e[TOGETHER][8];
#pragma unroll
        for (int s = 1; s < TOGETHER; ++s)
          if (s < parts) load8<TD>(dr + s * part_stride + c, e[s]);
#pragma unroll
        for (int s = 1; s < TOGETHER; ++s)
          if (s < parts) {
#pragma unroll
            for (int k = 0; k < 8; ++k) d[k] += e[s][k];
          }
        for (int s = TOGETHER; s < parts; ++s) {
          float f[8];
          load8<TD>(dr + s * part_stride + c, f);
#pragma unroll
          for (int k = 0; k < 8; ++k) d[k] += f[k];
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) v[it][k] += d[k];
        if (write_back) store8<float>(hr + c, v[it]);
      }
#pragma unroll
      for (int k = 0; k < 8; ++k) ss += v[it][k] * v[it][k];
    }
  }
  ss = block_sum(ss, scratch);
  const float inv = rsqrtf(ss / (float)hidden + eps);
  TY* yr = y + (size_t)i * hidden;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * 8;
    if (c < hidden) {
      float w[8];
      load8<TW>(weight + c, w);
#pragma unroll
      for (int k = 0; k < 8; ++k) w[k] = v[it][k] * inv * w[k];
      store8<TY>(yr + c, w);
      if (y2 != nullptr) {
        load8<TW>(weight2 + c, w);
#pragma unroll
        for (int k = 0; k < 8; ++k) w[k] = v[it][k] * inv * w[k];
        store8<TY>(y2 + (size_t)i * hidden + c, w);
      }
    }
  }
}

// h: [n_total, hidden] float (updated in place when delta is given and rows is null);
// delta: [n_total, hidden] of dtype `delta_dtype` or null, or `delta_parts` such tensors `delta_part_stride`
// elements apart whose sum it is; rows: [n_out] int32 or null;
// weight: [hidden] of dtype `weight_dtype`; y: [n_out, hidden] of dtype `out_dtype`; weight2, y2: a second weight and
// output of the same types, or both null (`rows` null).
JV_EXPORT int jv_rmsnorm(float* h, const void* delta, int delta_dtype, const int* rows,
                         const void* weight, int weight_dtype, void* y, int out_dtype, const void* weight2, void* y2,
                         int n_out, int n_total, int hidden, float eps, int delta_parts, long long delta_part_stride, int* status,
                         cudaStream_t stream) {
  if (n_out == 0) return JV_OK;
  if (delta_parts < 1 || (weight2 == nullptr) != (y2 == nullptr) || (y2 != nullptr && rows != nullptr))
    return JV_ERR_UNSUPPORTED;
  const int parts = delta_parts;
  const size_t part_stride = (size_t)delta_part_stride;
  const bool aligned = ((uintptr_t)h % 16) == 0 && ((uintptr_t)delta % 16) == 0 && ((uintptr_t)weight % 16) == 0 &&
                       ((uintptr_t)y % 16) == 0 && ((uintptr_t)weight2 % 16) == 0 && ((uintptr_t)y2 % 16) == 0;
  if (hidden % 8 == 0 && hidden <= 1024 * 8 * RM_ITERS && aligned && delta_part_stride % 8 == 0) {
    const int vecs = hidden / 8;
    int iters = vecs <= 640 ? 1 : (vecs + 511) / 512;     // up to 640 threads, then more passes per thread
    if (iters > RM_ITERS) iters = RM_ITERS;
    int vthreads = ((vecs + iters - 1) / iters + 31) / 32 * 32;
    if (vthreads > 1024) vthreads = 1024;
    if (iters == 1 && parts > 1 && n_out <= 256)
      JV_DISPATCH_DTYPE(out_dtype, TY, JV_DISPATCH_DTYPE(weight_dtype, TW, JV_DISPATCH_DTYPE(delta_dtype, TD,
          return jv_launch(rmsnorm_vec_kernel<TD, TW, TY, 1, 8>, dim3(n_out), dim3(vthreads), 0, stream,
                           h, (const TD*)delta, rows, (const TW*)weight, (TY*)y, (const TW*)weight2, (TY*)y2, hidden, eps, n_total, status, parts, part_stride))));
    if (iters == 1)
      JV_DISPATCH_DTYPE(out_dtype, TY, JV_DISPATCH_DTYPE(weight_dtype, TW, JV_DISPATCH_DTYPE(delta_dtype, TD,
          return jv_launch(rmsnorm_vec_kernel<TD, TW, TY, 1, 1>, dim3(n_out), dim3(vthreads), 0, stream,
                           h, (const TD*)delta, rows, (const TW*)weight, (TY*)y, (const TW*)weight2, (TY*)y2, hidden, eps, n_total, status, parts, part_stride))));
    JV_DISPATCH_DTYPE(out_dtype, TY, JV_DISPATCH_DTYPE(weight_dtype, TW, JV_DISPATCH_DTYPE(delta_dtype, TD,
        return jv_launch(rmsnorm_vec_kernel<TD, TW, TY, RM_ITERS, 1>, dim3(n_out), dim3(vthreads), 0, stream,
                         h, (const TD*)delta, rows, (const TW*)weight, (TY*)y, (const TW*)weight2, (TY*)y2, hidden, eps, n_total, status, parts, part_stride))));
    return JV_ERR_UNSUPPORTED;
  }
  int threads = 32;
  while (threads < 512 && threads * 4 < hidden) threads *= 2;
  JV_DISPATCH_DTYPE(out_dtype, TY, JV_DISPATCH_DTYPE(weight_dtype, TW, JV_DISPATCH_DTYPE(delta_dtype, TD,
      return jv_launch(rmsnorm_kernel<TD, TW, TY>, dim3(n_out), dim3(threads), 0, stream,
                       h, (const TD*)delta, rows, (const TW*)weight, (TY*)y, (const TW*)weight2, (TY*)y2, hidden, eps, n_total, status, parts, part_stride))));
  return JV_ERR_UNSUPPORTED;
}

// The norm behind a routed feed-forward.  What is added to row r is, in this order and in 32-bit,
//
//   delta[r, :]                                    (optional: float or 16-bit, as `parts` tensors like above)
//   sum_s coef[r, s] * picked[pick[r, s], :]       (s ascending: the weighted rows of its experts)
//   own_coef[r] * own[r, :]                        (optional: what identity experts give; a pick of -1 is then no row)
//
// and the sums are formed as they are added.  Rows of 8 elements a thread and pass where sizes and addresses allow (VEC),
// else one.
struct SumParams {
  float* h;
  const void* delta; int delta_f32, parts; size_t part_stride;
  const void* picked; const int* pick; const float* coef; int picks, picked_rows;
  const void* own; const float* own_coef;
  const int* rows;
  const void* weight; void* y;
  const void* weight2; void* y2;
  int hidden, n_rows_total;
  float eps;
  int* status;
};

template <typename TP, typename TW, typename TY, bool VEC>
__global__ void __launch_bounds__(1024) rmsnorm_sum_kernel(const SumParams p) {
  constexpr int V = VEC ? 8 : 1, TOGETHER = 4;
  extern __shared__ float kept[];                 // [hidden]: the row after the sum
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x, hidden = p.hidden;
  TY* yr = (TY*)p.y + (size_t)i * hidden;
  int r = i;
  if (p.rows != nullptr) {
    r = p.rows[i];
    if (r < 0 || r >= p.n_rows_total) {
      if (threadIdx.x == 0) atomicOr(p.status, JV_STATUS_BAD_ROW);
      for (int c = threadIdx.x; c < hidden; c += blockDim.x) yr[c] = from_f32<TY>(0.f);
      return;
    }
  }
  float* hr = p.h + (size_t)r * hidden;
  const int* pk = p.pick + (size_t)r * p.picks;
  const float* cf = p.coef + (size_t)r * p.picks;
  if (threadIdx.x < p.picks) {
    const int src = pk[threadIdx.x];
    if ((src < 0 || src >= p.picked_rows) && !(src == -1 && p.own != nullptr)) atomicOr(p.status, JV_STATUS_BAD_ROW);
  }
  const float oc = p.own != nullptr ? p.own_coef[r] : 0.f;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < hidden; c += blockDim.x * V) {
    float v[8], d[8];
    if (VEC) load8<float>(hr + c, v);
    else v[0] = hr[c];
#pragma unroll
    for (int k = 0; k < V; ++k) d[k] = 0.f;
    if (p.delta != nullptr) {
      const size_t at = (size_t)r * hidden + c;
      for (int s = 0; s < p.parts; ++s) {
        float e[8];
        if (p.delta_f32) {
          const float* src = (const float*)p.delta + s * p.part_stride + at;
          if (VEC) load8<float>(src, e);
          else e[0] = *src;
        } else {
          const __nv_bfloat16* src = (const __nv_bfloat16*)p.delta + s * p.part_stride + at;
          if (VEC) load8<__nv_bfloat16>(src, e);
          else e[0] = to_f32(*src);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) d[k] += e[k];
      }
    }
    for (int s0 = 0; s0 < p.picks; s0 += TOGETHER) {    // four rows ask for their loads together, then add in their order
      float e[TOGETHER][8], w[TOGETHER];
#pragma unroll
      for (int s = 0; s < TOGETHER; ++s) {
        const int src = s0 + s < p.picks ? pk[s0 + s] : -1;
        const bool ok = src >= 0 && src < p.picked_rows;
        w[s] = ok ? cf[s0 + s] : 0.f;
        const TP* row = (const TP*)p.picked + (size_t)(ok ? src : 0) * hidden + c;
        if (ok) {
          if (VEC) load8<TP>(row, e[s]);
          else e[s][0] = to_f32(*row);
        }
      }
#pragma unroll
      for (int s = 0; s < TOGETHER; ++s)
        if (w[s] != 0.f) {
#pragma unroll
          for (int k = 0; k < V; ++k) d[k] = fmaf(w[s], e[s][k], d[k]);
        }
    }
    if (oc != 0.f) {
      float e[8];
      const TP* row = (const TP*)p.own + (size_t)r * hidden + c;
      if (VEC) load8<TP>(row, e);
      else e[0] = to_f32(*row);
#pragma unroll
      for (int k = 0; k < V; ++k) d[k] = fmaf(oc, e[k], d[k]);
    }
#pragma unroll
    for (int k = 0; k < V; ++k) {
      v[k] += d[k];
      ss += v[k] * v[k];
      kept[c + k] = v[k];
    }
    if (p.rows == nullptr) {
      if (VEC) store8<float>(hr + c, v);
      else hr[c] = v[0];
    }
  }
  ss = block_sum(ss, scratch);
  const float inv = rsqrtf(ss / (float)hidden + p.eps);
  auto write = [&](const TW* weight, TY* out) {
    for (int c = threadIdx.x * V; c < hidden; c += blockDim.x * V) {   // a thread's own elements
      float w[8];
      if (VEC) load8<TW>(weight + c, w);
      else w[0] = to_f32(weight[c]);
#pragma unroll
      for (int k = 0; k < V; ++k) w[k] *= kept[c + k] * inv;
      if (VEC) store8<TY>(out + c, w);
      else out[c] = from_f32<TY>(w[0]);
    }
  };
  write((const TW*)p.weight, yr);
  if (p.y2 != nullptr) write((const TW*)p.weight2, (TY*)p.y2 + (size_t)i * hidden);
}

// As jv_rmsnorm, with a sum of picked rows in what is added: picked [picked_rows, hidden] and own [n_total, hidden] (or null)
// of dtype `picked_dtype`, pick and coef [n_total, picks], own_coef [n_total]; delta as for jv_rmsnorm, or null.
JV_EXPORT int jv_rmsnorm_sum(float* h, const void* delta, int delta_dtype, int delta_parts, long long delta_part_stride,
                             const void* picked, int picked_dtype, const int* pick, const float* coef, int picks,
                             int picked_rows, const void* own, const float* own_coef, const int* rows, const void* weight,
                             int weight_dtype, void* y, int out_dtype, const void* weight2, void* y2, int n_out, int n_total,
                             int hidden, float eps, int* status, cudaStream_t stream) {
  if (n_out == 0) return JV_OK;
  const size_t smem = sizeof(float) * (size_t)hidden;
  if (picks < 1 || picks > 64 || smem > 48 * 1024 - 256 || delta_parts < 1 || (own != nullptr && own_coef == nullptr) ||
      (weight2 == nullptr) != (y2 == nullptr) || (y2 != nullptr && rows != nullptr))
    return JV_ERR_UNSUPPORTED;
  SumParams p;
  p.h = h; p.delta = delta; p.delta_f32 = delta_dtype == 0; p.parts = delta_parts; p.part_stride = (size_t)delta_part_stride;
  p.picked = picked; p.pick = pick; p.coef = coef; p.picks = picks; p.picked_rows = picked_rows; p.own = own;
  p.own_coef = own_coef; p.rows = rows; p.weight = weight; p.y = y; p.weight2 = weight2; p.y2 = y2; p.hidden = hidden;
  p.n_rows_total = n_total; p.eps = eps; p.status = status;
  const bool vec = hidden % 8 == 0 && delta_part_stride % 8 == 0 && ((uintptr_t)h % 16) == 0 && ((uintptr_t)delta % 16) == 0 &&
                   ((uintptr_t)picked % 16) == 0 && ((uintptr_t)own % 16) == 0 && ((uintptr_t)weight % 16) == 0 &&
                   ((uintptr_t)y % 16) == 0 && ((uintptr_t)weight2 % 16) == 0 && ((uintptr_t)y2 % 16) == 0;
  const int units = vec ? hidden / 8 : hidden;
  int threads = 64;                               // `picks` threads at least
  while (threads < 512 && threads < units) threads *= 2;
  JV_DISPATCH_DTYPE(out_dtype, TY, JV_DISPATCH_DTYPE(weight_dtype, TW, JV_DISPATCH_DTYPE(picked_dtype, TP, {
      return jv_launch(vec ? rmsnorm_sum_kernel<TP, TW, TY, true> : rmsnorm_sum_kernel<TP, TW, TY, false>, dim3(n_out),
                       dim3(threads), smem, stream, p);
  })));
  return JV_ERR_UNSUPPORTED;
}

// Adds delta into the 32-bit stream without a norm: h[r, :] += delta[r, :].
template <typename TD>
__global__ void residual_add_kernel(float* __restrict__ h, const TD* __restrict__ delta, size_t n, int parts,
                                    size_t part_stride) {
  pdl_trigger();
  pdl_wait();
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; i < n; i += stride) {
    float d = to_f32(delta[i]);
    for (int s = 1; s < parts; ++s) d += to_f32(delta[s * part_stride + i]);
    h[i] += d;
  }
}

// delta as for jv_rmsnorm: one tensor (delta_parts 1) or the parts of a sum.
JV_EXPORT int jv_residual_add(float* h, const void* delta, int delta_dtype, long long n, int delta_parts,
                              long long delta_part_stride, cudaStream_t stream) {
  if (n == 0) return JV_OK;
  if (delta_parts < 1) return JV_ERR_UNSUPPORTED;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  JV_DISPATCH_DTYPE(delta_dtype, TD, return jv_launch(residual_add_kernel<TD>, dim3((int)blocks), dim3(256), 0, stream,
                                                      h, (const TD*)delta, (size_t)n, delta_parts,
                                                      (size_t)delta_part_stride));
  return JV_ERR_UNSUPPORTED;
}
