// The pass between two layers whose sublayers add into rows of their own: their sum joins the residual stream, and the norm that
// reads the stream next is done on the way.
//
//  * join_rows:   x += s * y per row of 32-bit numbers, y zeroed for the next layer to add into (with the partial sums that a
//                 up to two deferred products left for y added first); h = x / sqrt(mean(x^2) + eps) * w in the activation type, if wanted.
// One block per row; the row stays in registers between the sum and the norm.  All arithmetic is 32-bit.
#include <math.h>

#include "api.h"
#include "common.cuh"

namespace {

// VEC: groups of four numbers a thread holds (0: rows that are no multiple of 4, not aligned or too wide: a plain loop over
// memory).  SETTLE: of so many products partial sums are pending.  NORM: the norm follows.
template <typename TO, typename TW, int VEC, int SETTLE, bool NORM>
__global__ void __launch_bounds__(1024)
join_rows_kernel(float* x, float* y, float s, TO* h, const TW* w, int d, float eps, gi_settle_t st, gi_settle_t st2) {
  __shared__ float scratch[33];
  gi::pdl_launch_dependents();
  const size_t m = blockIdx.x;
  float* xr = x + m * d;
  float* yr = y + m * d;
  TO* hr = NORM ? h + m * d : nullptr;
  if (VEC > 0) {
    const int n4 = d / 4;
    // what no kernel of the step writes is read before the dependency wait
    float4 wv[VEC > 0 ? VEC : 1];
    gi_settle_span sp[VEC > 0 ? VEC : 1], sp2[VEC > 0 ? VEC : 1];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < n4) {
        if (NORM) wv[j] = gi::ld4(w + 4 * i);
        if (SETTLE > 0) sp[j] = gi_span_of(st, 4 * i);
        if (SETTLE > 1) sp2[j] = gi_span_of(st2, 4 * i);
      }
    }
    gi::pdl_wait();
    float4 v[VEC > 0 ? VEC : 1], u[VEC > 0 ? VEC : 1];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      v[j] = u[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < n4) {
        v[j] = reinterpret_cast<const float4*>(xr)[i];
        u[j] = reinterpret_cast<const float4*>(yr)[i];
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i >= n4) continue;
      if (SETTLE > 0 && sp[j].c_first != sp[j].c_last) {
        const float4 p = gi_sum_pieces4(st, sp[j], (int)m, 4 * i);
        u[j].x += p.x; u[j].y += p.y; u[j].z += p.z; u[j].w += p.w;
      }
      if (SETTLE > 1 && sp2[j].c_first != sp2[j].c_last) {
        const float4 p = gi_sum_pieces4(st2, sp2[j], (int)m, 4 * i);
        u[j].x += p.x; u[j].y += p.y; u[j].z += p.z; u[j].w += p.w;
      }
      v[j].x = fmaf(s, u[j].x, v[j].x); v[j].y = fmaf(s, u[j].y, v[j].y);
      v[j].z = fmaf(s, u[j].z, v[j].z); v[j].w = fmaf(s, u[j].w, v[j].w);
      reinterpret_cast<float4*>(xr)[i] = v[j];
      reinterpret_cast<float4*>(yr)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      ss = fmaf(v[j].x, v[j].x, ss); ss = fmaf(v[j].y, v[j].y, ss); ss = fmaf(v[j].z, v[j].z, ss); ss = fmaf(v[j].w, v[j].w, ss);
    }
    if (!NORM) return;
    const float r = 1.0f / sqrtf(gi::block_sum(ss, scratch) / (float)d + eps);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < n4) gi::st4(hr + 4 * i, make_float4(v[j].x * r * wv[j].x, v[j].y * r * wv[j].y, v[j].z * r * wv[j].z, v[j].w * r * wv[j].w));
    }
    return;
  }
  gi::pdl_wait();
  float ss = 0.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    const float v = fmaf(s, yr[i], xr[i]);
    xr[i] = v;
    yr[i] = 0.f;
    ss = fmaf(v, v, ss);
  }
  if (!NORM) return;
  const float r = 1.0f / sqrtf(gi::block_sum(ss, scratch) / (float)d + eps);
  for (int i = threadIdx.x; i < d; i += blockDim.x) gi::stf(hr + i, xr[i] * r * gi::ldf(w + i));     // a thread's own numbers
}

template <typename TO, typename TW, int SETTLE, bool NORM>
cudaError_t join_launch(int per, int rows, int threads, cudaStream_t stream, float* x, float* y, float s, TO* h, const TW* w, int d, float eps,
                        gi_settle_t st, gi_settle_t st2) {
  const dim3 g(rows), b(threads);
  if (per == 1) return gi::launch(join_rows_kernel<TO, TW, 1, SETTLE, NORM>, g, b, 0, stream, x, y, s, h, w, d, eps, st, st2);
  if (per == 2) return gi::launch(join_rows_kernel<TO, TW, 2, SETTLE, NORM>, g, b, 0, stream, x, y, s, h, w, d, eps, st, st2);
  if (per > 0) return gi::launch(join_rows_kernel<TO, TW, 4, SETTLE, NORM>, g, b, 0, stream, x, y, s, h, w, d, eps, st, st2);
  return gi::launch(join_rows_kernel<TO, TW, 0, 0, NORM>, g, b, 0, stream, x, y, s, h, w, d, eps, st, st2);
}

template <typename TO, typename TW, bool NORM>
cudaError_t join_pick(int settles, int per, int rows, int threads, cudaStream_t stream, float* x, float* y, float s, TO* h, const TW* w, int d,
                      float eps, gi_settle_t st, gi_settle_t st2) {
  if (settles == 2) return join_launch<TO, TW, 2, NORM>(per, rows, threads, stream, x, y, s, h, w, d, eps, st, st2);
  if (settles == 1) return join_launch<TO, TW, 1, NORM>(per, rows, threads, stream, x, y, s, h, w, d, eps, st, st2);
  return join_launch<TO, TW, 0, NORM>(per, rows, threads, stream, x, y, s, h, w, d, eps, st, st2);
}

}  // namespace

extern "C" int gi_join_rows(float* x, float* y, float scale, void* h, int h_dtype, const void* w, int w_dtype, int n_rows, int d, float eps,
                            gi_settle_t first, gi_settle_t second, void* stream) {
  if (n_rows <= 0) return GI_OK;
  if (d <= 0 || !x || !y || (h && !w)) return gi::fail(GI_ERR_ARG, "join rows: bad width %d or a missing pointer", d);
  if (first.partials == nullptr) { first = second; second = gi_settle_t{}; }
  const int settles = first.partials == nullptr ? 0 : (second.partials == nullptr ? 1 : 2);
  // a row's sum is formed in the order its width (and the type of the result) gives, whatever else the step holds, except that
  // many 16-bit rows take fewer threads each so that an SM holds more of them
  const bool many = n_rows >= 512 && h != nullptr && h_dtype != GI_F32;
  const int threads = d >= 4096 && !many ? 1024 : (d >= 2048 && !(many && d <= 4096) ? 512 : 256);
  const bool vec = d % 4 == 0 && d / 4 <= 4 * threads &&
                   (((uintptr_t)x | (uintptr_t)y | (uintptr_t)h | (uintptr_t)w) & 15) == 0;
  const int per = vec ? (d / 4 + threads - 1) / threads : 0;
  if (settles > 0 && per == 0)
    return gi::fail(GI_ERR_UNSUPPORTED, "join rows: settling partial sums needs aligned rows of a multiple of 4 and at most %d values", 16 * threads);
  cudaError_t e = cudaSuccess;
  if (h == nullptr) {
    e = join_pick<float, float, false>(settles, per, n_rows, threads, (cudaStream_t)stream, x, y, scale, (float*)nullptr, (const float*)nullptr,
                                       d, eps, first, second);
  } else {
    GI_DISPATCH_DTYPE(h_dtype, TO, GI_DISPATCH_DTYPE(w_dtype, TW,
        e = (join_pick<TO, TW, true>(settles, per, n_rows, threads, (cudaStream_t)stream, x, y, scale, (TO*)h, (const TW*)w, d, eps, first, second))));
  }
  return gi::check(e, "join rows");
}
