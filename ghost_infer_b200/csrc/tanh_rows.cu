// Row kernels for a residual stream whose norms are element-wise, tanh(alpha x) * w + b ("Dynamic Tanh": no mean, no variance),
// and for what sits around such a stream.
//
//  * tanh_rows:   one pass that joins a sublayer's output to the stream and prepares what the next reader of the stream wants:
//                     v = x + n1(y)           x or y may be absent; n1 a tanh norm, or y as it is
//                     x_out = v, or rows given ready made in its place (`base`); y is zeroed for the next sublayer to add into
//                     h = n2(v)               n2 a tanh norm, or v as it is, in the activation type
//                 x or y may have partial sums of a deferred product pending: they are added while the row is read.
//                 Since nothing here depends on a whole row, a thread takes four neighbouring channels and the grid is flat.
//  * softcap:     z = cap * tanh(z / cap) in place (logits).
//  * embed_pair:  e[t] = table[token] * scale + pairs[(prev * a + token * b) mod n], row n of the pair table for a sequence's
//                 first token.  The token before a step's first one comes from the sequence's state (one number per slot),
//                 which receives the step's last token of the sequence.
// All arithmetic is 32-bit.
#include <math.h>

#include "api.h"
#include "common.cuh"

namespace {

struct TanhRows {
  const float* x;          // null: no stream yet
  long ldx;
  const int* rows;         // null: every row in order; else output row r comes from row rows[r]
  float* y;                // null: nothing joins
  long ldy;
  int zero_y;
  float* x_out;            // null: the stream is not written; rows of d numbers, side by side
  const float* base;       // null: x_out takes the sum
  long ldb;
  float a1, a2;            // the norms' alphas
  const void *w1, *b1;     // null: y joins as it is
  const void *w2, *b2;     // null: h is the sum itself
  void* h;                 // null: nobody reads on
  int d, vec;
  int settle_of;           // 1: x, 2: y has partial sums pending, 0: neither
  gi_settle_t st;
};

template <typename T>
__device__ __forceinline__ float4 tr_get(const T* p, int n, int vec) {
  if (vec) return gi::ld4(p);
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  v.x = gi::ldf(p);
  if (n > 1) v.y = gi::ldf(p + 1);
  if (n > 2) v.z = gi::ldf(p + 2);
  if (n > 3) v.w = gi::ldf(p + 3);
  return v;
}
template <typename T>
__device__ __forceinline__ void tr_put(T* p, float4 v, int n, int vec) {
  if (vec) { gi::st4(p, v); return; }
  gi::stf(p, v.x);
  if (n > 1) gi::stf(p + 1, v.y);
  if (n > 2) gi::stf(p + 2, v.z);
  if (n > 3) gi::stf(p + 3, v.w);
}
// The tanh of the 16-bit path: gi::tanh_fast (good to about 1e-7 of 1), and below 0.2, where that would lose relative accuracy,
// the first four terms of the series x - x^3/3 + 2 x^5/15 - 17 x^7/315: a few units in the last place of a float everywhere, at a
// third of tanhf's instructions and without its branch, which leaves the pass to the memory.
template <bool QUICK>
__device__ __forceinline__ float tr_tanh(float x) {
  if (!QUICK) return tanhf(x);
  const float q = x * x;
  const float series = x * fmaf(q, fmaf(q, fmaf(q, -17.0f / 315.0f, 2.0f / 15.0f), -1.0f / 3.0f), 1.0f);
  const float wide = gi::tanh_fast(fminf(fmaxf(x, -16.0f), 16.0f));      // beyond, tanh is 1 to the last bit
  return fabsf(x) < 0.2f ? series : wide;
}
template <bool QUICK>
__device__ __forceinline__ float4 tr_norm(float4 v, float alpha, float4 w, float4 b) {
  return make_float4(fmaf(tr_tanh<QUICK>(alpha * v.x), w.x, b.x), fmaf(tr_tanh<QUICK>(alpha * v.y), w.y, b.y),
                     fmaf(tr_tanh<QUICK>(alpha * v.z), w.z, b.z), fmaf(tr_tanh<QUICK>(alpha * v.w), w.w, b.w));
}
__device__ __forceinline__ float4 tr_add(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }

// SETTLE: some row has sums pending (their loads in flight cost registers the plain pass does without).
template <typename TW, typename TH, bool QUICK, bool SETTLE>
__global__ void __launch_bounds__(256)
tanh_rows_kernel(const TanhRows a, unsigned total) {
  gi::pdl_launch_dependents();
  const unsigned g = blockIdx.x * blockDim.x + threadIdx.x;
  const unsigned per = (a.d + 3) / 4;
  const bool live = g < total;
  const unsigned r = live ? g / per : 0;
  const int c = live ? (int)(g - r * per) * 4 : 0;
  const int n = min(4, a.d - c);
  const float4 z4 = make_float4(0.f, 0.f, 0.f, 0.f);
  // weights and the tables of a deferred product's cut are written by no kernel of the step: read before the wait
  float4 w1 = z4, b1 = z4, w2 = z4, b2 = z4;
  if (a.w1 != nullptr) { w1 = tr_get((const TW*)a.w1 + c, n, a.vec); b1 = tr_get((const TW*)a.b1 + c, n, a.vec); }
  if (a.w2 != nullptr) { w2 = tr_get((const TW*)a.w2 + c, n, a.vec); b2 = tr_get((const TW*)a.b2 + c, n, a.vec); }
  gi_settle_span sp = {0, 0, 0};
  if (SETTLE) sp = gi_span_of(a.st, c);
  const long m = a.rows != nullptr ? gi::ld_step(a.rows + r) : (long)r;
  gi::pdl_wait();
  if (!live) return;
  float* yp = a.y + m * a.ldy + c;
  float4 v = z4, u = z4;
  if (a.x != nullptr) v = tr_get(a.x + m * a.ldx + c, n, a.vec);
  if (a.y != nullptr) u = tr_get((const float*)yp, n, a.vec);
  if (a.x != nullptr) {
    if (SETTLE && a.settle_of == 1 && sp.c_first != sp.c_last) v = tr_add(v, gi_sum_pieces4(a.st, sp, (int)m, c));
  }
  if (a.y != nullptr) {
    if (SETTLE && a.settle_of == 2 && sp.c_first != sp.c_last) u = tr_add(u, gi_sum_pieces4(a.st, sp, (int)m, c));
    if (a.w1 != nullptr) u = tr_norm<QUICK>(u, a.a1, w1, b1);
    v = a.x != nullptr ? tr_add(v, u) : u;
    if (a.zero_y) tr_put(yp, z4, n, a.vec);
  }
  if (a.x_out != nullptr) {
    float4 o = v;
    if (a.base != nullptr) o = tr_get(a.base + m * a.ldb + c, n, a.vec);
    tr_put(a.x_out + m * a.d + c, o, n, a.vec);
  }
  if (a.h != nullptr) {
    if (a.w2 != nullptr) v = tr_norm<QUICK>(v, a.a2, w2, b2);
    tr_put((TH*)a.h + (size_t)r * a.d + c, v, n, a.vec);
  }
}

__global__ void softcap_kernel(float* x, float cap, long total) {
  gi::pdl_prologue();
  const long e = ((long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (e >= total) return;
  const int n = (int)min(4L, total - e);
  const int vec = n == 4 && ((uintptr_t)x & 15) == 0;
  float4 v = tr_get((const float*)x + e, n, vec);
  v = make_float4(cap * tanhf(v.x / cap), cap * tanhf(v.y / cap), cap * tanhf(v.z / cap), cap * tanhf(v.w / cap));
  tr_put(x + e, v, n, vec);
}

// One block per token.
template <typename TW>
__global__ void __launch_bounds__(256)
embed_pair_kernel(float* __restrict__ out, const TW* __restrict__ table, const TW* __restrict__ pairs, const int* tokens,
                  const int* positions, const int* slots, const int* cu_seqlens, int n_seqs, int* state, long state_ld, int d,
                  int vocab, float scale, int buckets, long long mul_prev, long long mul_cur, int vec) {
  gi::pdl_prologue();
  const int t = blockIdx.x, slot = slots[t];
  int id = tokens[t];
  if (id < 0 || id >= vocab) id = 0;      // the host validates ids; padding rows may carry anything
  const bool opens = slot >= 0 && (t == 0 || slots[t - 1] != slot);     // the step's first token of its sequence
  long row = buckets;
  if (positions[t] > 0 && slot >= 0) {
    int prev = opens ? state[slot * state_ld] : tokens[t - 1];
    if (prev < 0 || prev >= vocab) prev = 0;
    row = (long)(((long long)prev * mul_prev + (long long)id * mul_cur) % buckets);
  }
  if (opens) {
    __syncthreads();                       // every thread has read the state
    for (int b = threadIdx.x; b < n_seqs; b += blockDim.x)
      if (cu_seqlens[b] == t && cu_seqlens[b + 1] > t) state[slot * state_ld] = tokens[cu_seqlens[b + 1] - 1];
  }
  const TW* e = table + (size_t)id * d;
  const TW* p = pairs + (size_t)row * d;
  float* o = out + (size_t)t * d;
  for (int c = threadIdx.x * 4; c < d; c += blockDim.x * 4) {
    const int n = min(4, d - c);
    const float4 ev = tr_get(e + c, n, vec), pv = tr_get(p + c, n, vec);
    tr_put(o + c, make_float4(fmaf(ev.x, scale, pv.x), fmaf(ev.y, scale, pv.y), fmaf(ev.z, scale, pv.z), fmaf(ev.w, scale, pv.w)), n, vec);
  }
}

}  // namespace

extern "C" int gi_tanh_rows(const float* x, long ldx, const int* rows, float* y, long ldy, int zero_y, float* x_out, const float* base,
                            long ldb, float alpha1, const void* w1, const void* b1, float alpha2, const void* w2, const void* b2,
                            int w_dtype, void* h, int h_dtype, int n_rows, int d, int quick, int settle_of, gi_settle_t settle, void* stream) {
  if (n_rows <= 0) return GI_OK;
  if (d <= 0 || (!x && !y)) return gi::fail(GI_ERR_ARG, "tanh rows: bad width %d or nothing to read", d);
  if ((w1 && !b1) || (w2 && !b2)) return gi::fail(GI_ERR_ARG, "tanh rows: a norm needs its weight and its bias");
  if (rows && (x_out || y)) return gi::fail(GI_ERR_ARG, "tanh rows: a selection of rows is only read");
  if (base && !x_out) return gi::fail(GI_ERR_ARG, "tanh rows: nowhere to put the ready-made rows");
  TanhRows a;
  a.x = x; a.ldx = ldx; a.rows = rows; a.y = y; a.ldy = ldy; a.zero_y = zero_y; a.x_out = x_out; a.base = base; a.ldb = ldb;
  a.a1 = alpha1; a.a2 = alpha2; a.w1 = w1; a.b1 = b1; a.w2 = w2; a.b2 = b2; a.h = h; a.d = d;
  a.vec = (d % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && ldb % 4 == 0 &&
           (((uintptr_t)x | (uintptr_t)y | (uintptr_t)x_out | (uintptr_t)base | (uintptr_t)w1 | (uintptr_t)b1 | (uintptr_t)w2 |
             (uintptr_t)b2 | (uintptr_t)h) & 15) == 0) ? 1 : 0;
  a.settle_of = settle.partials != nullptr ? settle_of : 0;
  a.st = settle;
  if (a.settle_of && d % 4 != 0) return gi::fail(GI_ERR_UNSUPPORTED, "tanh rows: settling partial sums needs rows of a multiple of 4 values");
  const long total = (long)n_rows * ((d + 3) / 4);
  const int threads = total <= 148L * 256 ? 64 : 256;      // few rows: more blocks, so that every SM takes part
  const long blocks = (total + threads - 1) / threads;
  if (total > 0x7fffff00L) return gi::fail(GI_ERR_UNSUPPORTED, "tanh rows: too many rows for one launch");
  cudaError_t e = cudaSuccess;
  GI_DISPATCH_DTYPE(w_dtype, TW, GI_DISPATCH_DTYPE(h_dtype, TH, {
    auto kern = a.settle_of ? (quick ? tanh_rows_kernel<TW, TH, true, true> : tanh_rows_kernel<TW, TH, false, true>)
                            : (quick ? tanh_rows_kernel<TW, TH, true, false> : tanh_rows_kernel<TW, TH, false, false>);
    e = gi::launch(kern, dim3((unsigned)blocks), dim3(threads), 0, (cudaStream_t)stream, a, (unsigned)total);
  }));
  return gi::check(e, "tanh rows");
}

extern "C" int gi_softcap_rows(float* x, float cap, long n_values, void* stream) {
  if (n_values <= 0) return GI_OK;
  if (!(cap > 0.f)) return gi::fail(GI_ERR_ARG, "softcap: the cap must be positive");
  const long blocks = (n_values + 1023) / 1024;
  if (blocks > 0x7fffffffL) return gi::fail(GI_ERR_UNSUPPORTED, "softcap: too many values for one launch");
  cudaError_t e = gi::launch(softcap_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, x, cap, n_values);
  return gi::check(e, "softcap");
}

extern "C" int gi_embed_pair(float* out, const void* table, const void* pairs, int w_dtype, const int* tokens, const int* positions,
                             const int* slots, const int* cu_seqlens, int n_seqs, int* state, long state_ld, int n_tokens, int d,
                             int vocab, float scale, int buckets, long long mul_prev, long long mul_cur, void* stream) {
  if (n_tokens <= 0) return GI_OK;
  if (d <= 0 || vocab <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0)
    return gi::fail(GI_ERR_ARG, "pair embedding: bad sizes (width %d, vocabulary %d, pairs %d)", d, vocab, buckets);
  if (!table || !pairs || !state || !cu_seqlens) return gi::fail(GI_ERR_ARG, "pair embedding: a missing pointer");
  const int vec = (d % 4 == 0 && (((uintptr_t)out | (uintptr_t)table | (uintptr_t)pairs) & 15) == 0) ? 1 : 0;
  cudaError_t e = cudaSuccess;
  GI_DISPATCH_DTYPE(w_dtype, TW,
      e = gi::launch(embed_pair_kernel<TW>, dim3(n_tokens), dim3(256), 0, (cudaStream_t)stream, out, (const TW*)table, (const TW*)pairs,
                     tokens, positions, slots, cu_seqlens, n_seqs, state, state_ld, d, vocab, scale, buckets, mul_prev, mul_cur, vec));
  return gi::check(e, "pair embedding");
}
