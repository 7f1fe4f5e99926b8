// Row kernels around attention whose heads are the difference of two maps (two pairs of query and key, one value).
//
//  * map_prepare:    one token's float32 row [q: H heads x 2 maps x n | k: G x 2 x n | v: G x m] of the projection.  Every channel
//                    passes a causal convolution over `taps` tokens of its sequence (no bias; the last tap is the token's own;
//                    inputs older than the step come from the sequence's state, its last taps - 1 inputs, oldest first; taps 0:
//                    none).  The first 2 * half numbers of every map of q and k turn by the token's angles (neighbours, or pairs
//                    half the rotated width apart).  A key row of the cache is the two maps side by side (2n numbers); a head's
//                    two queries become rows of that width, each with zeros in the other map's place; values go to the cache.
//                    In a step of one token a sequence the state takes the token's inputs in the same launch.
//  * map_difference: out[t][h] = f * (a - w b) / sqrt(mean((a - w b)^2) + eps), a and b the outputs of the head's two maps.
// Tokens of one sequence are neighbours in the step, so a token's predecessors in it are the rows before it with its slot.
// Everything between the loads and the stores is 32-bit.
#include <math.h>

#include "api.h"
#include "common.cuh"

namespace {

constexpr int MP_TOK = 8;       // tokens a thread of the vector form walks in a prompt step

struct MpArgs {
  void* q;
  long ldq;
  const float* in;
  long ld;
  const float* conv;            // [taps][channels], or null
  float* state;
  long state_ld;
  int state_rows, taps, renew;  // renew: the step brings one token a sequence, whose state is renewed here
  const float2* table;
  int half, adjacent;
  const int *positions, *slots, *block_table;
  int max_pages;
  void *kcache, *vcache;
  int n_tokens, H, G, n, m;
};

__device__ __forceinline__ int mp_rows_before(const int* slots, int t, int most) {
  const int slot = slots[t];
  int q = 0;
  while (q < most && t - q - 1 >= 0 && slots[t - q - 1] == slot) ++q;
  return q;
}

// Where channel c of token t goes: a query's place and the place of its zero, or a place in the cache.
template <typename T>
struct MpPlace {
  T* at;
  T* zero;
};
template <typename T>
__device__ __forceinline__ MpPlace<T> mp_place(const MpArgs& a, int t, int c, int page, int off) {
  const int n2 = 2 * a.n, qd = a.H * n2, kd = a.G * n2;
  MpPlace<T> p;
  p.zero = nullptr;
  if (c < qd) {
    const int h = c / n2, r = c - h * n2, j = r >= a.n ? 1 : 0;          // head, place in [map 1 | map 2], map
    T* base = (T*)a.q + (size_t)t * a.ldq + ((size_t)h * 2 + j) * n2;
    p.at = base + r;
    p.zero = base + (j ? r - a.n : r + a.n);
  } else if (c < qd + kd) {
    const int i = c - qd, g = i / n2;
    p.at = (T*)a.kcache + (((size_t)page * a.G + g) * PAGE_TOKENS + off) * n2 + (i - g * n2);
  } else {
    const int i = c - qd - kd, g = i / a.m;
    p.at = (T*)a.vcache + (((size_t)page * a.G + g) * PAGE_TOKENS + off) * a.m + (i - g * a.m);
  }
  return p;
}

// Any sizes: one block of 256 threads per token, the convolved row in shared memory.
template <typename T>
__global__ void __launch_bounds__(256)
map_prepare_any_kernel(const MpArgs a) {
  extern __shared__ float row[];
  gi::pdl_prologue();
  const int t = blockIdx.x;
  const int n2 = 2 * a.n, qk = (a.H + a.G) * n2, channels = qk + a.G * a.m;
  const int slot = a.slots[t], keep = a.taps - 1;
  const int before = a.taps > 1 ? mp_rows_before(a.slots, t, keep) : 0;
  float* st = a.taps > 1 ? a.state + (size_t)(slot >= 0 ? slot : a.state_rows - 1) * a.state_ld : nullptr;
  for (int c = threadIdx.x; c < channels; c += 256) {
    const float own = a.in[(size_t)t * a.ld + c];
    float v = own;
    if (a.taps > 0) {
      v = 0.f;
      for (int j = 0; j < a.taps; ++j) {
        const int back = keep - j;
        const float u = back == 0 ? own : (back <= before ? a.in[(size_t)(t - back) * a.ld + c] : st[(size_t)(keep - back + before) * channels + c]);
        v = fmaf(a.conv[(size_t)j * channels + c], u, v);
      }
      if (a.renew) {
        for (int j = 0; j + 1 < keep; ++j) st[(size_t)j * channels + c] = st[(size_t)(j + 1) * channels + c];
        if (keep > 0) st[(size_t)(keep - 1) * channels + c] = own;
      }
    }
    row[c] = v;
  }
  __syncthreads();
  const int pos = max(a.positions[t], 0);
  const int page = slot >= 0 ? a.block_table[(size_t)slot * a.max_pages + pos / PAGE_TOKENS] : 0;
  const int off = pos % PAGE_TOKENS, rot = 2 * a.half;
  const float2* cs = a.table + (size_t)t * a.half;
  for (int c = threadIdx.x; c < channels; c += 256) {
    float val = row[c];
    if (c < qk) {
      const int d = c % a.n;
      if (d < rot) {
        float ra, rb;
        if (a.adjacent) {
          const int dl = d & ~1;
          gi::rotate_pair(row[c - d + dl], row[c - d + dl + 1], cs[dl >> 1], &ra, &rb);
          val = (d & 1) ? rb : ra;
        } else {
          const int i = d < a.half ? d : d - a.half;
          gi::rotate_pair(row[c - d + i], row[c - d + i + a.half], cs[i], &ra, &rb);
          val = d < a.half ? ra : rb;
        }
      }
    }
    const MpPlace<T> p = mp_place<T>(a, t, c, page, off);
    gi::stf(p.at, val);
    if (p.zero != nullptr) gi::stf(p.zero, 0.f);
  }
}

// Sizes that are multiples of 4, neighbouring pairs: a thread takes four neighbouring channels of up to `per_block` tokens in
// order and keeps the last taps - 1 inputs in registers, so that a row is read once.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
map_prepare_kernel(const MpArgs a, int per_block) {
  constexpr int KEEP = TAPS > 1 ? TAPS - 1 : 0;
  gi::pdl_launch_dependents();
  const int n2 = 2 * a.n, qk = (a.H + a.G) * n2, channels = qk + a.G * a.m;
  const int c = (blockIdx.y * 128 + threadIdx.x) * 4;
  const bool live = c < channels;
  float4 w[TAPS > 0 ? TAPS : 1];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = live ? gi::ld4(a.conv + (size_t)j * channels + c) : make_float4(0.f, 0.f, 0.f, 0.f);   // no kernel writes the taps
  gi::pdl_wait();
  if (!live) return;
  const int t0 = blockIdx.x * per_block, t1 = min(a.n_tokens, t0 + per_block);
  const int d = c < qk ? c % a.n : a.n;                     // place inside a map (values: past every rotated number)
  const int rot = 2 * a.half;
  float4 past[KEEP > 0 ? KEEP : 1];                         // the inputs before the token, oldest first
  int prev = 0;
  for (int t = t0; t < t1; ++t) {
    const int slot = a.slots[t];
    float* st = KEEP > 0 ? a.state + (size_t)(slot >= 0 ? slot : a.state_rows - 1) * a.state_ld + c : nullptr;
    if (KEEP > 0 && (t == t0 || slot != prev)) {
      const int before = t == t0 ? mp_rows_before(a.slots, t, KEEP) : 0;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int back = KEEP - i;
        past[i] = back <= before ? gi::ld4(a.in + (size_t)(t - back) * a.ld + c)
                                 : *reinterpret_cast<const float4*>(st + (size_t)(i + before) * channels);
      }
    }
    prev = slot;
    const float4 own = gi::ld4(a.in + (size_t)t * a.ld + c);
    float4 v = own;
    if (TAPS > 0) {
      v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const float4 u = j < KEEP ? past[j < KEEP ? j : 0] : own;
        v.x = fmaf(w[j].x, u.x, v.x); v.y = fmaf(w[j].y, u.y, v.y); v.z = fmaf(w[j].z, u.z, v.z); v.w = fmaf(w[j].w, u.w, v.w);
      }
#pragma unroll
      for (int i = 0; i + 1 < KEEP; ++i) past[i] = past[i + 1];
      if (KEEP > 0) past[KEEP > 0 ? KEEP - 1 : 0] = own;
      if (KEEP > 0 && a.renew) {
#pragma unroll
        for (int i = 0; i < KEEP; ++i) *reinterpret_cast<float4*>(st + (size_t)i * channels) = past[i];
      }
    }
    if (d < rot) {
      float ra, rb;
      const float2* cs = a.table + (size_t)t * a.half + (d >> 1);
      gi::rotate_pair(v.x, v.y, cs[0], &ra, &rb);
      v.x = ra; v.y = rb;
      if (d + 2 < rot) {
        gi::rotate_pair(v.z, v.w, cs[1], &ra, &rb);
        v.z = ra; v.w = rb;
      }
    }
    const int pos = max(a.positions[t], 0);
    const int page = slot >= 0 ? a.block_table[(size_t)slot * a.max_pages + pos / PAGE_TOKENS] : 0;
    const MpPlace<T> p = mp_place<T>(a, t, c, page, pos % PAGE_TOKENS);
    gi::st4(p.at, v);
    if (p.zero != nullptr) gi::st4(p.zero, make_float4(0.f, 0.f, 0.f, 0.f));
  }
}

// a warp per token and head; NV: groups of four values a lane holds (0: any width, read twice)
template <typename T, int NV>
__global__ void __launch_bounds__(256)
map_difference_kernel(T* __restrict__ out, const T* in, int heads, int m, float weight, float factor, float eps, unsigned total) {
  gi::pdl_prologue();
  const unsigned i = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= total) return;
  const int lane = threadIdx.x & 31;
  const T* pa = in + (size_t)i * 2 * m;            // rows are [head][map][m]: item i is (token, head)
  const T* pb = pa + m;
  T* o = out + (size_t)i * m;
  float ss = 0.f;
  if (NV > 0) {
    float4 v[NV > 0 ? NV : 1];
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int e = lane * 4 + 128 * j;
      v[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (e < m) {
        const float4 x = gi::ld4(pa + e), y = gi::ld4(pb + e);
        v[j] = make_float4(fmaf(-weight, y.x, x.x), fmaf(-weight, y.y, x.y), fmaf(-weight, y.z, x.z), fmaf(-weight, y.w, x.w));
      }
      ss = fmaf(v[j].x, v[j].x, ss); ss = fmaf(v[j].y, v[j].y, ss); ss = fmaf(v[j].z, v[j].z, ss); ss = fmaf(v[j].w, v[j].w, ss);
    }
    const float r = factor / sqrtf(gi::warp_sum(ss) / (float)m + eps);
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int e = lane * 4 + 128 * j;
      if (e < m) gi::st4(o + e, make_float4(v[j].x * r, v[j].y * r, v[j].z * r, v[j].w * r));
    }
    return;
  }
  for (int e = lane; e < m; e += 32) {
    const float v = fmaf(-weight, gi::ldf(pb + e), gi::ldf(pa + e));
    ss = fmaf(v, v, ss);
  }
  const float r = factor / sqrtf(gi::warp_sum(ss) / (float)m + eps);
  for (int e = lane; e < m; e += 32) gi::stf(o + e, fmaf(-weight, gi::ldf(pb + e), gi::ldf(pa + e)) * r);
}

template <typename T>
cudaError_t mp_launch(const MpArgs& a, int channels, bool vec, cudaStream_t s, int* rc) {
  *rc = GI_OK;
  if (vec) {
    const int per = a.renew ? 1 : MP_TOK;
    const dim3 grid((a.n_tokens + per - 1) / per, (channels / 4 + 127) / 128), block(128);
    switch (a.taps) {
      case 0: return gi::launch(map_prepare_kernel<T, 0>, grid, block, 0, s, a, per);
      case 1: return gi::launch(map_prepare_kernel<T, 1>, grid, block, 0, s, a, per);
      case 2: return gi::launch(map_prepare_kernel<T, 2>, grid, block, 0, s, a, per);
      case 3: return gi::launch(map_prepare_kernel<T, 3>, grid, block, 0, s, a, per);
      default: return gi::launch(map_prepare_kernel<T, 4>, grid, block, 0, s, a, per);
    }
  }
  const size_t smem = (size_t)channels * sizeof(float);
  auto kern = map_prepare_any_kernel<T>;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) {
      *rc = gi::fail(GI_ERR_UNSUPPORTED, "map_prepare: rows of %zu bytes do not fit shared memory", smem);
      return cudaSuccess;
    }
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return gi::launch(kern, dim3(a.n_tokens), dim3(256), smem, s, a);
}

}  // namespace

extern "C" int gi_map_prepare(void* q, long ldq, int dtype, const float* in, long ld, const float* conv, int taps, float* state, long state_ld,
                              int state_rows, int one_token_each, const float* table, int half, int adjacent, const int* positions,
                              const int* slots, const int* block_table, int max_pages, void* kcache, void* vcache, int n_tokens,
                              int heads, int kv_heads, int n, int m, void* stream) {
  if (n_tokens <= 0) return GI_OK;
  if (heads <= 0 || kv_heads <= 0 || n <= 0 || m <= 0 || half < 0 || 2 * half > n || taps < 0)
    return gi::fail(GI_ERR_ARG, "map_prepare: bad sizes (heads %d, kv heads %d, maps of %d, values %d, rotated %d, taps %d)", heads, kv_heads, n, m, 2 * half, taps);
  if (half > 0 && table == nullptr) return gi::fail(GI_ERR_ARG, "map_prepare: rotation without a table of angles");
  if (taps > 0 && conv == nullptr) return gi::fail(GI_ERR_ARG, "map_prepare: a convolution without its taps");
  if (!q || !in || !positions || !slots || !block_table || !kcache || !vcache) return gi::fail(GI_ERR_ARG, "map_prepare: a missing pointer");
  const long channels = (long)(heads + kv_heads) * 2 * n + (long)kv_heads * m;
  if (taps > 1 && (state == nullptr || state_ld < (taps - 1) * channels))
    return gi::fail(GI_ERR_ARG, "map_prepare: state rows of %ld floats, wanted %ld", state_ld, (taps - 1) * channels);
  MpArgs a = {};
  a.q = q; a.ldq = ldq; a.in = in; a.ld = ld; a.conv = conv; a.state = state; a.state_ld = state_ld; a.state_rows = state_rows;
  a.taps = taps; a.renew = one_token_each; a.table = (const float2*)table; a.half = half; a.adjacent = adjacent;
  a.positions = positions; a.slots = slots; a.block_table = block_table; a.max_pages = max_pages; a.kcache = kcache; a.vcache = vcache;
  a.n_tokens = n_tokens; a.H = heads; a.G = kv_heads; a.n = n; a.m = m;
  const size_t wide = dtype == GI_BF16 ? 8 : 16;      // bytes of four numbers as stored
  const bool vec = n % 4 == 0 && m % 4 == 0 && ld % 4 == 0 && ldq % 4 == 0 && (adjacent || half == 0) && taps <= 4 &&
                   (taps <= 1 || (state_ld % 4 == 0 && ((uintptr_t)state & 15) == 0)) &&
                   (((uintptr_t)in | (uintptr_t)conv) & 15) == 0 && (((uintptr_t)q | (uintptr_t)kcache | (uintptr_t)vcache) & (wide - 1)) == 0;
  cudaError_t e = cudaSuccess;
  int rc = GI_OK;
  GI_DISPATCH_DTYPE(dtype, T, e = mp_launch<T>(a, (int)channels, vec, (cudaStream_t)stream, &rc));
  if (rc != GI_OK) return rc;
  return gi::check(e, "map_prepare");
}

extern "C" int gi_map_difference(void* out, const void* in, int dtype, int n_rows, int heads, int m, float weight, float factor, float eps,
                                 void* stream) {
  if (n_rows <= 0) return GI_OK;
  if (heads <= 0 || m <= 0) return gi::fail(GI_ERR_ARG, "map_difference: bad sizes (heads %d, values %d)", heads, m);
  const size_t total = (size_t)n_rows * heads;
  if (total > 0x7fffff00ul) return gi::fail(GI_ERR_UNSUPPORTED, "map_difference: too many rows for one launch");
  const int nv = (m % 4 == 0 && m <= 512 && (((uintptr_t)in | (uintptr_t)out) & 15) == 0) ? (m + 127) / 128 : 0;
  const dim3 grid((unsigned)((total + 7) / 8)), block(256);
  cudaError_t e = cudaSuccess;
  GI_DISPATCH_DTYPE(dtype, T, {
    auto kern = nv == 0 ? map_difference_kernel<T, 0> : (nv == 1 ? map_difference_kernel<T, 1> : (nv == 2 ? map_difference_kernel<T, 2> : map_difference_kernel<T, 4>));
    e = gi::launch(kern, grid, block, 0, (cudaStream_t)stream, (T*)out, (const T*)in, heads, m, weight, factor, eps, (unsigned)total);
  });
  return gi::check(e, "map_difference");
}
