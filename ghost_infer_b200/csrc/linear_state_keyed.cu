// Linear attention whose state decays by a number per token and key channel ("gated linear attention"): the recurrence of
// linear_state.cuh in that form, and the kernel that makes the decays.
//
//  * key_decays:  g[t][c] = sigmoid(z)^(1 / tau), z = sum_r low[t][r] up[r][c] + b[c]: the second of two matrices, its bias and
//                 the root in one pass, 32-bit (low: rows of the projection in the activation type).
#include "linear_state.cuh"

namespace {

constexpr int KD_TOK = 8;      // tokens per block
constexpr int KD_RANK = 64;    // numbers of a row in shared memory at a time
constexpr int KD_AHEAD = 16;   // numbers of a column of the matrix asked for at the start
static_assert(KD_TOK == 8 && KD_AHEAD <= KD_RANK, "a row of the buffer is two groups of four tokens");

// sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau).  The 16-bit path takes exponential and logarithm by the approximate instructions
// and log(1 + e) for small e by its series, so that softplus stays within about 1e-7, which is all a decay near 1 can feel.
template <bool QUICK>
__device__ __forceinline__ float kd_decay(float z, float inv_tau) {
  if (!QUICK) return expf(-inv_tau * ls_softplus(-z));
  const float e = __expf(-z);
  const float small = e * fmaf(e, fmaf(e, 1.0f / 3.0f, -0.5f), 1.0f);
  const float sp = z < -20.f ? -z : (e < 0.005f ? small : __logf(1.0f + e));
  return __expf(-inv_tau * sp);
}

// grid (token tiles, channel tiles): a thread takes one channel of eight tokens
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS)
key_decays_kernel(float* __restrict__ g, const T* low, long ldl, const float* __restrict__ up, const float* __restrict__ b, int n_tokens,
                  int rank, int channels, float inv_tau) {
  __shared__ __align__(16) float sl[KD_RANK][KD_TOK];
  gi::pdl_launch_dependents();
  const int t0 = blockIdx.x * KD_TOK, n = min(KD_TOK, n_tokens - t0);
  const int c = blockIdx.y * THREADS + threadIdx.x;
  const bool live = c < channels;
  // the matrix and the bias are written by no kernel: their first numbers are asked for before the dependency wait
  float u[KD_AHEAD];
#pragma unroll
  for (int r = 0; r < KD_AHEAD; ++r) u[r] = (live && r < rank) ? up[(size_t)r * channels + c] : 0.f;
  const float bias = live ? b[c] : 0.f;
  gi::pdl_wait();
  float z[KD_TOK];
#pragma unroll
  for (int t = 0; t < KD_TOK; ++t) z[t] = bias;
  auto add = [&](int r, float w) {
    const float4 x = *reinterpret_cast<const float4*>(&sl[r][0]), y = *reinterpret_cast<const float4*>(&sl[r][4]);
    z[0] = fmaf(x.x, w, z[0]); z[1] = fmaf(x.y, w, z[1]); z[2] = fmaf(x.z, w, z[2]); z[3] = fmaf(x.w, w, z[3]);
    z[4] = fmaf(y.x, w, z[4]); z[5] = fmaf(y.y, w, z[5]); z[6] = fmaf(y.z, w, z[6]); z[7] = fmaf(y.w, w, z[7]);
  };
  for (int r0 = 0; r0 < rank; r0 += KD_RANK) {
    const int nr = min(KD_RANK, rank - r0), padded = max(nr, KD_AHEAD);
    __syncthreads();
    for (int i = threadIdx.x; i < KD_TOK * padded; i += THREADS) {
      const int t = i / padded, r = i - t * padded;
      sl[r][t] = (t < n && r < nr) ? gi::ldf(low + (size_t)(t0 + t) * ldl + r0 + r) : 0.f;
    }
    __syncthreads();
    if (!live) continue;
    int r = 0;
    if (r0 == 0) {
#pragma unroll
      for (int k = 0; k < KD_AHEAD; ++k) add(k, u[k]);      // past the rank: zeros on both sides
      r = KD_AHEAD;
    }
    for (; r < nr; ++r) add(r, up[(size_t)(r0 + r) * channels + c]);
  }
  if (!live) return;
#pragma unroll
  for (int t = 0; t < KD_TOK; ++t)
    if (t < n) g[(size_t)(t0 + t) * channels + c] = kd_decay<sizeof(T) == 2>(z[t], inv_tau);
}

}  // namespace

extern "C" int gi_key_decays(float* g, const void* low, long ldl, int dtype, const float* up, const float* b, int n_tokens, int rank, int channels,
                             float tau, void* stream) {
  if (n_tokens <= 0) return GI_OK;
  if (rank <= 0 || channels <= 0 || !(tau > 0.f)) return gi::fail(GI_ERR_ARG, "key_decays: bad sizes (rank %d, channels %d, tau %g)", rank, channels, tau);
  if (!g || !low || !up || !b) return gi::fail(GI_ERR_ARG, "key_decays: a missing pointer");
  // few tokens: narrower blocks, so that more SMs take part
  const bool few = n_tokens <= 64;
  const int threads = few ? 64 : 256;
  const dim3 grid((n_tokens + KD_TOK - 1) / KD_TOK, (channels + threads - 1) / threads);
  if (grid.y > 65535) return gi::fail(GI_ERR_UNSUPPORTED, "key_decays: too many channels");
  cudaError_t e = cudaSuccess;
  GI_DISPATCH_DTYPE(dtype, T,
      e = few ? gi::launch(key_decays_kernel<T, 64>, grid, dim3(threads), 0, (cudaStream_t)stream, g, (const T*)low, ldl, up, b, n_tokens, rank, channels, 1.0f / tau)
              : gi::launch(key_decays_kernel<T, 256>, grid, dim3(threads), 0, (cudaStream_t)stream, g, (const T*)low, ldl, up, b, n_tokens, rank, channels, 1.0f / tau));
  return gi::check(e, "key_decays");
}

extern "C" int gi_linear_state_keyed(float* o, const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, int dtype,
                                     const float* decay, float q_scale, float* state, long state_ld, int state_rows,
                                     const int* cu_seqlens, const int* seq_slots, int n_seqs, int heads, int K, int V, int n_tokens,
                                     void* stream) {
  if (n_seqs <= 0) return GI_OK;
  if (decay == nullptr || ((uintptr_t)decay & 15)) return gi::fail(GI_ERR_ARG, "linear_state: the decays per key must start on a 16-byte boundary");
  LsArgs a = {};
  a.o = o; a.q = q; a.k = k; a.v = v;
  a.ldq = ldq; a.ldk = ldk; a.ldv = ldv;
  a.g_key = decay; a.state = state; a.state_ld = state_ld; a.state_rows = state_rows;
  a.cu_seqlens = cu_seqlens; a.seq_slots = seq_slots;
  a.heads = heads; a.qk_heads = heads; a.K = K; a.V = V;
  a.q_scale = q_scale; a.k_scale = 1.0f;
  return ls_run<false, true>(a, dtype, n_seqs, 0, n_tokens, stream);
}
