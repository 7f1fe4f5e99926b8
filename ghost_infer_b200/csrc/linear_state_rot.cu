// Linear attention with constant decays whose queries and keys are rotated by their position ("retention"): the recurrence of
// linear_state.cuh with the rotation on the way in.
#include "linear_state.cuh"

extern "C" int gi_linear_state_rot(float* o, const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, int dtype,
                                   const float* decay, const float* table, int half, int adjacent, float k_scale, float* state,
                                   long state_ld, int state_rows, const int* cu_seqlens, const int* seq_slots, int n_seqs, int heads,
                                   int K, int V, int n_tokens, void* stream) {
  if (n_seqs <= 0) return GI_OK;
  if (half < 0 || 2 * half > K) return gi::fail(GI_ERR_ARG, "linear_state: %d numbers cannot turn in keys of %d", 2 * half, K);
  if (half > 0 && table == nullptr) return gi::fail(GI_ERR_ARG, "linear_state: rotation without a table of angles");
  LsArgs a = {};
  a.o = o; a.q = q; a.k = k; a.v = v;
  a.ldq = ldq; a.ldk = ldk; a.ldv = ldv;
  a.decay_c = decay; a.state = state; a.state_ld = state_ld; a.state_rows = state_rows;
  a.cu_seqlens = cu_seqlens; a.seq_slots = seq_slots;
  a.heads = heads; a.qk_heads = heads; a.K = K; a.V = V;
  a.norm_eps = 0.f; a.q_scale = 1.0f;
  a.table = (const float2*)table; a.half = half; a.adjacent = adjacent; a.k_scale = k_scale;
  return ls_run<true>(a, dtype, n_seqs, 0, n_tokens, stream);
}
