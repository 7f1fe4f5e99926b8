// Linear attention with a matrix of state per head: the entry points of the delta rule, of constant decays and of ready-made
// gates (linear_state.cuh holds the kernel; linear_state_rot.cu the form whose queries and keys turn, linear_state_keyed.cu the one with decays per key).
#include "linear_state.cuh"

extern "C" int gi_linear_state(float* o, const void* q, long ldq, const void* k, long ldk, const void* v, long ldv,
                               const void* a_in, long lda, const void* b_in, long ldb, int dtype, const float* decay_c,
                               const float* dt_bias, float* state, long state_ld, int state_rows, const int* cu_seqlens,
                               const int* seq_slots, int n_seqs, int heads, int qk_heads, int K, int V, int in_act,
                               int unit_norm, float norm_eps, float q_scale, int delta, int n_tokens, void* stream) {
  return gi_linear_state_gated(o, q, ldq, k, ldk, v, ldv, a_in, lda, b_in, ldb, dtype, decay_c, dt_bias, nullptr, nullptr, state,
                               state_ld, state_rows, cu_seqlens, seq_slots, n_seqs, heads, qk_heads, K, V, in_act, unit_norm,
                               norm_eps, q_scale, delta, n_tokens, stream);
}

extern "C" int gi_linear_state_gated(float* o, const void* q, long ldq, const void* k, long ldk, const void* v, long ldv,
                                     const void* a_in, long lda, const void* b_in, long ldb, int dtype, const float* decay_c,
                                     const float* dt_bias, const float* g_direct, const float* u_direct, float* state,
                                     long state_ld, int state_rows, const int* cu_seqlens, const int* seq_slots, int n_seqs,
                                     int heads, int qk_heads, int K, int V, int in_act, int unit_norm, float norm_eps,
                                     float q_scale, int delta, int n_tokens, void* stream) {
  if (n_seqs <= 0) return GI_OK;
  if (u_direct != nullptr && delta) return gi::fail(GI_ERR_ARG, "linear_state: ready-made write strengths do not go with the delta rule");
  if (delta && b_in == nullptr) return gi::fail(GI_ERR_ARG, "linear_state: the delta rule needs its write strengths");
  LsArgs a = {};
  a.o = o; a.q = q; a.k = k; a.v = v; a.a_in = a_in; a.b_in = b_in;
  a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.lda = lda; a.ldb = ldb;
  a.decay_c = decay_c; a.dt_bias = dt_bias; a.g_direct = g_direct; a.u_direct = u_direct; a.state = state; a.state_ld = state_ld; a.state_rows = state_rows;
  a.cu_seqlens = cu_seqlens; a.seq_slots = seq_slots;
  a.heads = heads; a.qk_heads = qk_heads; a.K = K; a.V = V; a.in_act = in_act; a.unit_norm = unit_norm;
  a.norm_eps = norm_eps; a.q_scale = q_scale; a.k_scale = 1.0f;
  return ls_run<false>(a, dtype, n_seqs, delta, n_tokens, stream);
}
