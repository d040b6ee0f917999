// The gated delta rule with one decay a head and key channel (see conv_recurrence.cuh).
#include "conv_recurrence.cuh"

// As rlis_gated_delta, with the decay logits [T, a_stride] in rows of their own (nh heads of d from a_off) and dt_bias
// float32 [nh d].  act float32 [T, C + nh + nh d]; gram null (token by token) or float32 [T, nh * 48], with scaled float32
// [T, nh, 4 d].
extern "C" int rlis_channel_delta(const void* proj, long long stride, int qkv_off, int b_off, const void* decay,
                                  long long a_stride, int a_off, const float* conv_w, const float* a_log,
                                  const float* dt_bias, float* state, long long state_stride, const int* cu_seqlens,
                                  const int* ctx_lens, const int* state_slots, const int* seq_of_token, float* act,
                                  float* gram, float* scaled, float* out, int n_tokens, int n_seqs, int nh, int n_qk, int d,
                                  int dv, int taps, float unit_eps, float q_scale, int dtype, cudaStream_t stream) {
    const size_t es = dtype == RLIS_F32 ? 4 : 2;
    const char* p = (const char*)proj;
    const convrec::Args g{p + qkv_off * es, p + b_off * es, (const char*)decay + a_off * es, stride, a_stride, conv_w, nullptr,
                          a_log, dt_bias, nullptr, state, state_stride, {cu_seqlens, ctx_lens, state_slots, seq_of_token}, act,
                          gram, scaled, out, n_tokens, n_seqs, {nh, n_qk, d, dv, taps, 0, n_qk * d, 2 * n_qk * d}, unit_eps,
                          q_scale};
    return convrec::launch<convrec::CHANNEL_DECAY>(g, dtype, stream);
}
