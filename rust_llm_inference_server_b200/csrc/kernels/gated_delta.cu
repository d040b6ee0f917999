// The gated delta rule with one decay a head (see conv_recurrence.cuh).
#include "conv_recurrence.cuh"

// Floats of a request's state slot: S of every head, then the convolution's tail.
extern "C" int rlis_conv_recurrence_state_floats(int nh, int n_qk, int d, int dv, int taps) {
    return convrec::state_floats(nh, n_qk, d, dv, taps);
}

// proj [T, stride] in the element type: q | k | v columns from qkv_off (n_qk heads of d, n_qk of d, nh of dv),
// nh logits of beta from b_off and of the decay from a_off.  conv_w float32 [C, taps] in the same channel order.
// state float32 [slots, state_stride]; act float32 [T, C + 2 nh] (scratch); out float32 [T, nh dv].
// gram: null for the token-by-token kernel (steps of single tokens and short portions), else float32
// [T, n_qk * 32 + nh * 16] of scratch for the kernels that take 16 tokens at a time.
extern "C" int rlis_gated_delta(const void* proj, long long stride, int qkv_off, int b_off, int a_off,
                                const float* conv_w, const float* a_log, const float* dt_bias, float* state,
                                long long state_stride, const int* cu_seqlens, const int* ctx_lens,
                                const int* state_slots, const int* seq_of_token, float* act, float* gram, float* out,
                                int n_tokens, int n_seqs, int nh, int n_qk, int d, int dv, int taps, float unit_eps,
                                float q_scale, int dtype, cudaStream_t stream) {
    const size_t es = dtype == RLIS_F32 ? 4 : 2;
    const char* p = (const char*)proj;
    const convrec::Args g{p + qkv_off * es, p + b_off * es, p + a_off * es, stride, stride, conv_w, nullptr, a_log, dt_bias,
                          nullptr, state, state_stride, {cu_seqlens, ctx_lens, state_slots, seq_of_token}, act, gram, nullptr,
                          out, n_tokens, n_seqs, {nh, n_qk, d, dv, taps, 0, n_qk * d, 2 * n_qk * d}, unit_eps, q_scale};
    return convrec::launch<convrec::HEAD_DECAY>(g, dtype, stream);
}
