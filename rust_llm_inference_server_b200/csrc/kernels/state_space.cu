// The state-space dual form of Mamba-2 (see conv_recurrence.cuh).
#include "conv_recurrence.cuh"

// proj [T, stride] in the element type: x | B | C columns from conv_off (nh heads of dv, then groups of n twice), nh logits
// of the step size from dt_off.  conv_w float32 [nh dv + 2 groups n, taps] and conv_b (one a channel, or null) in the same
// order; a_log, dt_bias, skip float32 [nh].  state float32 [slots, state_stride]: S [nh, dv, n] and the convolution's tail.
// act float32 [T, channels + 2 nh]; gram null (token by token) or float32 [T, groups * 32]; out float32 [T, nh dv].
extern "C" int rlis_state_space(const void* proj, long long stride, int conv_off, int dt_off, const float* conv_w,
                                const float* conv_b, const float* a_log, const float* dt_bias, const float* skip, float* state,
                                long long state_stride, const int* cu_seqlens, const int* ctx_lens, const int* state_slots,
                                const int* seq_of_token, float* act, float* gram, float* out, int n_tokens, int n_seqs, int nh,
                                int groups, int n, int dv, int taps, int dtype, cudaStream_t stream) {
    const size_t es = dtype == RLIS_F32 ? 4 : 2;
    const char* p = (const char*)proj;
    const int inner = nh * dv;
    const convrec::Args g{p + conv_off * es, p + dt_off * es, nullptr, stride, 0, conv_w, conv_b, a_log, dt_bias, skip, state,
                          state_stride, {cu_seqlens, ctx_lens, state_slots, seq_of_token}, act, gram, nullptr, out, n_tokens,
                          n_seqs, {nh, groups, n, dv, taps, inner + groups * n, inner, 0}, 0.f, 1.f};
    return convrec::launch<convrec::STATE_SPACE>(g, dtype, stream);
}
