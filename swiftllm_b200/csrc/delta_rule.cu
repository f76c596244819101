// Gated delta rule with one decay per head (head_decay.cuh, DELTA).
#include "head_decay.cuh"

using namespace sllm;

extern "C" int sllm_delta_rule(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride,
                               const void* decay_logits, int64_t decay_stride, const void* beta_logits, int64_t beta_stride,
                               const void* decay_bias, const void* rate, float q_scale, const void* norm_w, float eps,
                               const void* gate, int64_t gate_stride, void* state, const void* seg_starts, const void* seq_ids,
                               const void* tok_pos, void* workspace, int64_t workspace_floats, void* out, int64_t out_stride,
                               int64_t num_tokens, int64_t num_prefill_tokens, int num_segs, int num_prefill_segs, int num_heads,
                               int num_kv_heads, int dk, int dv, sllm_dtype_t dtype, sllm_stream_t stream) {
    HeadDecayArgs a{};
    a.q = q; a.k = k; a.v = v; a.gate = gate;
    a.q_stride = q_stride; a.k_stride = k_stride; a.v_stride = v_stride; a.gate_stride = gate_stride;
    a.ga = (const float*)decay_logits; a.ga_stride = decay_stride; a.gb = (const float*)beta_logits; a.gb_stride = beta_stride;
    a.pa = (const float*)decay_bias; a.pb = (const float*)rate; a.cap = 1.f; a.q_scale = q_scale; a.eps = eps;
    a.norm_w = (const float*)norm_w; a.norm_step = 0; a.state = (float*)state;
    a.seg_starts = (const int*)seg_starts; a.seq_ids = (const int*)seq_ids; a.tok_pos = (const int*)tok_pos;
    a.o_raw = (float*)workspace; a.out = out; a.out_stride = out_stride;
    a.num_segs = num_segs; a.H = num_heads; a.G = num_kv_heads; a.dk = dk; a.dv = dv;
    return hd_run<true>(a, dtype, num_tokens, num_prefill_tokens, num_prefill_segs, workspace_floats, (cudaStream_t)stream);
}
