// Matrix memory with exponential input gate, normaliser and running maximum (head_decay.cuh, memory).
#include "head_decay.cuh"

using namespace sllm;

extern "C" int sllm_matrix_memory(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride,
                                  const void* forget_logits, int64_t forget_stride, const void* input_logits, int64_t input_stride,
                                  const void* forget_bias, const void* input_bias, float gate_cap, float q_scale, const void* norm_w,
                                  float eps, const void* gate, int64_t gate_stride, void* state, void* norm_state, void* max_state,
                                  const void* seg_starts, const void* seq_ids, const void* tok_pos, void* workspace,
                                  int64_t workspace_floats, void* out, int64_t out_stride, int64_t num_tokens,
                                  int64_t num_prefill_tokens, int num_segs, int num_prefill_segs, int num_heads, int dk, int dv,
                                  sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(gate_cap > 0.f, "matrix_memory: the gate cap must be positive");
    HeadDecayArgs a{};
    a.q = q; a.k = k; a.v = v; a.gate = gate;
    a.q_stride = q_stride; a.k_stride = k_stride; a.v_stride = v_stride; a.gate_stride = gate_stride;
    a.ga = (const float*)forget_logits; a.ga_stride = forget_stride; a.gb = (const float*)input_logits; a.gb_stride = input_stride;
    a.pa = (const float*)forget_bias; a.pb = (const float*)input_bias; a.cap = gate_cap; a.q_scale = q_scale; a.eps = eps;
    a.norm_w = (const float*)norm_w; a.norm_step = dv; a.state = (float*)state; a.nstate = (float*)norm_state; a.mstate = (float*)max_state;
    a.seg_starts = (const int*)seg_starts; a.seq_ids = (const int*)seq_ids; a.tok_pos = (const int*)tok_pos;
    a.o_raw = (float*)workspace; a.out = out; a.out_stride = out_stride;
    a.num_segs = num_segs; a.H = num_heads; a.G = num_heads; a.dk = dk; a.dv = dv;
    return hd_run<false>(a, dtype, num_tokens, num_prefill_tokens, num_prefill_segs, workspace_floats, (cudaStream_t)stream);
}
