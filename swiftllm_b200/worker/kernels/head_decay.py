"""Recurrences with a matrix state per head and ONE decay per head and token (csrc/head_decay.cuh): the gated delta rule and the matrix
memory with exponential input gate.  State tensors have one row per SEQUENCE (the sequence's block-table row), fp32; a step's rows are
segments of consecutive positions (infer_state.seg_starts / seq_ids), prompt portions first; a segment that starts at position 0
starts from the zero state, whatever its row still holds."""
import torch

from swiftllm_b200 import _lib


def _stride0(x: torch.Tensor) -> int:
    return x.stride(0) if x.shape[0] > 1 else max(x.stride(0), x.shape[1])


def _check(q, k, v, gate, za, zb, state, heads, kv_heads, dk, dv):
    T = q.shape[0]
    assert q.stride(1) == k.stride(1) == v.stride(1) == gate.stride(1) == za.stride(1) == zb.stride(1) == 1
    assert q.shape == k.shape == (T, kv_heads * dk) and v.shape == gate.shape == (T, heads * dv) and za.shape == zb.shape == (T, heads)
    assert q.dtype == k.dtype == v.dtype == gate.dtype and za.dtype == zb.dtype == state.dtype == torch.float32
    assert state.is_contiguous() and state.shape[1:] == (heads, dk, dv)
    _lib.require_device(q)


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay_logits: torch.Tensor, beta_logits: torch.Tensor,
               decay_bias: torch.Tensor, rate: torch.Tensor, norm_w: torch.Tensor, eps: float, gate: torch.Tensor, state: torch.Tensor,
               infer_state, heads: int, kv_heads: int, dk: int, dv: int) -> torch.Tensor:
    """q, k [T, G * dk], v, gate [T, H * dv] (column slices are fine); decay_logits, beta_logits fp32 [T, H]; decay_bias, rate fp32 [H];
    norm_w fp32 [dv]; state fp32 [rows, H, dk, dv] (moves on) -> [T, H * dv] = rms-normed heads * norm_w * silu(gate).  g = exp(-rate
    softplus(decay_logits + bias)), beta = sigmoid(beta_logits); q and k become unit vectors per head, q also times dk^-1/2."""
    _check(q, k, v, gate, decay_logits, beta_logits, state, heads, kv_heads, dk, dv)
    assert decay_bias.dtype == rate.dtype == norm_w.dtype == torch.float32 and decay_bias.shape == rate.shape == (heads,) and norm_w.shape == (dv,)
    st, T = infer_state, q.shape[0]
    out = torch.empty((T, heads * dv), dtype=q.dtype, device=q.device)
    size = st.num_prefill_tokens * heads * dv
    ws = torch.empty((size,), dtype=torch.float32, device=q.device)
    _lib.check(_lib.lib().sllm_delta_rule(
        q.data_ptr(), _stride0(q), k.data_ptr(), _stride0(k), v.data_ptr(), _stride0(v), decay_logits.data_ptr(), _stride0(decay_logits),
        beta_logits.data_ptr(), _stride0(beta_logits), decay_bias.data_ptr(), rate.data_ptr(), dk ** -0.5, norm_w.data_ptr(), eps,
        gate.data_ptr(), _stride0(gate), state.data_ptr(), st.seg_starts.data_ptr(), st.seq_ids.data_ptr(), st.token_positions.data_ptr(),
        ws.data_ptr(), size, out.data_ptr(), heads * dv, T, st.num_prefill_tokens, st.batch_size, st.num_prefill_seqs, heads, kv_heads,
        dk, dv, _lib.dtype_tag_f32(q.dtype), _lib.stream()), "delta_rule")
    return out


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, forget_logits: torch.Tensor, input_logits: torch.Tensor,
                  forget_bias: torch.Tensor, input_bias: torch.Tensor, gate_cap: float, norm_w: torch.Tensor, eps: float,
                  gate: torch.Tensor, state: torch.Tensor, norm_state: torch.Tensor, max_state: torch.Tensor, infer_state, heads: int,
                  dk: int, dv: int) -> torch.Tensor:
    """q, k [T, H * dk], v, gate [T, H * dv] (column slices are fine); gate logits fp32 [T, H], their biases fp32 [H]; norm_w fp32
    [H * dv]; state fp32 [rows, H, dk, dv], norm_state fp32 [rows, H, dk], max_state fp32 [rows, H] (all move on) -> [T, H * dv] =
    rms-normed heads * norm_w * sigmoid(gate).  Queries are scaled by dk^-1/2."""
    _check(q, k, v, gate, forget_logits, input_logits, state, heads, heads, dk, dv)
    assert forget_bias.dtype == input_bias.dtype == norm_w.dtype == norm_state.dtype == max_state.dtype == torch.float32
    assert forget_bias.shape == input_bias.shape == (heads,) and norm_w.shape == (heads * dv,) and norm_state.is_contiguous()
    assert norm_state.shape == (state.shape[0], heads, dk) and max_state.is_contiguous() and max_state.shape == (state.shape[0], heads)
    st, T = infer_state, q.shape[0]
    out = torch.empty((T, heads * dv), dtype=q.dtype, device=q.device)
    size = st.num_prefill_tokens * heads * dv + st.num_prefill_seqs * heads * (dk + 1)
    ws = torch.empty((size,), dtype=torch.float32, device=q.device)
    _lib.check(_lib.lib().sllm_matrix_memory(
        q.data_ptr(), _stride0(q), k.data_ptr(), _stride0(k), v.data_ptr(), _stride0(v), forget_logits.data_ptr(), _stride0(forget_logits),
        input_logits.data_ptr(), _stride0(input_logits), forget_bias.data_ptr(), input_bias.data_ptr(), gate_cap, dk ** -0.5,
        norm_w.data_ptr(), eps, gate.data_ptr(), _stride0(gate), state.data_ptr(), norm_state.data_ptr(), max_state.data_ptr(),
        st.seg_starts.data_ptr(), st.seq_ids.data_ptr(), st.token_positions.data_ptr(), ws.data_ptr(), size, out.data_ptr(), heads * dv,
        T, st.num_prefill_tokens, st.batch_size, st.num_prefill_seqs, heads, dk, dv, _lib.dtype_tag_f32(q.dtype), _lib.stream()),
        "matrix_memory")
    return out
