"""Gated linear attention with a decay per key channel and token (csrc/gla.cu).  Its state is one row per SEQUENCE (the sequence's
block-table row) of an fp32 tensor; a step's rows are segments of consecutive positions (infer_state.seg_starts / seq_ids); a
segment that starts at position 0 starts from the zero state, whatever its row still holds."""
import torch

from swiftllm_b200 import _lib


def _stride0(x: torch.Tensor) -> int:
    return x.stride(0) if x.shape[0] > 1 else max(x.stride(0), x.shape[1])


def gated_linear_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, z: torch.Tensor, bias: torch.Tensor, tau: float,
                           norm_w: torch.Tensor, eps: float, gate: torch.Tensor, state: torch.Tensor, infer_state, heads: int,
                           dk: int, dv: int) -> torch.Tensor:
    """q, k [T, H * dk], v, gate [T, H * dv] as projected (column slices are fine); z fp32 [T, H * dk], bias fp32 [H * dk]: decay
    logits; norm_w fp32 [dv]; state fp32 [rows, H, dk, dv] (moves on) -> [T, H * dv] = rms-normed heads * norm_w * silu(gate), ready
    for the output projection.  alpha = sigmoid(z + bias)^(1 / tau); queries are scaled by dk^-1/2."""
    T = q.shape[0]
    assert q.stride(1) == k.stride(1) == v.stride(1) == gate.stride(1) == z.stride(1) == 1
    assert q.shape == k.shape == z.shape == (T, heads * dk) and v.shape == gate.shape == (T, heads * dv)
    assert q.dtype == k.dtype == v.dtype == gate.dtype and z.dtype == bias.dtype == norm_w.dtype == state.dtype == torch.float32
    assert bias.shape == (heads * dk,) and norm_w.shape == (dv,) and state.is_contiguous() and state.shape[1:] == (heads, dk, dv)
    _lib.require_device(q)
    st = infer_state
    out = torch.empty((T, heads * dv), dtype=q.dtype, device=q.device)
    nseg, npre = st.num_prefill_seqs, st.num_prefill_tokens
    longest = min(npre, st.max_prefill_len)
    size = _lib.lib().sllm_gla_workspace_floats(T, nseg, longest, heads, dk, dv)
    ws = torch.empty((size,), dtype=torch.float32, device=q.device)
    _lib.check(_lib.lib().sllm_gla(
        q.data_ptr(), _stride0(q), k.data_ptr(), _stride0(k), v.data_ptr(), _stride0(v), z.data_ptr(), _stride0(z), bias.data_ptr(),
        1.0 / tau, dk ** -0.5, norm_w.data_ptr(), eps, gate.data_ptr(), _stride0(gate), state.data_ptr(), st.seg_starts.data_ptr(),
        st.seq_ids.data_ptr(), st.token_positions.data_ptr(), ws.data_ptr(), size, out.data_ptr(), heads * dv, T, npre, st.batch_size,
        nseg, longest, heads, dk, dv, _lib.dtype_tag_f32(q.dtype), _lib.stream()), "gla")
    return out
