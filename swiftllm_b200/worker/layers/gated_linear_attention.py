"""Gated linear attention mixer with per-sequence state: ONE fused GEMM [q ; k ; v ; gate ; a1] on the block's input -> the second
factor of the decay projection (fp32 output) -> decays + recurrence + read-out + head norm + SiLU gate (csrc/gla.cu, state in the
sequence's state row, fp32) -> o GEMM."""
import torch

from swiftllm_b200.worker.kernels.gla import gated_linear_attention
from swiftllm_b200.worker.kernels.linear import linear, linear_f32_out


class GatedLinearAttentionMixer:
    def __init__(self, spec, weight, eps: float, layer_id: int):
        self.spec, self.weight, self.eps = spec, weight, eps
        self.state_name = f"l{layer_id}.gla"

    def register(self, model):
        pass

    def state_layout(self) -> dict:
        m = self.spec
        return {self.state_name: ((m.heads, m.dim, m.vdim), torch.float32)}

    def forward(self, h: torch.Tensor, caches: dict, block_table: torch.Tensor, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        nk, nv = m.heads * m.dim, m.heads * m.vdim
        q, k, v, gate, low = torch.split(linear(h, w.in_proj), [nk, nk, nv, nv, w.a2.shape[1]], dim=1)
        if st.ignore_kvcache:
            return linear(torch.zeros((h.shape[0], nv), dtype=h.dtype, device=h.device), w.o)
        z = linear_f32_out(low, w.a2)
        y = gated_linear_attention(q, k, v, z, w.a2_bias, m.tau, w.head_norm, self.eps, gate, states[self.state_name], st, m.heads,
                                   m.dim, m.vdim)
        return linear(y, w.o)
