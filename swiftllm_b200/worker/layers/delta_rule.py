"""Gated delta rule mixer with per-sequence state: ONE fused GEMM [q ; k ; v ; gate] and ONE small GEMM with an fp32 result [beta ; decay] on
the block's input -> causal convolution with SiLU over q, k and v together (its last taps - 1 inputs are per-sequence state) -> unit
queries and keys, decays, recurrence, read-out, head norm, SiLU gate (csrc/delta_rule.cu, fp32 state) -> o GEMM."""
import torch

from swiftllm_b200.worker.kernels.head_decay import delta_rule
from swiftllm_b200.worker.kernels.linear import linear, linear_f32_out
from swiftllm_b200.worker.kernels.scan_ops import short_conv


class GatedDeltaRuleMixer:
    def __init__(self, spec, weight, eps: float, layer_id: int):
        self.spec, self.weight, self.eps = spec, weight, eps
        self.state_name, self.tail_name = f"l{layer_id}.delta", f"l{layer_id}.delta_conv_tail"

    def register(self, model):
        pass

    def state_layout(self) -> dict:
        m = self.spec
        out = {self.state_name: ((m.heads, m.dim, m.vdim), torch.float32)}
        if m.conv > 1:
            out[self.tail_name] = ((m.conv - 1, m.conv_channels), self.weight.dtype)
        return out

    def forward(self, h: torch.Tensor, caches, block_table, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        nk, nv = m.kv_heads * m.dim, m.heads * m.vdim
        proj = linear(h, w.in_proj)                                         # [T, q | k | v | gate]
        qkv, gate = proj[:, :m.conv_channels], proj[:, m.conv_channels:]
        if st.ignore_kvcache:
            return linear(torch.zeros((h.shape[0], nv), dtype=h.dtype, device=h.device), w.o)
        z = linear_f32_out(h, w.gate_proj)                                  # fp32 [T, beta | decay]
        tail = states[self.tail_name] if m.conv > 1 else None
        x = short_conv(qkv, w.conv, None, tail, st, h.dtype, silu=True, move_tail=True)
        q, k, v = torch.split(x, [nk, nk, nv], dim=1)
        y = delta_rule(q, k, v, z[:, m.heads:], z[:, :m.heads], w.decay_bias, w.rate, w.head_norm, self.eps, gate,
                       states[self.state_name], st, m.heads, m.kv_heads, m.dim, m.vdim)
        return linear(y, w.o)
