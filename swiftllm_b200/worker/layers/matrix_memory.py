"""Matrix memory mixer (mLSTM) with per-sequence state: ONE fused GEMM [q ; k ; v ; gate] and ONE small GEMM with an fp32 result
[forget ; input] on the block's input -> capped gates with their running maximum, recurrence of memory and normaliser, read-out, head
norm, sigmoid gate (csrc/matrix_memory.cu, fp32 state) -> o GEMM."""
import torch

from swiftllm_b200.worker.kernels.head_decay import matrix_memory
from swiftllm_b200.worker.kernels.linear import linear, linear_f32_out


class MatrixMemoryMixer:
    def __init__(self, spec, weight, eps: float, layer_id: int):
        self.spec, self.weight, self.eps = spec, weight, eps
        self.names = tuple(f"l{layer_id}.memory{part}" for part in ("", "_norm", "_max"))

    def register(self, model):
        pass

    def state_layout(self) -> dict:
        m = self.spec
        return dict(zip(self.names, (((m.heads, m.dim, m.vdim), torch.float32), ((m.heads, m.dim), torch.float32),
                                     ((m.heads,), torch.float32))))

    def forward(self, h: torch.Tensor, caches, block_table, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        nk, nv = m.heads * m.dim, m.heads * m.vdim
        q, k, v, gate = torch.split(linear(h, w.in_proj), [nk, nk, nv, nv], dim=1)
        if st.ignore_kvcache:
            return linear(torch.zeros((h.shape[0], nv), dtype=h.dtype, device=h.device), w.o)
        z = linear_f32_out(h, w.gate_proj)                                  # fp32 [T, forget | input]
        y = matrix_memory(q, k, v, z[:, :m.heads], z[:, m.heads:], w.forget_bias, w.input_bias, m.gate_cap, w.head_norm, self.eps, gate,
                          *(states[n] for n in self.names), st, m.heads, m.dim, m.vdim)
        return linear(y, w.o)
