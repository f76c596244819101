"""Latent-attention mixer: queries through a normed low-rank latent, keys / values through ONE normed latent per token that
all heads share, plus one rotated key part; sliding-window causal softmax; a sigmoid gate per head on the output.  Options of the
specification (model_config.LatentAttentionSpec): queries projected directly (q_rank = 0), stretched rotary frequencies, a learned
sink per head in the softmax, an element-wise gate (applied after the value up-projection).

Only the latent c [r] and the rotated key part [dr] are cached.  Keys and values are never expanded: with W_uk[h] [dn, r] and
W_uv[h] [dv, r]
    q_nope[h] . (W_uk[h] c_j) = (W_uk[h]^T q_nope[h]) . c_j = q_lat[h] . c_j         (one batched GEMM over heads)
    sum_j p_j (W_uv[h] c_j)   = W_uv[h] (sum_j p_j c_j)    = W_uv[h] out_lat[h]      (one batched GEMM over heads)
so the attention kernel reads each cached row once for all heads.  Op sequence per step:
    fused [dq ; g ; dkv] GEMM -> RMS norm of the query latent -> uq GEMM   (q_rank = 0: ONE [q ; g ; dkv] GEMM) -> (own latent: norm + rotary + cache store, one kernel)
    -> q_lat batched GEMM -> latent attention (rotary of q, window, softmax, gate: one kernel) -> uv batched GEMM
    (-> element-wise gate) -> o GEMM."""
import torch

from swiftllm_b200.worker.kernels.latent_attn import latent_attention, latent_kv_store
from swiftllm_b200.worker.kernels.linear import linear
from swiftllm_b200.worker.kernels.parallel_block import rmsnorm_strided
from swiftllm_b200.worker.kernels.stream_ops import sigmoid_gate_inplace


class LatentAttentionMixer:
    def __init__(self, spec, weight, eps: float, cache_key):
        self.spec, self.weight, self.eps = spec, weight, eps
        self.cache_width, self.cache_slot = cache_key          # which cache tensor and which of its slots this layer uses

    def register(self, model):
        m = self.spec
        model._register_rotary(m.rot_key, m.rot_base, m.rot_dims, m.rot_scaling)

    def state_layout(self) -> dict:
        return {}

    def forward(self, h: torch.Tensor, caches: dict, block_table: torch.Tensor, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        T, H, dn, dr, r = h.shape[0], m.heads, m.dim, m.rot_dim, m.kv_rank
        nq = m.q_rank if m.q_rank > 0 else H * (dn + dr)
        ng = H if m.gate == "head" else H * m.vdim
        proj = linear(h, w.in_proj)                             # [T, q_rank or H (dn + dr) | gate | (r + dr)]
        gate = proj[:, nq:nq + ng]
        if m.q_rank > 0:
            q = linear(rmsnorm_strided(proj[:, :nq], w.dq_norm, self.eps), w.uq).view(T, H, dn + dr)
        else:
            q = proj[:, :nq].unflatten(1, (H, dn + dr))
        out_lat = torch.empty((T, H, r), dtype=h.dtype, device=h.device)
        if st.ignore_kvcache:
            out_lat.zero_()
        else:
            cos, sin = st.rotary[m.rot_key] if m.rot_dims > 0 else (None, None)
            cache = caches[self.cache_width]
            if m.kv_from is None:
                latent_kv_store(proj[:, nq + ng:], w.dkv_norm, cache, self.cache_slot, block_table, st, r, dr, m.rot_dims,
                                self.eps, cos, sin)
            q_lat = torch.empty((T, H, r), dtype=h.dtype, device=h.device)
            torch.bmm(q[:, :, :dn].transpose(0, 1), w.uk, out=q_lat.transpose(0, 1))
            latent_attention(q_lat, q[:, :, dn:], gate if m.gate == "head" else None, cache, self.cache_slot, block_table, st, out_lat,
                             m.rot_dims, m.window, m.scale, cos, sin, w.sink if m.sink else None)
        v = torch.empty((T, H, m.vdim), dtype=h.dtype, device=h.device)
        torch.bmm(out_lat.transpose(0, 1), w.uv.transpose(1, 2), out=v.transpose(0, 1))
        v = v.view(T, H * m.vdim)
        if m.gate == "element":
            sigmoid_gate_inplace(v, gate)
        return linear(v, w.o)
