"""Softmax attention mixer with grouped key/value heads over the paged cache: ONE fused GEMM [q ; k ; v (; gate)] on the block's
input -> (rotary of k + cache store, one kernel) -> attention (rotary of q, window, softmax with an optional sink, optional
sigmoid output gate: one kernel) -> o GEMM.  The specification's options (model_config.WindowAttentionSpec: rotary pairs as
halves, stretched frequencies, unit-RMS queries and keys, capped scores, values turned by their position) go to the same two
kernels.  `attend` is the part between the two GEMMs, for mixers that fuse their projections with a neighbour's.

`SharedKeyValueAttentionMixer`: the values are the keys as projected, so there is ONE fused GEMM with bias [q ; k ; gate per head],
the cache holds the un-normed keys with their 1 / rms, and one staged tile serves the attention kernel as keys and values; scores
carry a bias on the distance; the first positions of the sequence stay visible beside the window.

`WholeNormAttentionMixer`: values that are the keys as projected, again, but queries and keys are normed over their whole projection and
turn on a part of every head; the cache row holds the un-normed keys, their 1 / rms and the turned entries; a learned sink per head.

`DifferentialAttentionMixer`: two score maps per head over the same values.  Every map is a query head of its own for the same two
kernels (twice the heads, `vshare` = 2 key heads per value head, fp32 output); one more kernel subtracts the maps, normalises
the head and applies the gate."""
import torch

from swiftllm_b200.worker.kernels.linear import linear, linear_bias
from swiftllm_b200.worker.kernels.window_attn import (AttnOptions, diff_combine, shared_kv_store, whole_norm_rope_store,
                                                      window_attention, window_kv_store)


class WindowAttentionMixer:
    def __init__(self, spec, weight, eps: float, cache_key):
        self.spec, self.weight = spec, weight
        self.cache_width, self.cache_slot = cache_key          # which cache tensor and which of its slots this layer uses
        self.options = AttnOptions(pair_halves=spec.pair_halves, qk_norm_eps=eps if spec.qk_unit_norm else -1.0,
                                   softcap=spec.softcap, out_scale=spec.out_scale)

    def register(self, model):
        m = self.spec
        model._register_rotary(m.rot_key, m.rot_base, m.rot_dims, m.rot_scaling)
        if m.value_rotation:
            model._register_rotary(m.vrot_key, m.rot_base, m.vdim)

    @property
    def proj_widths(self):
        """Columns of the fused input projection: q, k, v (, gate)."""
        m = self.spec
        return [m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim] + ([m.heads * m.vdim] if m.gate else [])

    def attend(self, q, k, v, gate, out, caches: dict, block_table, st):
        """q [T, H dk], k [T, G dk], v [T, G dv], gate [T, H dv] or None (column slices of a wider matrix are fine) -> out [T, H dv]."""
        m = self.spec
        if st.ignore_kvcache:
            out.zero_()
            return
        cos, sin = st.rotary[m.rot_key] if m.rot_dims > 0 else (None, None)
        vcos, vsin = st.rotary[m.vrot_key] if m.value_rotation else (None, None)
        cache = caches[self.cache_width]
        window_kv_store(k, v, cache, self.cache_slot, block_table, st, m.kv_heads, m.dim, m.vdim, m.rot_dims, cos, sin,
                        self.options, vcos, vsin)
        window_attention(q, gate, cache, self.cache_slot, block_table, st, out, m.heads, m.kv_heads, m.dim, m.vdim,
                         m.rot_dims, m.window, m.scale, m.sink, cos, sin, self.options, vcos, vsin)

    def forward(self, h: torch.Tensor, caches: dict, block_table: torch.Tensor, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        proj = linear(h, w.in_proj)                             # [T, H dk | G dk | G dv (| H dv)]
        parts = list(torch.split(proj, self.proj_widths, dim=1)) + [None]
        out = torch.empty((h.shape[0], m.heads * m.vdim), dtype=h.dtype, device=h.device)
        self.attend(parts[0], parts[1], parts[2], parts[3], out, caches, block_table, st)
        return linear(out, w.o)


def distance_slopes(heads: int) -> list:
    """Slope of every head's bias on the distance: 2^(-8 (h + 1) / heads)."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


class SharedKeyValueAttentionMixer:
    """ONE GEMM with bias [q ; k ; gate] -> 1 / rms of the keys + cache store (one kernel) -> attention (RMS norm of q with the
    product of both norms' weights, window + kept first positions, bias on the distance, softmax, gate per head: one kernel) ->
    o GEMM.  (q^ . (k / rms(k) * w_k) = (q^ * w_k) . k / rms(k): the cached row needs no weight.)"""

    def __init__(self, spec, weight, eps: float, cache_key):
        assert spec.shared_kv and spec.qk_weight_norm and spec.gate_per_head and spec.rot_dims == 0 and not spec.sink
        self.spec, self.weight, self.eps = spec, weight, eps
        self.cache_width, self.cache_slot = cache_key
        slopes = None
        if spec.distance_bias:
            slopes = torch.tensor(distance_slopes(spec.heads), dtype=torch.float32).to(weight.qk_norm.device)
        self.options = AttnOptions(q_norm=weight.qk_norm, prenorm_eps=eps, slopes=slopes, keep_first=spec.keep_first,
                                   gate_per_head=True, shared_kv=True)

    def register(self, model):
        pass

    def state_layout(self) -> dict:
        return {}

    def forward(self, h: torch.Tensor, caches: dict, block_table: torch.Tensor, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        q, k, gate = torch.split(linear_bias(h, w.in_proj, w.in_bias), [m.heads * m.dim, m.kv_heads * m.dim, m.heads], dim=1)
        out = torch.empty((h.shape[0], m.heads * m.dim), dtype=h.dtype, device=h.device)
        if st.ignore_kvcache:
            return linear(out.zero_(), w.o)
        cache = caches[self.cache_width]
        shared_kv_store(k, cache, self.cache_slot, block_table, st, m.kv_heads, m.dim, self.eps)
        window_attention(q, gate, cache, self.cache_slot, block_table, st, out, m.heads, m.kv_heads, m.dim, m.dim, 0, m.window, m.scale,
                         False, None, None, self.options)
        return linear(out, w.o)


class WholeNormAttentionMixer:
    """ONE GEMM [q ; k ; gate] -> norms over the whole projections, rotation, queries in score order, cache store (one kernel) ->
    attention (window, softmax with a learned sink, gate per head: one kernel) -> o GEMM.  A cached key is its projection (which is
    the value), 1 / rms of the token's keys, and its turned entries with the norm's weight: the un-turned entries' weight is part of
    the query (q . (k / rms * w) = (q * w) . k / rms)."""

    def __init__(self, spec, weight, eps: float, cache_key):
        assert spec.shared_kv and spec.whole_norm and spec.gate_per_head and spec.keep_first == 0 and spec.chunk == 0
        self.spec, self.weight, self.eps = spec, weight, eps
        self.cache_width, self.cache_slot = cache_key
        self.options = AttnOptions(gate_per_head=True, shared_kv=True, key_turned=spec.rot_dims, sinks=weight.sink)

    def register(self, model):
        m = self.spec
        model._register_rotary(m.rot_key, m.rot_base, m.rot_dims, m.rot_scaling)

    def state_layout(self) -> dict:
        return {}

    def forward(self, h: torch.Tensor, caches: dict, block_table: torch.Tensor, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        q, k, gate = torch.split(linear(h, w.in_proj), [m.heads * m.dim, m.kv_heads * m.dim, m.heads], dim=1)
        out = torch.empty((h.shape[0], m.heads * m.dim), dtype=h.dtype, device=h.device)
        if st.ignore_kvcache:
            return linear(out.zero_(), w.o)
        cos, sin = st.rotary[m.rot_key] if m.rot_dims > 0 else (None, None)
        cache = caches[self.cache_width]
        q = whole_norm_rope_store(q, k, w.q_norm, w.k_norm, self.eps, cos, sin, cache, self.cache_slot, block_table, st, m.heads,
                                  m.kv_heads, m.dim, m.rot_dims, m.pair_halves)
        window_attention(q, gate, cache, self.cache_slot, block_table, st, out, m.heads, m.kv_heads, m.dim, m.dim, 0, m.window, m.scale,
                         False, None, None, self.options)
        return linear(out, w.o)


class DifferentialAttentionMixer:
    """ONE GEMM with bias [q ; k ; v ; gate] (q rows ordered [key/value head][map][head of the group] at load time) -> per-part
    RMS norm with weight + rotary of k + cache store (one kernel; the row holds both maps' keys and ONE set of values) ->
    attention per map (norm + rotary of q, chunked causal mask, softmax, fp32 output: one kernel) -> map 0 - lambda * map 1,
    unit-RMS over the head, (1 - diff), sigmoid gate (one kernel) -> o GEMM with bias."""

    def __init__(self, spec, weight, eps: float, cache_key):
        assert spec.maps == 2 and spec.qk_weight_norm and spec.gate and not spec.value_rotation and not spec.sink
        self.spec, self.weight, self.eps = spec, weight, eps
        self.cache_width, self.cache_slot = cache_key
        self.options = AttnOptions(pair_halves=spec.pair_halves, softcap=spec.softcap, q_norm=weight.q_norm, k_norm=weight.k_norm,
                                   prenorm_eps=eps, chunk=spec.chunk, vshare=spec.maps, out_f32=True)

    def register(self, model):
        m = self.spec
        model._register_rotary(m.rot_key, m.rot_base, m.rot_dims, m.rot_scaling)

    def state_layout(self) -> dict:
        return {}

    @property
    def proj_widths(self):
        m = self.spec
        return [m.heads * m.maps * m.dim, m.kv_heads * m.maps * m.dim, m.kv_heads * m.vdim, m.heads * m.vdim]

    def forward(self, h: torch.Tensor, caches: dict, block_table: torch.Tensor, states, st) -> torch.Tensor:
        m, w = self.spec, self.weight
        T = h.shape[0]
        proj = torch.nn.functional.linear(h, w.in_proj, w.in_bias)
        q, k, v, gate = torch.split(proj, self.proj_widths, dim=1)
        out = torch.empty((T, m.heads * m.vdim), dtype=h.dtype, device=h.device)
        if st.ignore_kvcache:
            out.zero_()
            return torch.nn.functional.linear(out, w.o, w.o_bias)
        cos, sin = st.rotary[m.rot_key] if m.rot_dims > 0 else (None, None)
        cache = caches[self.cache_width]
        H2, G2 = m.heads * m.maps, m.kv_heads * m.maps
        window_kv_store(k, v, cache, self.cache_slot, block_table, st, G2, m.dim, m.vdim, m.rot_dims, cos, sin, self.options)
        a = torch.empty((T, H2 * m.vdim), dtype=torch.float32, device=h.device)
        window_attention(q, None, cache, self.cache_slot, block_table, st, a, H2, G2, m.dim, m.vdim, m.rot_dims, m.window,
                         m.scale, False, cos, sin, self.options)
        diff_combine(a, gate, out, m.heads, m.kv_heads, m.vdim, w.lam, self.eps, 1.0 - m.diff)
        return torch.nn.functional.linear(out, w.o, w.o_bias)
