"""Plain, slow restatement of the Zuzezen design, one function per mechanism.

TEST INFRASTRUCTURE ONLY: shares no code with `swiftllm_b200/`.  Everything is computed per sequence, over the whole sequence at
once, in one floating-point type (float32 or float64), token by token where the rule is a recurrence.

The design.  A decoder-only model on a residual stream x [n, width]:
  * embedding: x = embed[token] * a constant;
  * a layer:  x <- x + ls1 * norm1(mixer(x)),  x <- x + ls2 * norm2(ff(x)): the sublayers read the stream itself, their outputs go
    through an RMS norm (weight stored around zero) and an element-wise scale; a layer may lack the feed-forward;
  * mixer "latent_attention": keys and values of all heads come from one RMS-normed latent per token, plus one rotated key part
    that all heads share; rotation in interleaved pairs with stretched (ramped) frequencies; causal softmax whose denominator also
    holds exp(sink) of the head; element-wise sigmoid gate;
  * mixer "attention": grouped key heads whose un-normed projections are also the values; RMS norm with weight on queries and keys;
    no rotation, a bias of -slope * distance on the scores; sliding window plus the first tokens of the sequence; one sigmoid gate
    per head;
  * mixer "gla": linear attention with a decay per key channel that depends on the token; the heads' outputs are RMS-normed, gated
    by a SiLU and projected;
  * feed-forward: SiLU gated linear unit with biases;
  * output: the norm, then the head.
"""
from __future__ import annotations

import math

import torch


def sub(tensors: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


# ---------------------------------------------------------------- small pieces
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def offset_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def ramped_frequencies(rot: dict):
    """-> (frequency of every pair, factor on cos and sin): pairs that turn often over the original context keep their frequency,
    slow ones are divided by the factor, with a linear ramp between."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return plain, 1.0

    def pair(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair(s["fast"])), 0)
    hi = min(math.ceil(pair(s["slow"])), dims - 1)
    freqs = []
    for i, f in enumerate(plain):
        ramp = (i - lo) / max(hi - lo, 0.001)
        ramp = min(1.0, max(0.0, ramp))
        freqs.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return freqs, 0.1 * math.log(s["factor"]) + 1.0


def rotate(v: torch.Tensor, positions, rot: dict) -> torch.Tensor:
    """v [n, ..., d]: entries (2i, 2i + 1), i < dims / 2, turn by position * frequency_i; the rest pass."""
    freqs, amp = ramped_frequencies(rot)
    out = v.clone()
    for t, p in enumerate(positions):
        for i, f in enumerate(freqs):
            c, s = math.cos(p * f) * amp, math.sin(p * f) * amp
            a, b = v[t, ..., 2 * i].clone(), v[t, ..., 2 * i + 1].clone()
            out[t, ..., 2 * i] = a * c - b * s
            out[t, ..., 2 * i + 1] = b * c + a * s
    return out


# ---------------------------------------------------------------- latent attention
def softmax_with_sink(scores: torch.Tensor, sink) -> torch.Tensor:
    """scores [query, key] (-inf: not visible); the denominator also contains exp(sink)."""
    top = torch.clamp(scores.max(dim=1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(dim=1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h: torch.Tensor, positions, p: dict, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, dn, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ p["q"].T).reshape(n, H, dn + dr)
    down = h @ p["dkv"].T
    c = unit_rms(down[:, :r], eps) * p["dkv.norm"]
    k_rot = rotate(down[:, r:], positions, m["rot"])
    q_rot = rotate(q[:, :, dn:], positions, m["rot"])
    k = (c @ p["uk"].T).reshape(n, H, dn)
    v = (c @ p["uv"].T).reshape(n, H, dv)
    pos = torch.tensor(positions)
    visible = pos[None, :] <= pos[:, None]
    out = torch.zeros((n, H, dv), dtype=h.dtype)
    for hh in range(H):
        s = (q[:, hh, :dn] @ k[:, hh].T + q_rot[:, hh] @ k_rot.T) * m["scale"]
        out[:, hh] = softmax_with_sink(s.masked_fill(~visible, -math.inf), p["sink"][hh]) @ v[:, hh]
    return (out.reshape(n, H * dv) * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


# ---------------------------------------------------------------- windowed attention with kept first tokens
def distance_slope(head: int, heads: int) -> float:
    return 2.0 ** (-8.0 * (head + 1) / heads)


def visible_keys(positions, mask: dict) -> torch.Tensor:
    pos = torch.tensor(positions)
    i, j = pos[:, None], pos[None, :]
    return (j <= i) & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def window_attention(h: torch.Tensor, positions, p: dict, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ p["q"].T + p["q.b"]).reshape(n, H, d)
    k = (h @ p["k"].T + p["k.b"]).reshape(n, G, d)
    v = k                                                   # the values: the keys as projected
    q = unit_rms(q, eps) * p["q.norm"]
    k = unit_rms(k, eps) * p["k.norm"]
    pos = torch.tensor(positions)
    dist = (pos[:, None] - pos[None, :]).to(h.dtype)
    visible = visible_keys(positions, m["mask"])
    gate = torch.sigmoid(h @ p["g"].T)                      # [n, H]
    out = torch.zeros((n, H, d), dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"] - distance_slope(hh, H) * dist
        out[:, hh] = (torch.softmax(s.masked_fill(~visible, -math.inf), dim=1) @ v[:, g]) * gate[:, hh:hh + 1]
    return out.reshape(n, H * d) @ p["o"].T


# ---------------------------------------------------------------- gated linear attention
def channel_decays(h: torch.Tensor, p: dict, m: dict) -> torch.Tensor:
    """-> [n, heads, dim], each in (0, 1)."""
    z = (h @ p["a1"].T) @ p["a2"].T + p["a2.b"]
    log_sigmoid = torch.where(z < 0, z - torch.log1p(torch.exp(-z.abs())), -torch.log1p(torch.exp(-z.abs())))
    return torch.exp(log_sigmoid / m["tau"]).reshape(h.shape[0], m["heads"], m["dim"])


def gla_states(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, alpha: torch.Tensor) -> torch.Tensor:
    """q, k, alpha [n, H, dk], v [n, H, dv] -> o [n, H, dv]."""
    n, H, dk = q.shape
    S = torch.zeros((H, dk, v.shape[2]), dtype=q.dtype)
    out = []
    for t in range(n):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(dim=1))
    return torch.stack(out)


def gated_linear_attention(h: torch.Tensor, p: dict, m: dict, eps: float) -> torch.Tensor:
    n, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ p["q"].T * dk ** -0.5).reshape(n, H, dk)
    k = (h @ p["k"].T).reshape(n, H, dk)
    v = (h @ p["v"].T).reshape(n, H, dv)
    o = gla_states(q, k, v, channel_decays(h, p, m))
    o = unit_rms(o, eps) * p["norm"]
    return (o.reshape(n, H * dv) * silu(h @ p["g"].T)) @ p["o"].T


# ---------------------------------------------------------------- feed-forward
def silu_glu(h: torch.Tensor, p: dict) -> torch.Tensor:
    return (silu(h @ p["gate"].T + p["gate.b"]) * (h @ p["up"].T + p["up.b"])) @ p["down"].T + p["down.b"]


# ---------------------------------------------------------------- the model
def forward(config: dict, tensors: dict, tokens, dtype=torch.float32, keep_layers: bool = False):
    """-> logits [n, vocab] (and the stream after every layer, [layers, n, width])."""
    tens = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    positions = list(range(len(tokens)))
    x = tens["embed"][torch.tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    kept = []
    for i, layer in enumerate(config["layers"]):
        p = sub(tens, f"l{i}.")
        mp, m = sub(p, "mix."), layer["mixer"]
        if layer["type"] == "latent_attention":
            y = latent_attention(x, positions, mp, m, eps)
        elif layer["type"] == "attention":
            y = window_attention(x, positions, mp, m, eps)
        else:
            assert layer["type"] == "gla"
            y = gated_linear_attention(x, mp, m, eps)
        x = x + offset_norm(y, p["norm1"], eps) * p["ls1"]
        if layer.get("mlp") is not None:
            x = x + offset_norm(silu_glu(x, sub(p, "mlp.")), p["norm2"], eps) * p["ls2"]
        kept.append(x.clone())
    logits = offset_norm(x, tens["final.norm"], eps) @ tens["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


def tensor_shapes(config: dict, rank: int = 5) -> dict:
    """name -> shape of every tensor of a checkpoint of this configuration (`rank`: inner size of the decays' projection, which
    only the checkpoint's shapes tell)."""
    W, V = config["width"], config["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(config["layers"]):
        m, f, pre = layer["mixer"], layer.get("mlp"), f"l{i}."
        out[pre + "norm1"], out[pre + "ls1"] = (W,), (W,)
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "latent_attention":
            r, dr = m["kv_rank"], m["rot_dim"]
            out.update({pre + "mix.q": (H * (dk + dr), W), pre + "mix.dkv": (r + dr, W), pre + "mix.dkv.norm": (r,),
                        pre + "mix.uk": (H * dk, r), pre + "mix.uv": (H * dv, r), pre + "mix.sink": (H,), pre + "mix.g": (H * dv, W),
                        pre + "mix.o": (W, H * dv)})
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            out.update({pre + "mix.q": (H * dk, W), pre + "mix.q.b": (H * dk,), pre + "mix.k": (G * dk, W), pre + "mix.k.b": (G * dk,),
                        pre + "mix.q.norm": (dk,), pre + "mix.k.norm": (dk,), pre + "mix.g": (H, W), pre + "mix.o": (W, H * dv)})
        else:
            out.update({pre + "mix.q": (H * dk, W), pre + "mix.k": (H * dk, W), pre + "mix.v": (H * dv, W), pre + "mix.g": (H * dv, W),
                        pre + "mix.o": (W, H * dv), pre + "mix.norm": (dv,), pre + "mix.a1": (rank, W), pre + "mix.a2": (H * dk, rank),
                        pre + "mix.a2.b": (H * dk,)})
        if f is not None:
            F = f["ff"]
            out[pre + "norm2"], out[pre + "ls2"] = (W,), (W,)
            out.update({pre + "mlp.gate": (F, W), pre + "mlp.gate.b": (F,), pre + "mlp.up": (F, W), pre + "mlp.up.b": (F,),
                        pre + "mlp.down": (W, F), pre + "mlp.down.b": (W,)})
    return out


def random_tensors(config: dict, seed: int = 0, dtype=torch.bfloat16, rank: int = 5) -> dict:
    """Random weights for tests: projections N(0, 1 / fan-in) so that every mechanism contributes, norm weights around zero (the
    block's) or one (the mixers' own), layer scales around 0.7, decay biases around 1."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config, rank).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        if leaf in ("norm1", "norm2", "final.norm"):
            t = 0.3 * torch.randn(shape, generator=g)
        elif leaf.endswith(".norm"):
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif leaf in ("ls1", "ls2"):
            t = 0.7 + 0.3 * torch.randn(shape, generator=g)
        elif leaf == "mix.a2.b":
            t = 1.0 + torch.randn(shape, generator=g)
        elif leaf == "mix.sink":
            t = torch.randn(shape, generator=g)
        elif len(shape) == 1:
            t = 0.3 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out
