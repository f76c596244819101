"""Plain, slow restatement of the Vorerax design, one function per mechanism.

TEST INFRASTRUCTURE ONLY: shares no code with `swiftllm_b200/`.  Everything is computed per sequence, over the whole sequence at
once, in one floating-point type (float32 or float64), token by token where the rule is a recurrence.

The design.  A decoder-only model:
  * embedding: embed[token] * a constant, plus a row of a second table picked by a hash of (previous token, token);
  * several residual streams, all equal to the embedding at the start; a sublayer reads a weighted sum of the streams through an RMS
    norm; afterwards the streams are mixed by a small matrix and each takes a weighted share of the sublayer's output (without
    streams: the plain residual sum); a layer may lack the feed-forward;
  * mixer "attention": grouped key heads whose un-normed projections are also the values; RMS norm of the whole query / key
    projection; partial rotation in the halves layout with piecewise scaled frequencies; sliding window; a learned softmax sink and
    a sigmoid gate per head;
  * mixer "delta": the gated delta rule behind short convolutions, with unit queries and keys;
  * mixer "mlstm": a matrix memory with exponential input gate, its normaliser and a running maximum;
  * feed-forward: SiLU-gated experts, sigmoid scores with a correction that takes part in the choice only, groups of experts;
  * output: the sum of the streams, the norm, the head.
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


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def embedding(tokens, tens: dict, spec: dict) -> torch.Tensor:
    x = tens["embed"][torch.tensor(tokens, dtype=torch.long)] * spec.get("scale", 1.0)
    pair = spec.get("bigram")
    if pair:
        rows = [pair["buckets"]]
        for before, now in zip(tokens[:-1], tokens[1:]):
            rows.append((before * pair["mul_prev"] + now * pair["mul_cur"]) % pair["buckets"])
        x = x + tens["bigram"][torch.tensor(rows, dtype=torch.long)]
    return x


# ---------------------------------------------------------------- streams
def read_streams(xs: torch.Tensor, weights: torch.Tensor) -> torch.Tensor:
    """xs [n, streams, width] -> the sublayer's input before its norm."""
    return sum(weights[s] * xs[:, s] for s in range(xs.shape[1]))


def write_streams(xs: torch.Tensor, mix: torch.Tensor, share: torch.Tensor, y: torch.Tensor, mult: float) -> torch.Tensor:
    """mix [from, to]."""
    S = xs.shape[1]
    return torch.stack([sum(mix[s, t] * xs[:, s] for s in range(S)) + mult * share[t] * y for t in range(S)], dim=1)


# ---------------------------------------------------------------- attention
def frequencies(rot: dict) -> list:
    """Long waves are stretched by the factor, short ones kept, with a blend between."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif not wave < s["original"] / s["high"]:
                u = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - u) * f / s["factor"] + u * f
        out.append(f)
    return out


def rotate(v: torch.Tensor, positions, rot) -> torch.Tensor:
    """v [n, heads, d]: entries (i, i + dims / 2) turn by position * frequency_i; entries from dims on pass."""
    if not rot or not rot["dims"]:
        return v
    half, out = rot["dims"] // 2, v.clone()
    for t, p in enumerate(positions):
        for i, f in enumerate(frequencies(rot)):
            c, s = math.cos(p * f), math.sin(p * f)
            out[t, :, i] = v[t, :, i] * c - v[t, :, i + half] * s
            out[t, :, i + half] = v[t, :, i + half] * c + v[t, :, i] * s
    return out


def softmax_with_sink(scores: torch.Tensor, sink) -> torch.Tensor:
    """scores [query, key] (-inf: not visible); the denominator also contains exp(sink)."""
    top = torch.clamp(scores.max(dim=1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(dim=1, keepdim=True) + torch.exp(sink - top))


def attention(h: torch.Tensor, positions, p: dict, m: dict, eps: float) -> torch.Tensor:
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ p["q"].T, h @ p["k"].T
    v = k.reshape(n, G, d)                                               # the values: the keys as projected
    q = rotate((unit_rms(q, eps) * p["q.norm"]).reshape(n, H, d), positions, m.get("rot"))
    k = rotate((unit_rms(k, eps) * p["k.norm"]).reshape(n, G, d), positions, m.get("rot"))
    pos = torch.tensor(positions)
    dist = pos[:, None] - pos[None, :]
    visible = dist >= 0
    if m.get("mask"):
        visible = visible & (dist < m["mask"]["size"])
    gate = torch.sigmoid(h @ p["g"].T)
    out = torch.zeros((n, H, d), dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        out[:, hh] = softmax_with_sink(s.masked_fill(~visible, -math.inf), p["sink"][hh]) @ v[:, g] * gate[:, hh:hh + 1]
    return out.reshape(n, H * d) @ p["o"].T


# ---------------------------------------------------------------- gated delta rule
def short_convolution(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [n, C], taps [C, K] (last column: the current token), then silu."""
    n, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(n):
        for b in range(K):
            if t - b >= 0:
                out[t] += taps[:, K - 1 - b] * x[t - b]
    return silu(out)


def unit_length(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_states(q, k, v, decay, beta) -> torch.Tensor:
    """q, k [n, H, dk], v [n, H, dv], decay, beta [n, H] -> o [n, H, dv]."""
    n, H, dk = q.shape
    S = torch.zeros((H, dk, v.shape[2]), dtype=q.dtype)
    out = []
    for t in range(n):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out)


def delta(h: torch.Tensor, p: dict, m: dict, eps: float) -> torch.Tensor:
    n, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_convolution(h @ p[c].T, p[c + ".conv"]) for c in "qkv")
    which = torch.arange(H) // (H // G)
    q = unit_length(q.reshape(n, G, dk))[:, which] * dk ** -0.5
    k = unit_length(k.reshape(n, G, dk))[:, which]
    beta = torch.sigmoid(h @ p["b"].T)
    decay = torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o = delta_states(q, k, v.reshape(n, H, dv), decay, beta)
    o = unit_rms(o, eps) * p["norm"]
    return (o.reshape(n, H * dv) * silu(h @ p["g"].T)) @ p["o"].T


# ---------------------------------------------------------------- matrix memory
def mlstm_states(q, k, v, log_in, log_forget) -> torch.Tensor:
    """q, k [n, H, dk], v [n, H, dv], gates [n, H] -> o [n, H, dv]."""
    n, H, dk = q.shape
    S, norm = torch.zeros((H, dk, v.shape[2]), dtype=q.dtype), torch.zeros((H, dk), dtype=q.dtype)
    top = torch.zeros((H,), dtype=q.dtype)
    out = []
    for t in range(n):
        new = torch.maximum(log_forget[t] + top, log_in[t])
        keep, take = torch.exp(log_forget[t] + top - new), torch.exp(log_in[t] - new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        norm = keep[:, None] * norm + take[:, None] * k[t]
        top = new
        size = torch.maximum((norm * q[t]).sum(dim=1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hkv,hk->hv", S, q[t]) / size[:, None])
    return torch.stack(out)


def mlstm(h: torch.Tensor, p: dict, m: dict, eps: float) -> torch.Tensor:
    n, H, dk, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ p["q"].T * dk ** -0.5).reshape(n, H, dk)
    k = (h @ p["k"].T).reshape(n, H, dk)
    v = (h @ p["v"].T).reshape(n, H, dv)
    log_in = cap * torch.tanh((h @ p["i"].T + p["i.b"]) / cap)
    log_forget = -softplus(-cap * torch.tanh((h @ p["f"].T + p["f.b"]) / cap))
    o = unit_rms(mlstm_states(q, k, v, log_in, log_forget), eps)
    return (o.reshape(n, H * dv) * p["norm"] * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


# ---------------------------------------------------------------- feed-forward
def routing_weights(z: torch.Tensor, correction: torch.Tensor, top: int, groups) -> torch.Tensor:
    """z [n, experts] router logits -> [n, experts] weights (0: not used)."""
    s = torch.sigmoid(z)
    out = torch.zeros_like(s)
    E = z.shape[1]
    for t in range(z.shape[0]):
        choice = [float(a) for a in s[t] + correction]
        allowed = set(range(E))
        if groups and groups["count"] > 1:
            size = E // groups["count"]
            score = [sum(sorted(choice[g * size:(g + 1) * size])[-2:]) for g in range(groups["count"])]
            best = sorted(range(groups["count"]), key=lambda g: -score[g])[:groups["keep"]]
            allowed = {e for g in best for e in range(g * size, (g + 1) * size)}
        for e in sorted(allowed, key=lambda e: -choice[e])[:top]:
            out[t, e] = s[t, e]
    return out


def experts(h: torch.Tensor, p: dict, f: dict) -> torch.Tensor:
    r = f["router"]
    w = routing_weights(h @ p["router"].T, p["correction"], r["top"], r.get("groups"))
    y = torch.zeros_like(h)
    for e in range(r["experts"]):
        y = y + w[:, e:e + 1] * ((silu(h @ p[f"e{e}.gate"].T) * (h @ p[f"e{e}.up"].T)) @ p[f"e{e}.down"].T)
    return y


# ---------------------------------------------------------------- the model
def forward(config: dict, tensors: dict, tokens, dtype=torch.float32, keep_layers: bool = False):
    """-> logits [n, vocab] (and the sum of the streams after every layer, [layers, n, width])."""
    tens = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps, mult = config["norm"]["eps"], config.get("residual_mult", 1.0)
    positions = list(range(len(tokens)))
    streams = config.get("streams")
    x = embedding(tokens, tens, config.get("embedding") or {})
    xs = torch.stack([x] * (streams or 1), dim=1)
    kept = []
    for i, layer in enumerate(config["layers"]):
        p = sub(tens, f"l{i}.")
        mp, m = sub(p, "mix."), layer["mixer"]
        for q in (1, 2):
            if q == 2 and layer.get("mlp") is None:
                continue
            u = read_streams(xs, p[f"hc{q}.in"]) if streams else xs[:, 0]
            h = unit_rms(u, eps) * p[f"norm{q}"]
            if q == 2:
                y = experts(h, sub(p, "mlp."), layer["mlp"])
            elif layer["type"] == "attention":
                y = attention(h, positions, mp, m, eps)
            elif layer["type"] == "delta":
                y = delta(h, mp, m, eps)
            else:
                assert layer["type"] == "mlstm"
                y = mlstm(h, mp, m, eps)
            if streams:
                xs = write_streams(xs, p[f"hc{q}.mix"], p[f"hc{q}.out"], y, mult)
            else:
                xs = xs + mult * y[:, None]
        kept.append(xs.sum(dim=1))
    logits = (unit_rms(xs.sum(dim=1), eps) * tens["final.norm"]) @ tens["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


def tensor_shapes(config: dict) -> dict:
    """name -> shape of every tensor of a checkpoint of this configuration."""
    W, V, S = config["width"], config["vocab"], config.get("streams")
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    pair = (config.get("embedding") or {}).get("bigram")
    if pair:
        out["bigram"] = (pair["buckets"] + 1, W)
    for i, layer in enumerate(config["layers"]):
        m, f, pre = layer["mixer"], layer.get("mlp"), f"l{i}."
        for q in ((1,) if f is None else (1, 2)):
            out[f"{pre}norm{q}"] = (W,)
            if S:
                out.update({f"{pre}hc{q}.in": (S,), f"{pre}hc{q}.out": (S,), f"{pre}hc{q}.mix": (S, S)})
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            shapes = {"q": (H * dk, W), "k": (G * dk, W), "q.norm": (H * dk,), "k.norm": (G * dk,), "sink": (H,), "g": (H, W),
                      "o": (W, H * dv)}
        elif layer["type"] == "delta":
            G, K = m["kv_heads"], m["conv"]
            shapes = {"q": (G * dk, W), "q.conv": (G * dk, K), "k": (G * dk, W), "k.conv": (G * dk, K), "v": (H * dv, W),
                      "v.conv": (H * dv, K), "b": (H, W), "a": (H, W), "A_log": (H,), "dt_bias": (H,), "norm": (dv,), "g": (H * dv, W),
                      "o": (W, H * dv)}
        else:
            shapes = {"q": (H * dk, W), "k": (H * dk, W), "v": (H * dv, W), "g": (H * dv, W), "o": (W, H * dv), "norm": (H * dv,),
                      "i": (H, W), "i.b": (H,), "f": (H, W), "f.b": (H,)}
        out.update({f"{pre}mix.{k}": s for k, s in shapes.items()})
        if f is not None:
            E, F = f["router"]["experts"], f["expert"]["ff"]
            out.update({pre + "mlp.router": (E, W), pre + "mlp.correction": (E,)})
            for e in range(E):
                out.update({f"{pre}mlp.e{e}.gate": (F, W), f"{pre}mlp.e{e}.up": (F, W), f"{pre}mlp.e{e}.down": (W, F)})
    return out


def random_tensors(config: dict, seed: int = 0, dtype=torch.bfloat16) -> dict:
    """Random weights for tests: projections N(0, 1 / fan-in) so that every mechanism contributes, norm weights around one, stream
    weights of order one with every entry different, gate biases that keep what was written for some tokens."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        if "norm" in leaf:
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif leaf.endswith(".mix") and leaf.startswith("hc"):
            t = torch.eye(shape[0]) * 0.7 + torch.randn(shape, generator=g) * 0.3 / math.sqrt(shape[0])
        elif leaf.endswith((".in", ".out")) and leaf.startswith("hc"):
            t = 0.5 + 0.5 * torch.randn(shape, generator=g)
        elif leaf == "mix.A_log":
            t = torch.randn(shape, generator=g) - 1.0
        elif leaf == "mix.dt_bias":
            t = torch.randn(shape, generator=g) - 1.0
        elif leaf == "mix.f.b":
            t = 2.0 + torch.randn(shape, generator=g)
        elif leaf == "mix.i.b":
            t = torch.randn(shape, generator=g)
        elif leaf == "mix.sink":
            t = torch.randn(shape, generator=g)
        elif leaf == "mlp.correction":
            t = 0.2 * torch.randn(shape, generator=g) - 0.1
        elif name in ("embed", "bigram"):
            t = torch.randn(shape, generator=g)
        elif leaf.endswith(".conv"):
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out
