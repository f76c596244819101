"""GPU: the Vorerax worker and its CUDA kernels (csrc/hyper_streams.cu, csrc/delta_rule.cu, csrc/matrix_memory.cu; the turned shared keys
and learned sinks of csrc/window_attn.cu; the group-limited router of csrc/stream_ops.cu) - every kernel alone against a plain loop
written here or in oracle/vorerax.py, then the scenarios of tests/bupozen_cases.py and tests/vorerax_cases.py through the worker (fp32
tight, bf16 loose)."""
import math
import types

import pytest
import torch

import bupozen_cases as B
import vorerax_cases as C
from oracle import vorerax as O
from test_bupozen_gpu import _make
from test_buzarax_gpu import _schedule, _step

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def _tol(dtype):
    return 1e-5 if dtype == torch.float32 else 1.2e-2


# ---------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams,width", [(1, 48), (2, 45), (3, 1000), (4, 4096), (5, 50), (7, 260), (12, 36), (4, 12000)])
def test_streams_write_and_read(dtype, streams, width):
    from swiftllm_b200.worker.kernels.hyper_streams import stream_mix_norm
    g = torch.Generator().manual_seed(streams * width)
    T, eps = 9, 1e-3
    x, y = torch.randn(T, streams, width, generator=g) * 2, torch.randn(T, width, generator=g).to(dtype)
    mix, share, read = torch.randn(streams, streams, generator=g), torch.randn(streams, generator=g), torch.randn(streams, generator=g)
    w = 1 + 0.3 * torch.randn(width, generator=g)
    new = O.write_streams(x, mix, share, y.float(), 1.0)
    ref = O.unit_rms(O.read_streams(new, read), eps) * w
    d = lambda a: a.to(DEV)
    conn = dict(y=d(y), mix=d(mix), share=d(share), out_dtype=dtype)
    xd = d(x)
    h = stream_mix_norm(xd, streams, x_out=xd, read=d(read), norm_w=d(w), eps=eps, **conn)               # in place
    assert B.rel_err(xd, new) < 1e-6 and B.rel_err(h.float(), ref) < _tol(dtype)
    rows = torch.tensor([7, 0, 7, 3], dtype=torch.int32)
    h = stream_mix_norm(d(x), streams, read=d(read), norm_w=d(w), eps=eps, rows=d(rows), **conn)          # some rows, streams dropped
    assert h.shape == (4, width) and B.rel_err(h.float(), ref[rows.long()]) < _tol(dtype)
    out = torch.empty(T, streams, width, device=DEV)
    assert stream_mix_norm(d(x), streams, x_out=out, **conn) is None and B.rel_err(out, new) < 1e-6      # write only
    e = x[:, 0].contiguous()                                                                             # all streams equal
    same = e[:, None].expand(-1, streams, -1)
    h = stream_mix_norm(d(e), streams, x_out=out, read=d(read), norm_w=d(w), eps=eps, **conn)
    new = O.write_streams(same, mix, share, y.float(), 1.0)
    assert B.rel_err(out, new) < 1e-6 and B.rel_err(h.float(), O.unit_rms(O.read_streams(new, read), eps) * w) < _tol(dtype)
    h = stream_mix_norm(d(e), streams, read=d(read), norm_w=d(w), eps=eps, out_dtype=dtype)               # read only
    assert B.rel_err(h.float(), O.unit_rms(O.read_streams(same, read), eps) * w) < _tol(dtype)


@pytest.mark.parametrize("experts,top,groups,keep", [(6, 2, 3, 1), (12, 5, 4, 2), (64, 8, 8, 3), (7, 3, 7, 4), (40, 40, 1, 1), (33, 2, 1, 1)])
def test_group_limited_sigmoid_router(experts, top, groups, keep):
    from swiftllm_b200.worker.kernels.stream_ops import moe_route_sigmoid
    g = torch.Generator().manual_seed(experts)
    z, c = torch.randn(57, experts, generator=g) * 2, torch.randn(experts, generator=g) - 2.5
    w = moe_route_sigmoid(z.to(DEV), c.to(DEV), top, groups, keep)
    ref = O.routing_weights(z, c, top, {"count": groups, "keep": keep})
    assert torch.equal(w.cpu() > 0, ref > 0) and torch.allclose(w.cpu(), ref, atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [64, 30, 33])
def test_expert_activation(dtype, ff):
    from swiftllm_b200.worker.kernels.stream_ops import moe_silu_glu_scale
    g = torch.Generator().manual_seed(ff)
    E, T = 5, 11
    u, w = (torch.randn(T, E * 2 * ff, generator=g) * 2).to(dtype), torch.rand(T, E, generator=g) * (torch.rand(T, E, generator=g) > 0.5)
    b = u.float().view(T, E, 2, ff)
    ref = O.silu(b[:, :, 0]) * b[:, :, 1] * w[:, :, None]
    assert B.rel_err(moe_silu_glu_scale(u.to(DEV), w.to(DEV), E, ff).float(), ref.reshape(T, E * ff)) < _tol(dtype)


def _run_recurrence(call, parts, lens, rows, plan, prompt):
    """Feed `lens` sequences (rows of the state tensors) through `call(step, cat)` in the steps of `plan`."""
    got = [[] for _ in lens]
    for segs in _schedule(lens, plan):
        segs = sorted(segs, key=lambda e: e[2] == 1)       # prompt portions first
        st = _step([(rows[s], p0, n) for s, p0, n in segs])
        long = [n for _, _, n in segs if n > 1 or prompt]
        st.num_prefill_seqs, st.num_prefill_tokens = len(long), sum(long)
        out = call(st, lambda name: torch.cat([parts[name][s][p0:p0 + n] for s, p0, n in segs]).to(DEV))
        out, at = out.float().cpu(), 0
        for s, p0, n in segs:
            got[s].append((p0, out[at:at + n])); at += n
    return [torch.cat([o for _, o in sorted(g, key=lambda e: e[0])]) for g in got]


LENS, ROWS = [300, 37], [2, 0]
PLAN = [[(0, 1), (1, 2)], [(0, 2), (1, 1)], [(0, 217), (1, 1)], [(1, 33)], [(0, 79)], [(0, 1)]]
SHAPES = [(4, 2, 10, 6), (1, 1, 37, 70), (3, 1, 1, 2), (6, 3, 64, 64), (2, 2, 130, 33), (3, 3, 96, 160), (4, 2, 128, 128), (1, 1, 300, 20),
          (2, 1, 256, 36), (8, 8, 16, 8)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [True, False])
@pytest.mark.parametrize("H,G,dk,dv", SHAPES)
def test_delta_rule_state_through_portions(dtype, H, G, dk, dv, prompt):
    """Two sequences in rows 2 and 0 of the state tensor (which starts full of junk), fed in portions down to one token; some heads forget
    within a token, some hardly at all.  `prompt`: every segment as a prompt portion; otherwise one-token segments go through the launch
    of single decoded tokens."""
    from swiftllm_b200.worker.kernels.head_decay import delta_rule
    g = torch.Generator().manual_seed(H * dk + dv)
    r = lambda width, scale=1.0: [torch.randn(n, width, generator=g) * scale for n in LENS]
    parts = {"q": [x.to(dtype) for x in r(G * dk)], "k": [x.to(dtype) for x in r(G * dk)], "v": [x.to(dtype) for x in r(H * dv)],
             "gate": [x.to(dtype) for x in r(H * dv)], "a": r(H), "b": r(H, 2.0)}
    rate, bias, w = torch.exp(torch.linspace(-7.0, 4.5, H)), torch.randn(H, generator=g), 1 + 0.3 * torch.randn(dv, generator=g)
    which = torch.arange(H) // (H // G)
    ref = []
    for s, n in enumerate(LENS):
        q, k = (O.unit_length(parts[c][s].double().view(n, G, dk))[:, which] for c in "qk")
        decay = torch.exp(-rate.double() * O.softplus(parts["a"][s].double() + bias))
        o = O.delta_states(q * dk ** -0.5, k, parts["v"][s].double().view(n, H, dv), decay, torch.sigmoid(parts["b"][s].double()))
        ref.append((O.unit_rms(o, 1e-5) * w).reshape(n, H * dv) * O.silu(parts["gate"][s].double()))
    state = torch.full((3, H, dk, dv), 1e4, device=DEV)
    call = lambda st, cat: delta_rule(cat("q"), cat("k"), cat("v"), cat("a"), cat("b"), bias.to(DEV), rate.to(DEV), w.to(DEV), 1e-5,
                                      cat("gate"), state, st, H, G, dk, dv)
    for s, full in enumerate(_run_recurrence(call, parts, LENS, ROWS, PLAN, prompt)):
        row_err = (full - ref[s]).pow(2).mean(-1).sqrt() / ref[s].pow(2).mean(-1).sqrt()
        assert B.rel_err(full, ref[s]) < (3e-5 if dtype == torch.float32 else 1.2e-2) and float(row_err.max()) < (1e-3 if dtype == torch.float32 else 3e-2), s
    assert bool((state[1] == 1e4).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [True, False])
@pytest.mark.parametrize("H,G,dk,dv", SHAPES)
def test_matrix_memory_state_through_portions(dtype, H, G, dk, dv, prompt):
    """As above for the matrix memory: input gates that leap, forget gates near zero and near one, state, normaliser and maximum in junk
    rows; queries small enough that the denominator's floor counts in one head."""
    from swiftllm_b200.worker.kernels.head_decay import matrix_memory
    g = torch.Generator().manual_seed(H * dk + dv + 1)
    cap = 7.0
    r = lambda width, scale=1.0: [torch.randn(n, width, generator=g) * scale for n in LENS]
    parts = {"q": [x.to(dtype) for x in r(H * dk)], "k": [x.to(dtype) for x in r(H * dk)], "v": [x.to(dtype) for x in r(H * dv)],
             "gate": [x.to(dtype) for x in r(H * dv)], "f": r(H), "i": r(H, 4.0)}
    for s in range(2):
        parts["q"][s][:, :dk] *= 0.05
    fb, ib = torch.linspace(-4.0, 9.0, H), torch.randn(H, generator=g)
    w = 1 + 0.3 * torch.randn(H * dv, generator=g)
    ref = []
    for s, n in enumerate(LENS):
        q, k, v = (parts[c][s].double().view(n, H, -1) for c in "qkv")
        li = cap * torch.tanh((parts["i"][s].double() + ib) / cap)
        lf = -O.softplus(-cap * torch.tanh((parts["f"][s].double() + fb) / cap))
        o = O.unit_rms(O.mlstm_states(q * dk ** -0.5, k, v, li, lf), 1e-3).reshape(n, H * dv)
        ref.append(o * w * torch.sigmoid(parts["gate"][s].double()))
    junk = lambda *shape: torch.full(shape, 1e4, device=DEV)
    states = junk(3, H, dk, dv), junk(3, H, dk), junk(3, H)
    call = lambda st, cat: matrix_memory(cat("q"), cat("k"), cat("v"), cat("f"), cat("i"), fb.to(DEV), ib.to(DEV), cap, w.to(DEV), 1e-3,
                                         cat("gate"), *states, st, H, dk, dv)
    for s, full in enumerate(_run_recurrence(call, parts, LENS, ROWS, PLAN, prompt)):
        row_err = (full - ref[s]).pow(2).mean(-1).sqrt() / ref[s].pow(2).mean(-1).sqrt()
        assert B.rel_err(full, ref[s]) < (5e-5 if dtype == torch.float32 else 1.2e-2) and float(row_err.max()) < (2e-3 if dtype == torch.float32 else 3e-2), s
    assert all(bool((t[1] == 1e4).all()) for t in states)


@pytest.mark.parametrize("segments,H,dk,dv", [(40, 4, 128, 128), (80, 4, 64, 100), (100, 2, 128, 64), (50, 4, 200, 64)])
def test_recurrences_of_many_segments_at_once(segments, H, dk, dv):
    """Enough prompt portions to fill the GPU (wider column slices, the head norm inside the kernel) beside single decoded tokens, inputs
    as columns of a wider matrix, states carried in: both recurrences against the token-by-token rule on a few of the segments."""
    from swiftllm_b200.worker.kernels.head_decay import delta_rule, matrix_memory
    g = torch.Generator().manual_seed(segments)
    segs = [(i, 0 if i % 3 == 0 else 40 + i, 3 + i % 19) for i in range(segments)] + [(segments + i, 0 if i == 0 else 9, 1) for i in range(5)]
    T, R = sum(n for _, _, n in segs), segments + 5
    st = _step(segs)
    st.num_prefill_seqs, st.num_prefill_tokens = segments, T - 5
    wide = torch.randn(T, 2 * H * dk + 2 * H * dv + 5, generator=g)
    q, k, v, gate, _ = torch.split(wide, [H * dk, H * dk, H * dv, H * dv, 5], dim=1)
    za, zb, pa, pb = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g), torch.randn(H, generator=g), torch.rand(H, generator=g)
    S0, n0, m0 = torch.randn(R, H, dk, dv, generator=g) * 0.3, torch.randn(R, H, dk, generator=g), torch.randn(R, H, generator=g)
    wd, d = wide.to(DEV), lambda a: a.to(DEV)
    qd, kd, vd, gd, _ = torch.split(wd, [H * dk, H * dk, H * dv, H * dv, 5], dim=1)
    ones = torch.ones(H * dv)
    for kind in ("delta", "memory"):
        S, n_, m_ = d(S0), d(n0), d(m0)
        if kind == "delta":
            out = delta_rule(qd, kd, vd, d(za), d(zb), d(pa), d(pb), d(ones[:dv]), 1e-4, gd, S, st, H, H, dk, dv).cpu()
        else:
            out = matrix_memory(qd, kd, vd, d(za), d(zb), d(pa), d(pb), 5.0, d(ones), 1e-4, gd, S, n_, m_, st, H, dk, dv).cpu()
        at = 0
        for row, p0, n in segs:
            if row in (0, 1, 17, segments - 1, segments, segments + 3):
                D = torch.float64
                Sr = S0[row].to(D) if p0 else torch.zeros(H, dk, dv, dtype=D)
                nr, mr = (n0[row].to(D), m0[row].to(D)) if p0 else (torch.zeros(H, dk, dtype=D), torch.zeros(H, dtype=D))
                for t in range(at, at + n):
                    qt, kt, vt = (x[t].to(D).view(H, -1) for x in (q, k, v))
                    if kind == "delta":
                        qt, kt = O.unit_length(qt), O.unit_length(kt)
                        Sr = torch.exp(-pb * O.softplus(za[t] + pa)).to(D)[:, None, None] * Sr
                        u = torch.sigmoid(zb[t].to(D))[:, None] * (vt - torch.einsum("hkv,hk->hv", Sr, kt))
                        Sr = Sr + kt[:, :, None] * u[:, None, :]
                        o, act = torch.einsum("hkv,hk->hv", Sr, qt * dk ** -0.5), O.silu
                    else:
                        li, lf = 5.0 * torch.tanh((zb[t].to(D) + pb) / 5.0), -O.softplus(-5.0 * torch.tanh((za[t].to(D) + pa) / 5.0))
                        top = torch.maximum(lf + mr, li)
                        keep, take, mr = torch.exp(lf + mr - top), torch.exp(li - top), top
                        Sr = keep[:, None, None] * Sr + take[:, None, None] * kt[:, :, None] * vt[:, None, :]
                        nr = keep[:, None] * nr + take[:, None] * kt
                        den = torch.maximum((nr * qt * dk ** -0.5).sum(1).abs(), torch.exp(-mr)) + 1e-6
                        o, act = torch.einsum("hkv,hk->hv", Sr, qt * dk ** -0.5) / den[:, None], torch.sigmoid
                    ref = O.unit_rms(o, 1e-4).reshape(-1) * act(gate[t].to(D))
                    assert B.rel_err(out[t], ref) < 1e-3, (kind, row, t - at)
                assert B.rel_err(S[row], Sr) < 1e-4, (kind, row)
                if kind == "memory":
                    assert B.rel_err(n_[row], nr) < 1e-4 and B.rel_err(m_[row], mr) < 1e-5, row
            at += n


def _cached_step(H, G, d, rot, dtype, g, bs=16):
    """A mixed step (prompt portions that start inside a sequence, decoded tokens) with its cache filled by the store kernel; the queries
    come back from the same call as all tokens' queries."""
    from swiftllm_b200.worker.kernels import window_attn as WA
    lens, new = [300, 77, 1, 200, 130], [150, 40, 1, 1, 1]
    nb = sum((n + bs - 1) // bs for n in lens)
    perm = torch.randperm(nb, generator=g).tolist()
    table = torch.full((5, 32), -1, dtype=torch.int32)
    for s, n in enumerate(lens):
        for b in range((n + bs - 1) // bs):
            table[s, b] = perm.pop()
    table = table.to(DEV)
    cache = torch.full((nb, 2, bs, WA.shared_row_width(G, d, rot)), 3.0, dtype=dtype, device=DEV)
    seq, pos = [s for s, n in enumerate(lens) for _ in range(n)], [p for n in lens for p in range(n)]
    st_all = types.SimpleNamespace(token_seq_ids=torch.tensor(seq, dtype=torch.int32, device=DEV),
                                   token_positions=torch.tensor(pos, dtype=torch.int32, device=DEV))
    k = (torch.randn(sum(lens), G * d + 3, generator=g) * torch.linspace(0.2, 4.0, G * d + 3)).to(dtype)
    q = torch.randn(sum(lens), H * d + 5, generator=g).to(dtype)
    qn, kn = 1 + 0.4 * torch.randn(H * d, generator=g), 1 + 0.4 * torch.randn(G * d, generator=g)
    freq = torch.tensor([40.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
    ang = torch.tensor(pos, dtype=torch.float64)[:, None] * freq
    cos, sin = (torch.cos(ang).float().to(DEV), torch.sin(ang).float().to(DEV)) if rot else (None, None)
    qs = WA.whole_norm_rope_store(q.to(DEV)[:, 5:], k.to(DEV)[:, 3:], qn.to(DEV), kn.to(DEV), 1e-4, cos, sin, cache, 1, table, st_all, H, G,
                                  d, rot, True)
    first = [0]
    for n in lens:
        first.append(first[-1] + n)
    tok_seq = [s for s, n in enumerate(new) for _ in range(n)]
    tok_pos = [lens[s] - n + p for s, n in enumerate(new) for p in range(n)]
    st = types.SimpleNamespace(token_seq_ids=torch.tensor(tok_seq, dtype=torch.int32, device=DEV),
                               token_positions=torch.tensor(tok_pos, dtype=torch.int32, device=DEV), num_prefill_tokens=191)
    rows = torch.tensor([first[s] + p for s, p in zip(tok_seq, tok_pos)])
    qf = O.rotate((O.unit_rms(q[:, 5:].float(), 1e-4) * qn).view(-1, H, d), pos, {"dims": rot, "base": 40.0})
    kf = O.rotate((O.unit_rms(k[:, 3:].float(), 1e-4) * kn).view(-1, G, d), pos, {"dims": rot, "base": 40.0})
    return cache, table, qs[rows.to(DEV)], qf[rows], kf, k[:, 3:].float().view(-1, G, d), st, tok_seq, tok_pos, first


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,rot,window", [(4, 2, 32, 8, 64), (8, 1, 64, 64, 50), (6, 3, 48, 24, 33), (10, 10, 16, 16, 7), (6, 2, 128, 64, 0),
                                              (6, 2, 128, 128, 90), (12, 1, 48, 40, 60), (32, 2, 112, 16, 90), (18, 1, 32, 0, 25), (3, 1, 80, 6, 1),
                                              (6, 2, 10, 4, 20), (5, 5, 7, 2, 9), (2, 1, 200, 100, 30)])
def test_attention_over_turned_shared_keys(dtype, H, G, d, rot, window):
    """Both attention kernels on the same step (the CUDA-core one is forced for the second run) and a plain loop: norms over the whole
    projections, partial rotation, un-normed keys as values, learned sinks, one gate per head."""
    from swiftllm_b200.worker.kernels import window_attn as WA
    g = torch.Generator().manual_seed(H * d + window)
    cache, table, qs, qf, kf, vf, st, tok_seq, tok_pos, first = _cached_step(H, G, d, rot, dtype, g)
    T = len(tok_seq)
    gate, sinks = torch.randn(T, H + 5, generator=g).to(dtype), torch.linspace(-6.0, 8.0, H)
    opt = WA.AttnOptions(gate_per_head=True, shared_kv=True, key_turned=rot, sinks=sinks.to(DEV))
    scale, outs = 1.2 / math.sqrt(d), []
    for simt in (False, True):
        old = WA.set_simt(simt)
        try:
            out = torch.zeros(T, H * d, dtype=dtype, device=DEV)
            WA.window_attention(qs, gate.to(DEV)[:, 5:], cache, 1, table, st, out, H, G, d, d, 0, window, scale, False, None, None, opt)
            outs.append(out.float().cpu())
        finally:
            WA.set_simt(old)
    assert B.rel_err(outs[0], outs[1]) < (1e-5 if dtype == torch.float32 else 1.5e-2)
    assert bool((cache[:, 0] == 3.0).all())                          # the other slot is untouched
    picked = sorted({r for r in range(T) if tok_pos[r] in (0, 37, window - 1, window, window + 1)} | {0, 100, 149, 160, T - 3, T - 2, T - 1})
    for r in picked:
        s, p = tok_seq[r], tok_pos[r]
        js = torch.tensor([first[s] + j for j in range(p + 1) if window == 0 or p - j < window])
        for h in range(H):
            gg = h // (H // G)
            sc = torch.cat([(kf[js, gg] @ qf[r, h]) * scale, sinks[h:h + 1]])
            ref = (torch.softmax(sc, dim=0)[:-1] @ vf[js, gg]) * torch.sigmoid(gate[r, 5 + h].float())
            for o in outs:
                assert B.rel_err(o[r].view(H, d)[h], ref) < (2e-4 if dtype == torch.float32 else 3e-2), (r, s, p, h)


# ---------------------------------------------------------------- the worker
@pytest.mark.parametrize("name", sorted(C.SINGLE))
def test_single_mechanisms(name):
    B.case_whole_prompt(_make, C.SINGLE[name], n=17)


def test_whole_prompt():
    B.case_whole_prompt(_make, C.full_config())


def test_prefill_vs_decode():
    B.case_prefill_vs_decode(_make, C.full_config())


def test_portions():
    B.case_portions(_make, C.full_config())


def test_mixed_batch():
    B.case_mixed_batch(_make, C.full_config())


def test_blocks_and_rows_reused():
    B.case_blocks_and_rows_reused(_make, C.full_config())


def test_long_decode():
    B.case_long_decode(_make, C.full_config())


def test_greedy_generation():
    B.case_greedy_generation(_make, C.config([(C.delta(), C.moe()), (C.attn(), C.moe()), (C.mlstm(), None)]))


@pytest.mark.parametrize("case", C.PROBES)
def test_probes(case):
    getattr(C, "case_" + case)(_make)


def _tc_config():
    """Head sizes that are multiples of 16 (the shapes the 16-bit tensor-core attention kernels take), sequences over several key tiles
    and windows."""
    return C.config([(C.attn(heads=8, kv_heads=2, dim=32, rot=16, window=40), C.moe(ff=48)),
                     (C.delta(heads=4, kv_heads=2, dim=40, vdim=24, conv=4), C.moe(ff=32)),
                     (C.mlstm(heads=4, dim=24, vdim=48, cap=8.0), None),
                     (C.attn(heads=6, kv_heads=6, dim=64, rot=64, window=70, base=1000.0), None)], width=64, streams=4)


def test_bfloat16_worker_close_to_fp32_oracle():
    """bf16 projections / cache, fp32 streams, norms, attention weights, gates and states: the logits stay within bf16 rounding of the
    fp32 oracle on the same weights, and do not depend on how the prompt was cut beyond that.  The corrections are further apart than
    the scores, so that rounding cannot turn a choice of experts."""
    for cfg, n, cuts, bs, nb in ((C.full_config(eps=1e-2, mult=0.1), 33, [5, 2, 1, 1, 24], 4, 40), (_tc_config(), 150, [61, 4, 64, 2, 1, 1, 17], 8, 60)):
        t = O.random_tensors(cfg, seed=11)
        for name in t:
            if name.endswith("correction"):
                t[name] = (-1.25 * torch.randperm(len(t[name]), generator=torch.Generator().manual_seed(3))).to(t[name].dtype)
        toks = B.tokens_for(cfg, n, 11)
        ref = O.forward(cfg, t, toks)[-40:]
        m = B.make_worker(_make, cfg, t, dtype="bfloat16", block_size=bs, num_blocks=nb)
        whole = B.run_portions(m, toks, 0, [n])[-40:]
        cut = B.run_portions(m, toks, 1, cuts)[-40:]
        assert B.rel_err(whole, ref) < 2e-2 and B.rel_err(cut, ref) < 2e-2 and B.rel_err(cut, whole) < 2e-2


def test_cuda_graph_decode_matches_eager():
    """Pure-decode steps replayed from a CUDA graph: state rows, convolution tails and the previous token move on inside the graph exactly
    as in eager steps."""
    cfg = C.config([(C.delta(), C.moe()), (C.attn(), C.moe()), (C.mlstm(), None)], width=64)
    t = O.random_tensors(cfg, seed=13)
    t["head"] = (t["head"].float() * 4).to(t["head"].dtype)
    prompts = [B.tokens_for(cfg, n, 70 + k) for k, n in enumerate((7, 3, 12))]
    runs = []
    for graph in (False, True):
        m = B.make_worker(_make, cfg, t, dtype="float32", block_size=4, num_blocks=40)
        m.engine_config.use_cuda_graph = graph
        last = m.forward(prompts, [0, 1, 2], [])
        lens, toks = [len(p) for p in prompts], [list(last)]
        for step in range(9):
            live = [0, 1, 2] if step < 6 else [0, 2]
            for i in live:
                lens[i] += 1
            out = m.forward([[toks[-1][i]] for i in live], live, [lens[i] for i in live])
            nxt = list(toks[-1])
            for i, o in zip(live, out):
                nxt[i] = o
            toks.append(nxt)
        assert m.gpu_block_manager.check_device_status() >= 0
        runs.append(toks)
    assert runs[0] == runs[1]
    assert [s[0] for s in runs[0]] == B.oracle_greedy(cfg, t, prompts[0], 10)


def test_memory_profile_then_generation():
    """The entry point's order of calls: the forged profiling batch (no cache, no state tensors yet) sizes the pool, then the worker
    generates through the scheduler loop as the oracle does."""
    from swiftllm_b200.worker.chunking import run_greedy
    cfg = C.config([(C.attn(), C.moe()), (C.delta(), None), (C.mlstm(), C.moe())])
    t = O.random_tensors(cfg, seed=19)
    t["head"] = (t["head"].float() * 4).to(t["head"].dtype)
    import swiftllm_b200
    from swiftllm_b200.worker.weight import dict_getter
    ec = swiftllm_b200.EngineConfig(model_path="", use_dummy=False, block_size=4, gpu_mem_utilization=0.5, num_cpu_blocks=0,
                                    max_seqs_in_block_table=4, max_blocks_per_seq=16, max_batch_size=4, max_tokens_in_batch=64,
                                    dtype="float32")
    m = swiftllm_b200.create_model(ec, swiftllm_b200.registry.model_config_from_dict(cfg))
    m.load_weights(dict_getter(t))
    n = m.profile_num_blocks()
    assert n == 4 * 16                                    # capped by the block table
    m.init_kvcache_and_swap(n)
    prompts = [B.tokens_for(cfg, k, 80 + k) for k in (9, 2, 14)]
    got = run_greedy(m, prompts, new_tokens=4, max_tokens_in_step=10, max_chunk=5, seq_ids=[1, 3, 0])
    assert got == [B.oracle_greedy(cfg, t, p, 4) for p in prompts]


def test_trace_replay_command_line(tmp_path):
    """bin/trace_run on a checkpoint folder of this design: a mixed schedule (portions beside decoded tokens, requests that end and whose
    rows, blocks and state rows are used again) in both dtypes, against the oracle run on each whole sequence."""
    import json
    import os
    import subprocess
    import numpy as np
    from safetensors.torch import save_file
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = C.config([
        (C.attn(heads=10, kv_heads=2, dim=16, rot=8, window=24), C.moe(ff=30)),
        (C.mlstm(heads=5, dim=12, vdim=20, cap=6.0), C.moe(experts=8, top=3, groups=4, keep=2)),
        (C.delta(heads=4, kv_heads=2, dim=24, vdim=16, conv=4), C.moe()),
        (C.attn(heads=3, kv_heads=3, dim=8, rot=4, window=9), None),
        (C.mlstm(heads=1, dim=48, vdim=16, cap=16.0), None),
    ], width=72, vocab=131, eps=1e-3, embed_scale=2.5, streams=2)
    t = O.random_tensors(cfg, seed=22)
    model_dir = tmp_path / "model"
    model_dir.mkdir()
    (model_dir / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in t.items()}, str(model_dir / "model.safetensors"))
    reqs = {k: B.tokens_for(cfg, n, s) for s, (k, n) in enumerate((("a", 70), ("b", 41), ("c", 17), ("d", 5), ("e", 30)))}
    ref = {k: O.forward(cfg, t, v).numpy() for k, v in reqs.items()}
    plan = [[("a", 33), ("b", 2)], [("a", 31), ("b", 30), ("c", 17)], [("a", 1), ("b", 1), ("d", 5)], [("a", 1), ("b", 1), ("e", 3)],
            [("a", 2), ("b", 7), ("e", 27)], [("a", 2)]]
    for dtype, limit in (("float32", 1e-4), ("bfloat16", 5e-2)):
        out = tmp_path / dtype
        out.mkdir()
        at, lines, rows = {k: 0 for k in reqs}, [], []
        for n, step in enumerate(plan):
            entries, end, rr = [], [], []
            for k, c in step:
                lo, hi = at[k], at[k] + c
                entries.append({"id": k, "tokens": reqs[k][lo:hi], "want": list(range(0, c, 2))})
                rr += [(k, p) for p in range(lo, hi, 2)]
                at[k] = hi
                if hi == len(reqs[k]):
                    end.append(k)
            lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
            rows.append(rr)
        p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(model_dir), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "192"], input="\n".join(lines) + "\n", capture_output=True, text=True, cwd=root)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {n}" for n in range(len(plan))]
        errs = []
        for n, rr in enumerate(rows):
            got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(rr), -1)
            for j, (k, pos) in enumerate(rr):
                errs.append(np.sqrt(((got[j] - ref[k][pos]) ** 2).mean() / (ref[k][pos] ** 2).mean()))
        assert np.sqrt(np.mean(np.square(errs))) < limit and np.median(errs) < limit / 2, (dtype, max(errs))
