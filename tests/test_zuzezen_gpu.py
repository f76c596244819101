"""GPU: the Zuzezen worker and its CUDA kernels (csrc/gla.cu; the sink of csrc/latent_attn.cu; the kept positions, distance bias,
gate per head and shared key / value rows of csrc/window_attn.cu; the per-channel gain, SiLU unit, sigmoid gate and embedding scale of
csrc/stream_ops.cu) - every kernel alone against a plain loop written here or in oracle/zuzezen.py, then the scenarios of
tests/bupozen_cases.py and tests/zuzezen_cases.py through the worker (fp32 tight, bf16 loose)."""
import math
import types

import pytest
import torch

import bupozen_cases as B
import zuzezen_cases as C
from oracle import zuzezen as O
from test_bupozen_gpu import _make, _paged
from test_buzarax_gpu import _schedule, _step

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def _tol(dtype):
    return 1e-5 if dtype == torch.float32 else 1.2e-2


# ---------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [48, 50, 1000, 4096, 8200])
def test_post_norm_with_a_gain_per_channel(dtype, width):
    from swiftllm_b200.worker.kernels.stream_ops import postnorm_add_mix
    g = torch.Generator().manual_seed(width)
    x, y, gain = torch.randn(9, width, generator=g) * 3, torch.randn(9, width, generator=g).to(dtype), torch.randn(width, generator=g)
    for gn in (gain, gain[:1]):
        xd, h = x.to(DEV), torch.zeros(9, width, dtype=dtype, device=DEV)
        postnorm_add_mix(xd, y.to(DEV), gn.to(DEV), 1e-3, h)
        ref = x + O.unit_rms(y.float(), 1e-3) * gn
        assert B.rel_err(xd, ref) < 1e-6 and B.rel_err(h.float(), ref) < _tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [64, 70, 33])
def test_silu_unit_and_sigmoid_gate(dtype, n):
    from swiftllm_b200.worker.kernels.stream_ops import sigmoid_gate_inplace, silu_glu
    g = torch.Generator().manual_seed(n)
    u = (torch.randn(19, 2 * n, generator=g) * 2).to(dtype)
    assert B.rel_err(silu_glu(u.to(DEV)).float(), O.silu(u[:, :n].float()) * u[:, n:].float()) < _tol(dtype)
    x, wide = torch.randn(19, n, generator=g).to(dtype), (torch.randn(19, n + 12, generator=g) * 3).to(dtype)
    for off in (4, 5):
        xd = x.to(DEV)
        sigmoid_gate_inplace(xd, wide.to(DEV)[:, off:off + n])
        assert B.rel_err(xd.float(), x.float() * torch.sigmoid(wide[:, off:off + n].float())) < _tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_scaled_embedding(dtype):
    from swiftllm_b200.worker.kernels.stream_ops import embed_pair_hash
    e = torch.randn(31, 40, generator=torch.Generator().manual_seed(4)).to(dtype)
    toks = torch.tensor([3, 30, 0, 7], dtype=torch.int32)
    st = _step([(1, 0, 4)])
    x, h = embed_pair_hash(toks.to(DEV), st, None, e.to(DEV), None, 0, 0, 0, scale=2.7)
    ref = e[toks.long()].float() * 2.7
    assert B.rel_err(x, ref) < 1e-6 and B.rel_err(h.float(), ref) < _tol(dtype)


GLA_SHAPES = [(3, 10, 6, 4.0), (1, 37, 70, 16.0), (2, 1, 2, 1.0), (5, 64, 64, 8.0), (2, 130, 33, 16.0), (3, 96, 160, 16.0), (2, 128, 128, 2.0),
              (1, 300, 20, 16.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [True, False])
@pytest.mark.parametrize("H,dk,dv,tau", GLA_SHAPES)
def test_gated_linear_attention_state_through_portions(dtype, H, dk, dv, tau, prompt):
    """Two sequences in rows 2 and 0 of the state tensor (which starts full of junk), fed in portions down to one token; some channels
    forget within a token (their decays cannot be folded into the staged vectors), some hardly at all.  `prompt`: every segment as a
    prompt portion; otherwise one-token segments go through the launch of single decoded tokens."""
    from swiftllm_b200.worker.kernels.gla import gated_linear_attention
    g = torch.Generator().manual_seed(H * dk + dv)
    lens, rows = [300, 37], [2, 0]
    plan = [[(0, 1), (1, 2)], [(0, 2), (1, 1)], [(0, 217), (1, 1)], [(1, 33)], [(0, 79)], [(0, 1)]]
    q, k = ([torch.randn(n, H * dk, generator=g).to(dtype) for n in lens] for _ in range(2))
    v, gate = ([torch.randn(n, H * dv, generator=g).to(dtype) for n in lens] for _ in range(2))
    z = [torch.randn(n, H * dk, generator=g) * 2 for n in lens]
    bias = torch.randn(H * dk, generator=g) + 2.0
    bias[::5] = -25.0 * tau
    bias[1::5] = 9.0
    z[0][100:140] = 8.0                                    # a stretch in which nothing decays steeply except the forgetful channels
    w = 1 + 0.3 * torch.randn(dv, generator=g)
    ref = []
    for s in range(2):
        n = lens[s]
        alpha = torch.exp(torch.nn.functional.logsigmoid((z[s] + bias).double()) / tau).view(n, H, dk)
        o = O.gla_states((q[s].double() * dk ** -0.5).view(n, H, dk), k[s].double().view(n, H, dk), v[s].double().view(n, H, dv), alpha)
        ref.append(((O.unit_rms(o, 1e-5) * w.double()).reshape(n, H * dv) * O.silu(gate[s].double())).float())
    state = torch.full((3, H, dk, dv), 1e4, device=DEV)
    got = [[] for _ in lens]
    for segs in _schedule(lens, plan):
        segs = sorted(segs, key=lambda e: e[2] == 1)       # prompt portions first
        st = _step([(rows[s], p0, n) for s, p0, n in segs])
        long = [n for _, _, n in segs if n > 1 or prompt]
        st.num_prefill_seqs, st.num_prefill_tokens, st.max_prefill_len = len(long), sum(long), max(long, default=0)
        cat = lambda parts: torch.cat([parts[s][p0:p0 + n] for s, p0, n in segs]).to(DEV)
        out = gated_linear_attention(cat(q), cat(k), cat(v), cat(z), bias.to(DEV), tau, w.to(DEV), 1e-5, cat(gate), state, st, H, dk, dv)
        out, at = out.float().cpu(), 0
        for s, p0, n in segs:
            got[s].append((p0, out[at:at + n])); at += n
    for s in range(2):
        full = torch.cat([o for _, o in sorted(got[s], key=lambda e: e[0])])
        assert B.rel_err(full, ref[s]) < (2e-5 if dtype == torch.float32 else 1.2e-2), s
        row_err = (full - ref[s]).pow(2).mean(-1).sqrt() / ref[s].pow(2).mean(-1).sqrt()
        assert float(row_err.max()) < (5e-4 if dtype == torch.float32 else 3e-2), s


def test_gated_linear_attention_prompt_and_decode_in_one_step():
    """Prompt portions beside single decoded tokens (two launch shapes in one call), columns of a wider matrix as inputs."""
    from swiftllm_b200.worker.kernels.gla import gated_linear_attention
    H, dk, dv, tau = 3, 48, 80, 16.0
    g = torch.Generator().manual_seed(7)
    segs = [(4, 0, 90), (1, 33, 17), (0, 5, 1), (3, 200, 1), (2, 0, 1)]
    T = sum(n for _, _, n in segs)
    wide = torch.randn(T, 2 * H * dk + 2 * H * dv + 5, generator=g)
    q, k, v, gate, _ = torch.split(wide, [H * dk, H * dk, H * dv, H * dv, 5], dim=1)
    z, bias, w = torch.randn(T, H * dk, generator=g), torch.randn(H * dk, generator=g), torch.ones(dv)
    state0 = torch.randn(5, H, dk, dv, generator=g)
    st = _step(segs)
    st.num_prefill_seqs, st.num_prefill_tokens, st.max_prefill_len = 2, 107, 90
    state = state0.to(DEV)
    wd = wide.to(DEV)
    qd, kd, vd, gd, _ = torch.split(wd, [H * dk, H * dk, H * dv, H * dv, 5], dim=1)
    out = gated_linear_attention(qd, kd, vd, z.to(DEV), bias.to(DEV), tau, w.to(DEV), 1e-6, gd, state, st, H, dk, dv).cpu()
    at = 0
    for row, p0, n in segs:
        S = state0[row].double().clone() if p0 > 0 else torch.zeros(H, dk, dv, dtype=torch.float64)
        for t in range(at, at + n):
            alpha = torch.exp(torch.nn.functional.logsigmoid((z[t] + bias).double()) / tau).view(H, dk, 1)
            S = alpha * S + k[t].double().view(H, dk, 1) * v[t].double().view(H, 1, dv)
            o = (S * (q[t].double() * dk ** -0.5).view(H, dk, 1)).sum(1)
            ref = (O.unit_rms(o, 1e-6)).reshape(-1) * O.silu(gate[t].double())
            assert B.rel_err(out[t], ref) < 1e-4, (row, t)
        assert B.rel_err(state[row], S) < 1e-5
        at += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,r,dr,bs", [(3, 24, 6, 4), (20, 64, 16, 16), (5, 128, 32, 8), (16, 512, 64, 16)])
def test_latent_attention_with_learned_sink(dtype, H, r, dr, bs):
    """Sinks from far below to far above the scores, long and one-key contexts, few queries (key splits) and many (none)."""
    from swiftllm_b200.worker.kernels.latent_attn import latent_attention
    n, scale = 700, 0.3
    g = torch.Generator().manual_seed(H + r)
    cache, bt = _paged([n], bs, r + dr, dtype, seed=r)
    rows = (torch.randn(n, r + dr, generator=g) * 0.4).to(dtype)
    for p in range(n):
        cache[int(bt[0, p // bs]), 2, p % bs] = rows[p]
    sink = torch.linspace(-12.0, 12.0, H)
    for positions in ([0, 1, 63, 64, 699], list(range(0, 700, 2))):
        T = len(positions)
        q_lat, q_rot = torch.randn(T, H, r, generator=g).to(dtype), torch.randn(T, H, dr, generator=g).to(dtype)
        st = types.SimpleNamespace(token_seq_ids=torch.zeros(T, dtype=torch.int32, device=DEV),
                                   token_positions=torch.tensor(positions, dtype=torch.int32, device=DEV))
        out = torch.empty(T, H, r, dtype=dtype, device=DEV)
        latent_attention(q_lat.to(DEV), q_rot.to(DEV), None, cache.to(DEV), 2, bt.to(DEV), st, out, 0, 0, scale, None, None,
                         sink.to(DEV))
        qa, rf = torch.cat([q_lat, q_rot], dim=2).float(), rows.float()
        for t in list(range(T))[:: max(1, T // 8)]:
            p = positions[t]
            s = (qa[t] @ rf[:p + 1].T) * scale
            wt = torch.softmax(torch.cat([s, sink[:, None]], dim=1), dim=1)[:, :p + 1]
            ref = wt @ rf[:p + 1, :r]
            got = out[t].float().cpu()
            err = (got - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean(-1).sqrt()
            assert float(err.max()) < (1e-4 if dtype == torch.float32 else 3e-2), (p, err)


def _windowed_step(H, G, d, dtype, g, bs=16):
    """A mixed step (prompt portions that start inside a sequence, decoded tokens) with its cache filled by the store kernel."""
    from swiftllm_b200.worker.kernels import window_attn as WA
    lens, new = [300, 77, 1, 200, 130], [150, 40, 1, 1, 1]
    nb = sum((n + bs - 1) // bs for n in lens)
    perm = torch.randperm(nb, generator=g).tolist()
    table = torch.full((5, 32), -1, dtype=torch.int32)
    for s, n in enumerate(lens):
        for b in range((n + bs - 1) // bs):
            table[s, b] = perm.pop()
    table = table.to(DEV)
    width = WA.shared_row_width(G, d)
    cache = torch.full((nb, 2, bs, width), 3.0, dtype=dtype, device=DEV)
    st_all = types.SimpleNamespace(token_seq_ids=torch.tensor([s for s, n in enumerate(lens) for _ in range(n)], dtype=torch.int32, device=DEV),
                                   token_positions=torch.tensor([p for n in lens for p in range(n)], dtype=torch.int32, device=DEV))
    k = (torch.randn(sum(lens), G * d + 3, generator=g) * torch.linspace(0.2, 4.0, G * d + 3)).to(dtype)
    WA.shared_kv_store(k.to(DEV)[:, 3:], cache, 1, table, st_all, G, d, 1e-4)
    tok_seq = [s for s, n in enumerate(new) for _ in range(n)]
    tok_pos = [lens[s] - n + p for s, n in enumerate(new) for p in range(n)]
    st = types.SimpleNamespace(token_seq_ids=torch.tensor(tok_seq, dtype=torch.int32, device=DEV),
                               token_positions=torch.tensor(tok_pos, dtype=torch.int32, device=DEV), num_prefill_tokens=191)
    first = [0]
    for n in lens:
        first.append(first[-1] + n)
    return cache, table, k[:, 3:].float().view(-1, G, d), st, tok_seq, tok_pos, first


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,window,keep", [(4, 2, 32, 64, 4), (8, 1, 64, 50, 0), (6, 3, 48, 33, 40), (10, 10, 16, 7, 1), (6, 2, 128, 1000, 5),
                                               (12, 1, 48, 60, 2), (32, 2, 112, 90, 3), (18, 1, 32, 25, 4), (3, 1, 80, 1, 2), (6, 2, 10, 20, 3), (5, 5, 7, 9, 2), (2, 1, 200, 30, 6)])
def test_window_attention_whose_values_are_its_keys(dtype, H, G, d, window, keep):
    """Both attention kernels on the same step (the CUDA-core one is forced for the second run) and a plain loop: kept first
    positions, distance bias, norm of keys and queries, un-normed keys as values, one gate per head."""
    from swiftllm_b200.worker.kernels import window_attn as WA
    g = torch.Generator().manual_seed(H * d + window)
    cache, table, kf, st, tok_seq, tok_pos, first = _windowed_step(H, G, d, dtype, g)
    T = len(tok_seq)
    q, gate = torch.randn(T, H * d, generator=g).to(dtype), torch.randn(T, H + 5, generator=g).to(dtype)
    qn = 1 + 0.3 * torch.randn(d, generator=g)
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)])
    opt = WA.AttnOptions(q_norm=qn.to(DEV), prenorm_eps=1e-4, slopes=slopes.to(DEV), keep_first=keep, gate_per_head=True, shared_kv=True)
    scale, outs = 2.0 / math.sqrt(d), []
    for simt in (False, True):
        old = WA.set_simt(simt)
        try:
            out = torch.zeros(T, H * d, dtype=dtype, device=DEV)
            WA.window_attention(q.to(DEV), gate.to(DEV)[:, 5:], cache, 1, table, st, out, H, G, d, d, 0, window, scale, False, None, None, opt)
            outs.append(out.float().cpu())
        finally:
            WA.set_simt(old)
    assert B.rel_err(outs[0], outs[1]) < (1e-5 if dtype == torch.float32 else 1.5e-2)
    assert bool((cache[:, 0] == 3.0).all())                          # the other slot is untouched
    qf = O.unit_rms(q.float().view(T, H, d), 1e-4) * qn
    kn = O.unit_rms(kf, 1e-4)
    picked = sorted({r for r in range(T) if tok_pos[r] in (0, 37, keep, keep + window - 1, keep + window, window)} | {0, 100, 149, 160, T - 3, T - 2, T - 1})
    for r in picked:
        s, p = tok_seq[r], tok_pos[r]
        js = torch.tensor([j for j in range(p + 1) if p - j < window or j < keep])
        keys, vals = kn[first[s] + js], kf[first[s] + js]
        for h in range(H):
            gg = h // (H // G)
            sc = (keys[:, gg] @ qf[r, h]) * scale - slopes[h] * (p - js).float()
            ref = (torch.softmax(sc, dim=0) @ vals[:, gg]) * torch.sigmoid(gate[r, 5 + h].float())
            for o in outs:
                assert B.rel_err(o[r].view(H, d)[h], ref) < (1e-4 if dtype == torch.float32 else 2.5e-2), (r, s, p, h)


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
    B.case_greedy_generation(_make, C.config([(C.gla(), C.dense()), (C.attn(), C.dense()), (C.latent(), None)]))


@pytest.mark.parametrize("case", ["window_edges", "kept_keys_far_away", "values_are_unnormed_keys", "far_latent", "sink",
                                  "first_tokens_and_block_borders", "rotation_far_out", "slow_channels_remember", "state_rows_used_again"])
def test_probes(case):
    getattr(C, "case_" + case)(_make)


def _tc_config():
    """Head sizes that are multiples of 16 (the shapes the 16-bit tensor-core attention kernels take), sequences over several key
    tiles and windows."""
    return C.config([(C.latent(heads=6, dim=32, rot_dim=32, vdim=16, kv_rank=96, base=1000.0, scaling=(4.0, 64, 8.0, 1.0)), C.dense(ff=96)),
                     (C.attn(heads=8, kv_heads=2, dim=32, window=40, keep=5), C.dense(ff=80)),
                     (C.gla(heads=4, dim=40, vdim=24, tau=16.0), None),
                     (C.latent(heads=20, dim=16, rot_dim=16, vdim=32, kv_rank=48), None),
                     (C.attn(heads=6, kv_heads=6, dim=64, window=70, keep=1), None)], width=64)


def test_bfloat16_worker_close_to_fp32_oracle():
    """bf16 projections / cache, fp32 stream, norms, attention weights, decays and states: the logits stay within bf16 rounding of the
    fp32 oracle on the same weights, and do not depend on how the prompt was cut beyond that."""
    for cfg, n, cuts, bs, nb in ((C.full_config(), 33, [5, 2, 1, 1, 24], 4, 40), (_tc_config(), 150, [61, 4, 64, 2, 1, 1, 17], 8, 60)):
        t = O.random_tensors(cfg, seed=11)
        toks = B.tokens_for(cfg, n, 11)
        ref = O.forward(cfg, t, toks)[-40:]
        m = B.make_worker(_make, cfg, t, dtype="bfloat16", block_size=bs, num_blocks=nb)
        whole = B.run_portions(m, toks, 0, [n])[-40:]
        cut = B.run_portions(m, toks, 1, cuts)[-40:]
        assert B.rel_err(whole, ref) < 4e-2 and B.rel_err(cut, ref) < 4e-2 and B.rel_err(cut, whole) < 3e-2


def test_cuda_graph_decode_matches_eager():
    """Pure-decode steps replayed from a CUDA graph: the linear attention's state rows move on inside the graph exactly as in eager
    steps."""
    cfg = C.config([(C.gla(), C.dense()), (C.attn(), C.dense()), (C.latent(), None)], width=64)
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
    """The entry point's order of calls: the forged profiling batch (no cache, no state tensors yet) sizes the pool, then the
    worker generates through the scheduler loop as the oracle does."""
    from swiftllm_b200.worker.chunking import run_greedy
    cfg = C.config([(C.attn(), C.dense()), (C.gla(), None), (C.latent(), C.dense())])
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
    """bin/trace_run on a checkpoint folder of this design: a mixed schedule (portions beside decoded tokens, requests that end
    and whose rows, blocks and state rows are used again) in both dtypes, against the oracle run on each whole sequence."""
    import json
    import os
    import subprocess
    import numpy as np
    from safetensors.torch import save_file
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = C.config([
        (C.attn(heads=10, kv_heads=2, dim=16, window=24, keep=3), C.dense(ff=60)),
        (C.latent(heads=4, dim=16, rot_dim=16, vdim=24, kv_rank=48, base=5000.0, scaling=(8.0, 32, 6.0, 0.7)), C.dense(ff=50)),
        (C.gla(heads=5, dim=12, vdim=20, tau=8.0), C.dense(ff=24)),
        (C.attn(heads=3, kv_heads=3, dim=8, window=9, keep=2), None),
        (C.gla(heads=1, dim=48, vdim=16, tau=16.0), None),
    ], width=72, vocab=131, eps=1e-6, embed_scale=2.5)
    # weights under which no position is ill-conditioned (a head's output that nearly cancels is blown up by the norm behind it)
    t = O.random_tensors(cfg, seed=22, rank=7)
    model_dir = tmp_path / "model"
    model_dir.mkdir()
    (model_dir / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in t.items()}, str(model_dir / "model.safetensors"))
    reqs = {k: B.tokens_for(cfg, n, s) for s, (k, n) in enumerate((("a", 70), ("b", 41), ("c", 17), ("d", 5), ("e", 30)))}
    ref = {k: O.forward(cfg, t, v).numpy() for k, v in reqs.items()}
    plan = [[("a", 33), ("b", 2)], [("a", 31), ("b", 30), ("c", 17)], [("a", 1), ("b", 1), ("d", 5)], [("a", 1), ("b", 1), ("e", 3)],
            [("a", 2), ("b", 7), ("e", 27)], [("a", 2)]]
    for dtype, limit in (("float32", 1e-4), ("bfloat16", 4e-2)):
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
                assert errs[-1] < 2.5 * limit, (dtype, n, k, pos, errs[-1])         # no single position far off ...
        assert np.sqrt(np.mean(np.square(errs))) < limit, dtype                     # ... and all of them within rounding
