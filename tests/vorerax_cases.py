"""Configurations and scenarios for the Vorerax worker (swiftllm_b200.worker.vorerax_model) against the plain restatement of the design in
oracle/vorerax.py.  The schedule scenarios (whole prompts, decoding, portions, mixed batches, reused blocks and rows, greedy
generation) are the ones of tests/bupozen_cases.py; here are the design's own configurations and the scenarios whose weights are made
so that one particular fault would show.  They run on the CPU (kernels replaced by tests/cpu_shim.py) and on a GPU (the CUDA kernels):
tests/test_vorerax_cpu.py and tests/test_vorerax_gpu.py call them with the `make` factory of their world.

All configurations are small and deliberately irregular: head sizes that are not multiples of 16 or of each other, value sizes unrelated
to key sizes, one / several / as many key heads as query heads, no / partial / full rotation with bands that stretch all, some or none of
the pairs, windows of 1, 5, 7 and more positions than the sequence has, convolutions of 1 to 5 taps, one to five streams and none,
groups of one, two and more experts, layers of every type with and without feed-forward."""
import math

import torch

from bupozen_cases import TOL, make_worker, rel_err, run_portions, tokens_for
from oracle import vorerax as O

BANDS = {"factor": 3.0, "low": 0.8, "high": 2.5, "original": 40}


def attn(heads=6, kv_heads=2, dim=10, window=7, base=100.0, rot=6, scaling=BANDS, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else 1.4 / math.sqrt(dim),
         "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(scaling)
    if not rot:
        del m["rot"]
    if window:
        m["mask"] = {"size": window}
    return "attention", m


def delta(heads=6, kv_heads=3, dim=10, vdim=7, conv=3):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def mlstm(heads=3, dim=10, vdim=6, cap=9.0):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def moe(experts=6, top=2, ff=20, groups=3, keep=2):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        f["router"]["groups"] = {"count": groups, "keep": keep}
    return f


def config(layers, width=44, vocab=97, eps=1e-5, mult=0.6, streams=3, embed_scale=1.75, pair=(53, 7, 11)):
    cfg = {"architecture": "Vorerax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
           "residual_mult": mult, "layers": [{"type": kind, "mixer": m, "mlp": f} for (kind, m), f in layers]}
    if streams:
        cfg["streams"] = streams
    if pair:
        cfg["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), pair))
    return cfg


def full_config(**kw):
    """Every branch at once."""
    return config([
        (delta(), moe()),
        (attn(), None),
        (mlstm(), moe(experts=5, top=3, groups=0)),
        (attn(heads=5, kv_heads=1, dim=6, rot=2, window=5, scaling=None), moe(experts=8, top=1, groups=4, keep=1, ff=9)),
        (mlstm(heads=2, dim=5, vdim=33, cap=2.0), None),
        (delta(heads=4, kv_heads=4, dim=5, vdim=33, conv=5), None),
        (attn(heads=4, kv_heads=4, dim=7, rot=0, window=0), moe(experts=12, top=5, groups=2, keep=1)),
    ], **kw)


SINGLE = {
    "attention_experts": config([(attn(), moe())]),
    "attention_mha_plain_frequencies": config([(attn(heads=3, kv_heads=3, window=4, scaling=None), None)]),
    "attention_mqa_wide": config([(attn(heads=5, kv_heads=1, dim=70, rot=36, window=3), moe())]),
    "attention_whole_head_turned": config([(attn(dim=8, rot=8), None)]),
    "attention_all_pairs_stretched": config([(attn(dim=12, rot=8, scaling={"factor": 4.0, "low": 900.0, "high": 1000.0, "original": 60}), None)]),
    "attention_no_pair_stretched": config([(attn(dim=12, rot=8, scaling={"factor": 4.0, "low": 1e-4, "high": 1e-3, "original": 60}), None)]),
    "attention_window_of_one": config([(attn(window=1), None)]),
    "attention_full_causal": config([(attn(window=0), None)]),
    "attention_no_rotation": config([(attn(rot=0), None)]),
    "attention_16bit_shapes": config([(attn(heads=4, kv_heads=2, dim=16, rot=8, window=6), None)]),
    "delta_experts": config([(delta(), moe())]),
    "delta_one_head_no_convolution": config([(delta(heads=1, kv_heads=1, dim=37, vdim=70, conv=1), None)]),
    "delta_many_heads_per_key_head": config([(delta(heads=12, kv_heads=2, dim=3, vdim=2, conv=2), None)]),
    "delta_long_convolution": config([(delta(heads=2, kv_heads=1, dim=20, vdim=3, conv=8), moe())]),
    "mlstm_experts": config([(mlstm(), moe())]),
    "mlstm_one_head": config([(mlstm(heads=1, dim=37, vdim=70, cap=15.0), None)]),
    "mlstm_tiny_heads": config([(mlstm(heads=7, dim=1, vdim=2, cap=1.0), moe())]),
    "no_streams": config([(mlstm(), moe()), (attn(), None)], streams=0),
    "one_stream": config([(delta(), moe())], streams=1),
    "five_streams_no_pairs": config([(attn(), moe()), (mlstm(), None)], streams=5, pair=None, embed_scale=1.0),
    "groups_of_one": config([(attn(), moe(experts=7, top=2, groups=7, keep=3))]),
    "all_experts_of_the_kept_groups": config([(attn(), moe(experts=8, top=4, groups=4, keep=2))]),
    "every_expert": config([(attn(), moe(experts=5, top=5, groups=0))]),
    "odd_width": config([(attn(), moe()), (delta(), None)], width=45),
}


# ---------------------------------------------------------------- scenarios made so that one fault shows
def _attention_probe(n, key_pos, window, H=2, G=1, d=8, width=16, vocab=32, scale=1.5, rot=0, sink=-2.0):
    """One attention layer in which every query points along one direction: the key of the marked token (token 1) points the same way,
    all other keys are orthogonal to it.  Queries and keys are normed, so `scale` alone sets how far the marked score stands above the
    others; the marked token also has its own value.  A rotated pair, if any, carries nothing."""
    cfg = config([(attn(heads=H, kv_heads=G, dim=d + rot, window=window, rot=rot, scale=scale, scaling=None), None)], width=width,
                 vocab=vocab, embed_scale=1.0, pair=None, streams=2, mult=1.0)
    t = O.random_tensors(cfg, seed=11, dtype=torch.float32)
    t["embed"] = torch.randn(vocab, width, generator=torch.Generator().manual_seed(1)) * 0.1
    t["embed"][:, 0] = 1.0                       # every query reads this constant ...
    t["embed"][:, 1] = 0.0
    t["embed"][:, 2] = 1.0                       # ... every ordinary key this one ...
    t["embed"][1, 1] = 4.0                       # ... and only the marked token carries these
    t["embed"][1, 2] = 0.0
    t["l0.norm1"] = torch.ones(width)
    q = torch.zeros(H, d + rot, width); q[:, rot:, 0] = 2.0            # all plain entries equal, direction (1, ..., 1)
    k = torch.zeros(G, d + rot, width)
    k[:, rot:, 1] = 2.0                                                # marked key: along the queries
    k[:, rot:rot + d // 2, 2], k[:, rot + d // 2:, 2] = 1.0, -1.0       # ordinary keys: orthogonal to the queries
    t["l0.mix.q"], t["l0.mix.k"] = q.reshape(-1, width), k.reshape(-1, width)
    t["l0.mix.q.norm"], t["l0.mix.k.norm"] = torch.ones(H * (d + rot)), torch.ones(G * (d + rot))
    t["l0.mix.sink"] = torch.full((H,), sink)
    toks = [2 + (i % (vocab - 2)) for i in range(n)]
    toks[key_pos] = 1
    return cfg, t, toks


def case_window_edges(make):
    """The marked key at the first positions and in the middle: queries up to the window's end see it, later ones do not - in a prompt,
    decoded, and with portions cut at, before and after the edge."""
    w = 12
    for key_pos in (0, 1, w - 1, 17):
        cfg, t, toks = _attention_probe(n=3 * w + 2, key_pos=key_pos, window=w)
        ref = O.forward(cfg, t, toks)
        for dw in (-1, 1):                                            # a window that is one position off shows
            m = {**cfg["layers"][0]["mixer"], "mask": {"size": w + dw}}
            other = {**cfg, "layers": [{**cfg["layers"][0], "mixer": m}]}
            assert rel_err(O.forward(other, t, toks), ref) > 0.02, (key_pos, dw)
        edge = key_pos + w                                            # first position whose window no longer holds the marked key
        for cuts in ([3 * w + 2], [w, w, w + 2], [edge - 1, 2, 3 * w + 1 - edge], [edge, 1, 1, 3 * w - edge], [5] + [1] * (3 * w - 3),
                     [2] * (w + w // 2) + [2]):
            model = make_worker(make, cfg, t, block_size=8, num_blocks=8)
            got = run_portions(model, toks, 1, cuts)
            assert rel_err(got, ref) < TOL, (key_pos, cuts)
            for p in (key_pos, edge - 1, edge, edge + 1):             # just inside and just outside, one by one
                assert rel_err(got[p], ref[p]) < TOL, (key_pos, cuts, p)


def case_far_key(make):
    """A marked key hundreds of positions back among keys that all score the same, in a layer without a window: across blocks, in prompt
    portions and when decoding."""
    cfg, t, toks = _attention_probe(n=390, key_pos=3, window=0, H=4, G=2, scale=3.0, rot=4)
    ref = O.forward(cfg, t, toks)
    plain = list(toks); plain[3] = 5
    assert rel_err(O.forward(cfg, t, plain)[-1], ref[-1]) > 0.02
    model = make_worker(make, cfg, t, block_size=8, num_blocks=50)
    got = run_portions(model, toks, 0, [200, 150, 38, 1, 1])
    assert rel_err(got[-8:], ref[-8:]) < TOL and rel_err(got, ref) < TOL


def case_sink(make):
    """Sinks from far below to far above the scores, different per head; the first token (alone with the sink) shows them most."""
    for sinks in ([-20.0, 3.0], [9.0, 2.0], [1.5, 30.0]):
        cfg, t, toks = _attention_probe(n=21, key_pos=4, window=15, scale=0.6)
        t["l0.mix.sink"] = torch.tensor(sinks)
        ref = O.forward(cfg, t, toks)
        for wrong in (torch.full((2,), -1e4), torch.tensor(sinks[::-1]), torch.tensor(sinks) * 0.6):      # left out, swapped, scaled
            assert rel_err(O.forward(cfg, {**t, "l0.mix.sink": wrong}, toks), ref) > 0.02
        for cuts in ([21], [1] * 21, [2, 3, 1, 15]):
            model = make_worker(make, cfg, t, block_size=8, num_blocks=6)
            assert rel_err(run_portions(model, toks, 1, cuts), ref) < TOL, (sinks, cuts)


def case_first_tokens_and_block_borders(make):
    """The marked row at the first position, at the last slot of a block and at the first slot of the next one; queries right behind
    it, in a prompt and decoded."""
    for key_pos in (0, 7, 8):
        cfg, t, toks = _attention_probe(n=20, key_pos=key_pos, window=13, rot=2)
        ref = O.forward(cfg, t, toks)
        for cuts in ([20], [key_pos + 1, 1, 1, 17 - key_pos], [2] + [1] * 18, [8, 8, 4]):
            model = make_worker(make, cfg, t, block_size=8, num_blocks=6)
            assert rel_err(run_portions(model, toks, 1, cuts), ref) < TOL, (key_pos, cuts)


def case_rotation_far_out(make):
    """Positions far beyond the original context, a band in which all three kinds of pairs occur, scores that the turned entries
    dominate: every constant of the scaling shows."""
    cfg = config([(attn(heads=2, kv_heads=1, dim=14, rot=12, window=0, base=50.0,
                        scaling={"factor": 5.0, "low": 0.7, "high": 3.0, "original": 24}, scale=1.5), None)], streams=2)
    t = O.random_tensors(cfg, seed=13, dtype=torch.float32)
    toks = tokens_for(cfg, 150, 13)
    ref = O.forward(cfg, t, toks, dtype=torch.float64)
    rot = cfg["layers"][0]["mixer"]["rot"]
    plain = [50.0 ** (-2.0 * i / 12) for i in range(6)]
    kinds = [0 if a == b else 1 if abs(a - b / 5.0) < 1e-12 else 2 for a, b in zip(O.frequencies(rot), plain)]
    assert set(kinds) == {0, 1, 2}                                    # kept, stretched and blended pairs
    for change in ({"factor": 4.0}, {"original": 30}, {"low": 0.9}, {"high": 2.0}):
        m = {**cfg["layers"][0]["mixer"], "rot": {**rot, "scaling": {**rot["scaling"], **change}}}
        assert rel_err(O.forward({**cfg, "layers": [{**cfg["layers"][0], "mixer": m}]}, t, toks, dtype=torch.float64), ref) > 2e-3, change
    model = make_worker(make, cfg, t, block_size=8, num_blocks=20)
    assert rel_err(run_portions(model, toks, 0, [70, 2, 60, 1, 1, 1, 15]), ref) < TOL


def case_norms_over_the_whole_projection(make):
    """Heads and entries of very different size: one head's size shows in the other heads' scores; the values keep their size; norm
    weights far from one, negative too, different for every head."""
    cfg = config([(attn(heads=4, kv_heads=2, dim=6, rot=4, window=9), moe())])
    t = O.random_tensors(cfg, seed=21, dtype=torch.float32)
    t["l0.mix.k"][:6] *= 30.0
    t["l0.mix.q"][6:12] *= 20.0
    g = torch.Generator().manual_seed(5)
    t["l0.mix.k.norm"] = torch.randn(12, generator=g) * 2
    t["l0.mix.q.norm"] = torch.randn(24, generator=g) * 2
    toks = tokens_for(cfg, 25, 21)
    ref = O.forward(cfg, t, toks)
    model = make_worker(make, cfg, t)
    assert rel_err(run_portions(model, toks, 0, [11, 1, 1, 12]), ref) < TOL


def case_states_remember(make):
    """Decays so close to one that what the first tokens wrote is still in the state hundreds of tokens later, through portions and
    decoding, beside heads that forget within a token."""
    cfg = config([(mlstm(heads=3, dim=12, vdim=7, cap=20.0), None), (delta(heads=4, kv_heads=2, dim=16, vdim=5, conv=2), None)], width=32, streams=2)
    t = O.random_tensors(cfg, seed=14, dtype=torch.float32)
    t["l0.mix.f"] *= 0.1
    t["l0.mix.i"] *= 0.3
    t["l0.mix.f.b"] = torch.tensor([14.0, -12.0, 6.0])
    t["l0.mix.i.b"] = torch.tensor([0.0, 1.0, -3.0])
    t["l1.mix.a"] *= 0.1
    t["l1.mix.A_log"] = torch.tensor([-4.0, 4.0, -8.0, 0.0])
    t["l1.mix.dt_bias"] = torch.tensor([-6.0, 3.0, -3.0, -3.0])
    t["l1.mix.b"] *= 0.3
    toks = tokens_for(cfg, 300, 14)
    ref = O.forward(cfg, t, toks, dtype=torch.float64)
    other = list(toks); other[0] = (toks[0] + 1) % cfg["vocab"]; other[1] = (toks[1] + 3) % cfg["vocab"]
    assert rel_err(O.forward(cfg, t, other, dtype=torch.float64)[-1], ref[-1]) > 1e-4     # the start still matters at the end
    model = make_worker(make, cfg, t, block_size=16, num_blocks=20)
    got = run_portions(model, toks, 2, [130, 2, 100, 3, 1, 1] + [1] * 63)
    assert rel_err(got, ref) < TOL and rel_err(got[-1], ref[-1]) < TOL


def case_running_maximum(make):
    """Input gates that leap far up and down (the maximum follows at once and falls slowly), forget gates near zero and near one, and
    the floor of the denominator: a maximum that starts anywhere but at zero, or is not carried over a cut, shows."""
    cfg = config([(mlstm(heads=2, dim=6, vdim=5, cap=30.0), None)], width=24, streams=2, vocab=40, eps=1e-3)
    t = O.random_tensors(cfg, seed=15, dtype=torch.float32)
    t["l0.mix.i"] *= 8.0
    t["l0.mix.i.b"] = torch.tensor([-6.0, 3.0])
    t["l0.mix.f"] *= 3.0
    t["l0.mix.f.b"] = torch.tensor([1.0, -1.0])
    t["l0.mix.q"] *= 0.05                                             # |n . q| below the floor for many tokens
    toks = tokens_for(cfg, 60, 15)
    ref = O.forward(cfg, t, toks, dtype=torch.float64)
    for cuts in ([60], [1] * 60, [2, 9, 1, 1, 30, 17], [8, 8, 16, 28]):
        model = make_worker(make, cfg, t, block_size=8, num_blocks=10)
        assert rel_err(run_portions(model, toks, 0, cuts), ref) < TOL, cuts


def case_convolution_tails(make):
    """Taps whose far ends dominate, portions shorter than the taps, decoded tokens right behind them: a tail that is one input off
    shows."""
    cfg = config([(delta(heads=2, kv_heads=2, dim=6, vdim=5, conv=5), None)], width=24, streams=2)
    t = O.random_tensors(cfg, seed=16, dtype=torch.float32)
    for name in ("q", "k", "v"):
        c = torch.full_like(t[f"l0.mix.{name}.conv"], 0.1)
        c[:, 0], c[:, 1] = 1.5, -0.8                                  # the oldest inputs
        t[f"l0.mix.{name}.conv"] = c
    toks = tokens_for(cfg, 26, 16)
    ref = O.forward(cfg, t, toks)
    shifted = {k: (torch.roll(v, 1, dims=1) if k.endswith(".conv") else v) for k, v in t.items()}
    assert rel_err(O.forward(cfg, shifted, toks), ref) > 0.05
    for cuts in ([26], [1] * 26, [2, 2, 2, 2, 18], [3, 1, 2, 1, 1, 2, 16], [4, 4, 18]):
        model = make_worker(make, cfg, t, block_size=8, num_blocks=6)
        assert rel_err(run_portions(model, toks, 1, cuts), ref) < TOL, cuts


def case_pair_table(make):
    """The token pairs' table dominates: the first token's own row, pairs across portions, across decoded tokens and after a row was used
    by another sequence."""
    cfg = config([(attn(), None)], embed_scale=0.1, pair=(211, 31, 17))
    t = O.random_tensors(cfg, seed=18, dtype=torch.float32)
    t["bigram"] *= 3.0
    toks = tokens_for(cfg, 20, 18)
    ref = O.forward(cfg, t, toks)
    model = make_worker(make, cfg, t)
    for cuts in ([20], [1] * 20, [2, 1, 2, 15]):
        assert rel_err(run_portions(model, toks, 2, cuts), ref) < TOL, cuts
        model.free_seqs_resources([2])


def case_group_limited_choice(make):
    """Corrections that make every choice score negative (an expert outside the kept groups must count as minus infinity, not zero), a
    group that holds the best expert but loses by its second, and weights without the correction."""
    cfg = config([(attn(window=3), moe(experts=6, top=2, groups=3, keep=1, ff=8))], streams=2)
    t = O.random_tensors(cfg, seed=19, dtype=torch.float32)
    t["l0.mlp.correction"] = torch.tensor([-3.0, -5.0, -3.2, -3.2, -3.3, -4.0])      # group 0 has the best expert, group 1 the best pair
    t["l0.mlp.router"] *= 0.05
    toks = tokens_for(cfg, 20, 19)
    ref = O.forward(cfg, t, toks)
    w = O.routing_weights(0.05 * torch.randn(9, 6), t["l0.mlp.correction"], 2, {"count": 3, "keep": 1})
    assert bool((w[:, 2:4] > 0.4).all()) and float(w[:, [0, 1, 4, 5]].abs().max()) == 0.0
    model = make_worker(make, cfg, t)
    assert rel_err(run_portions(model, toks, 0, [9, 1, 10]), ref) < TOL


def case_streams_stay_apart(make):
    """Mixing matrices far from symmetric (a transposed one shows), shares of different sign, a stream that only one sublayer reads."""
    cfg = config([(mlstm(), moe()), (attn(), moe())], streams=4)
    t = O.random_tensors(cfg, seed=20, dtype=torch.float32)
    for i in (0, 1):
        for q in (1, 2):
            t[f"l{i}.hc{q}.mix"] = torch.tensor([[1.0, 0.9, 0.0, 0.0], [0.0, 1.0, -0.7, 0.0], [0.0, 0.0, 1.0, 0.5], [0.0, 0.0, 0.0, 1.0]])
            t[f"l{i}.hc{q}.out"] = torch.tensor([1.0, -0.5, 0.0, 2.0])
            t[f"l{i}.hc{q}.in"] = torch.tensor([0.0, 0.3, -1.0, 0.6])
    toks = tokens_for(cfg, 17, 20)
    ref = O.forward(cfg, t, toks)
    flipped = {k: (v.T.contiguous() if k.endswith(".mix") and ".hc" in k else v) for k, v in t.items()}
    assert rel_err(O.forward(cfg, flipped, toks), ref) > 0.05
    model = make_worker(make, cfg, t)
    assert rel_err(run_portions(model, toks, 0, [7, 1, 9]), ref) < TOL


def case_state_rows_used_again(make):
    """A row whose previous sequence left states of every recurrent layer: the next sequence in that row starts from nothing, also when
    its first portion is a single token."""
    cfg = config([(delta(), None), (mlstm(), moe()), (attn(), None), (delta(heads=2, kv_heads=1, dim=17, vdim=4, conv=4), moe())])
    t = O.random_tensors(cfg, seed=17, dtype=torch.float32)
    model = make_worker(make, cfg, t, block_size=4, num_blocks=24, rows=2)
    a, b, c = tokens_for(cfg, 30, 50), tokens_for(cfg, 9, 51), tokens_for(cfg, 12, 52)
    ra, rb, rc = (O.forward(cfg, t, s) for s in (a, b, c))
    assert rel_err(run_portions(model, a, 1, [30]), ra) < TOL
    model.free_seqs_resources([1])
    assert rel_err(run_portions(model, b, 1, [1, 1, 7]), rb) < TOL            # one-token first portion in the used row
    model.free_seqs_resources([1])
    assert rel_err(run_portions(model, c, 1, [5, 7]), rc) < TOL
    assert rel_err(run_portions(model, a[:10], 0, [10]), ra[:10]) < TOL       # the other row, never used before


PROBES = ["window_edges", "far_key", "sink", "first_tokens_and_block_borders", "rotation_far_out", "norms_over_the_whole_projection",
          "states_remember", "running_maximum", "convolution_tails", "pair_table", "group_limited_choice", "streams_stay_apart",
          "state_rows_used_again"]
