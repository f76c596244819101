"""Configurations and scenarios for the Zuzezen worker (swiftllm_b200.worker.zuzezen_model) against the plain restatement of the
design in oracle/zuzezen.py.  The schedule scenarios (whole prompts, decoding, portions, mixed batches, reused blocks and rows,
greedy generation) are the ones of tests/bupozen_cases.py; here are the design's own configurations and the scenarios whose weights
are made so that one particular fault would show.  They run on the CPU (kernels replaced by tests/cpu_shim.py) and on a GPU (the
CUDA kernels): tests/test_zuzezen_cpu.py and tests/test_zuzezen_gpu.py call them with the `make` factory of their world.

All configurations are small and deliberately irregular: head sizes that are not multiples of 16 or of each other, value sizes
unrelated to key sizes, several latent widths, one / several / as many key heads as query heads, windows of 1, 5, 7 and more
positions than the sequence has, none / one / more kept positions than the window, frequency ramps that cover all / some / none of
the pairs, decays near one and near zero, layers of every type with and without feed-forward."""
import math

import torch

from bupozen_cases import TOL, make_worker, rel_err, run_portions, tokens_for
from oracle import zuzezen as O


def latent(heads=3, dim=8, rot_dim=6, vdim=5, kv_rank=24, base=100.0, scaling=(3.0, 40, 4.0, 0.5), scale=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
                                "scale": scale if scale is not None else 1.3 / math.sqrt(dim + rot_dim)}


def attn(heads=6, kv_heads=2, dim=10, window=7, keep=2, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window, "keep_first": keep},
                         "scale": scale if scale is not None else 1.7 / math.sqrt(dim)}


def gla(heads=3, dim=10, vdim=6, tau=4.0):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def config(layers, width=48, vocab=97, eps=1e-5, embed_scale=1.75):
    return {"architecture": "Zuzezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "layers": [{"type": kind, "mixer": m, "mlp": f} for (kind, m), f in layers]}


def full_config():
    """Every branch at once."""
    return config([
        (gla(), dense()),
        (latent(), None),
        (attn(), dense(ff=17)),
        (latent(heads=11, dim=4, rot_dim=4, vdim=9, kv_rank=72, scaling=(2.0, 16, 2.0, 1.0)), dense()),
        (attn(heads=5, kv_heads=1, dim=6, window=5, keep=0), None),
        (gla(heads=2, dim=5, vdim=33, tau=1.0), None),
        (attn(heads=4, kv_heads=4, dim=7, window=64, keep=3), dense(ff=33)),
    ])


SINGLE = {
    "latent_dense": config([(latent(), dense())]),
    "latent_no_ff_one_head": config([(latent(heads=1, kv_rank=9, vdim=70), None)], embed_scale=1.0),
    "latent_many_heads_wide_latent": config([(latent(heads=17, dim=3, rot_dim=2, vdim=4, kv_rank=136), dense())]),
    "latent_all_pairs_slowed": config([(latent(rot_dim=8, scaling=(4.0, 8, 32.0, 8.0)), None)]),
    "latent_no_pair_slowed": config([(latent(rot_dim=8, scaling=(4.0, 100000, 1.0, 0.01)), None)]),
    "latent_factor_of_one": config([(latent(scaling=(1.0, 64, 8.0, 1.0)), None)]),
    "latent_plain_frequencies": config([(latent(scaling=None), None)]),
    "latent_16bit_shapes": config([(latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32), None)]),
    "attention_dense": config([(attn(), dense())]),
    "attention_mha_no_kept": config([(attn(heads=3, kv_heads=3, window=4, keep=0), None)]),
    "attention_mqa_wide": config([(attn(heads=5, kv_heads=1, dim=70, window=3, keep=1), dense())]),
    "attention_window_of_one": config([(attn(window=1, keep=1), None)]),
    "attention_more_kept_than_window": config([(attn(window=3, keep=9), None)]),
    "attention_window_longer_than_sequence": config([(attn(window=50, keep=4), None)]),
    "attention_16bit_shapes": config([(attn(heads=4, kv_heads=2, dim=16, window=6, keep=3), None)]),
    "gla_dense": config([(gla(), dense())]),
    "gla_no_ff_one_head": config([(gla(heads=1, dim=37, vdim=70, tau=16.0), None)]),
    "gla_tau_one_tiny_head": config([(gla(heads=7, dim=1, vdim=2, tau=1.0), None)]),
    "gla_values_narrower_than_keys": config([(gla(heads=2, dim=20, vdim=3, tau=0.5), dense())]),
}


# ---------------------------------------------------------------- scenarios made so that one fault shows
def _attention_probe(n, key_pos, window, keep, H=2, G=1, d=8, width=16, vocab=32, scale=3.0):
    """One windowed-attention layer in which every query points along one direction: the key of the marked token (token 1) points
    the same way, all other keys are orthogonal to it.  Queries and keys are RMS-normed, so `scale` alone sets how far the marked
    score (scale * d) stands above the others (0); the values are the un-normed keys, so the marked token also has its own value."""
    cfg = config([(attn(heads=H, kv_heads=G, dim=d, window=window, keep=keep, scale=scale), None)], width=width, vocab=vocab,
                 embed_scale=1.0)
    t = O.random_tensors(cfg, seed=11, dtype=torch.float32)
    t["embed"] = torch.randn(vocab, width, generator=torch.Generator().manual_seed(1)) * 0.1
    t["embed"][:, 0] = 1.0                       # every query reads this constant ...
    t["embed"][:, 1] = 0.0
    t["embed"][:, 2] = 1.0                       # ... every ordinary key this one ...
    t["embed"][1, 1] = 4.0                       # ... and only the marked token carries these
    t["embed"][1, 2] = 0.0
    q = torch.zeros(H, d, width); q[:, :, 0] = 2.0                     # all entries equal, direction (1, ..., 1)
    k = torch.zeros(G, d, width)
    k[:, :, 1] = 2.0                                                   # marked key: along the queries
    k[:, : d // 2, 2], k[:, d // 2:, 2] = 1.0, -1.0                    # ordinary keys: orthogonal to the queries
    t["l0.mix.q"], t["l0.mix.k"] = q.reshape(H * d, width), k.reshape(G * d, width)
    for name in ("q.b", "k.b"):
        t[f"l0.mix.{name}"] = torch.zeros_like(t[f"l0.mix.{name}"])
    t["l0.mix.q.norm"], t["l0.mix.k.norm"] = torch.ones(d), torch.ones(d)
    t["l0.ls1"] = torch.full((width,), 2.0)
    toks = [2 + (i % (vocab - 2)) for i in range(n)]
    toks[key_pos] = 1
    return cfg, t, toks


def case_window_edges(make):
    """The marked key just before, at and after the kept positions, and in the middle: queries up to the window's end see it, later
    ones only when it is kept - in a prompt, decoded, and with portions cut at, before and after every edge."""
    w, keep = 12, 3
    for key_pos in (0, keep - 1, keep, keep + 1, w - 1, 17):
        cfg, t, toks = _attention_probe(n=3 * w + 2, key_pos=key_pos, window=w, keep=keep)
        ref = O.forward(cfg, t, toks)
        kept = key_pos < keep
        for dw, dk in ((-1, 0), (1, 0), (0, -1 if kept else 1)):      # one position off in the window or in the kept positions shows
            if kept and dk == 0 or (dk and key_pos not in (keep - 1, keep)):
                continue
            m = {**cfg["layers"][0]["mixer"], "mask": {"size": w + dw, "keep_first": keep + dk}}
            other = {**cfg, "layers": [{**cfg["layers"][0], "mixer": m}]}
            assert rel_err(O.forward(other, t, toks), ref) > 0.02, (key_pos, dw, dk)
        edge = key_pos + w                                            # first position whose window no longer holds the marked key
        for cuts in ([3 * w + 2], [w, w, w + 2], [edge - 1, 2, 3 * w + 1 - edge], [edge, 1, 1, 3 * w - edge], [5] + [1] * (3 * w - 3),
                     [2] * (w + w // 2) + [2], [keep, 2, 3 * w - keep]):
            model = make_worker(make, cfg, t, block_size=8, num_blocks=8)
            got = run_portions(model, toks, 1, cuts)
            assert rel_err(got, ref) < TOL, (key_pos, cuts)
            for p in (key_pos, edge - 1, edge, edge + 1):             # just inside and just outside, one by one
                assert rel_err(got[p], ref[p]) < TOL, (key_pos, cuts, p)


def case_kept_keys_far_away(make):
    """A kept first position hundreds of positions back, with its true distance in the bias: across blocks, in prompt portions and
    when decoding; a capped distance or a forgotten kept key gives other logits."""
    cfg, t, toks = _attention_probe(n=390, key_pos=1, window=40, keep=2, H=4, G=2)
    ref = O.forward(cfg, t, toks)
    m = cfg["layers"][0]["mixer"]
    forgotten = {**cfg, "layers": [{**cfg["layers"][0], "mixer": {**m, "mask": {"size": 40, "keep_first": 1}}}]}
    assert rel_err(O.forward(forgotten, t, toks)[-1], ref[-1]) > 0.02
    assert rel_err(ref[60], ref[-1]) > 1e-3                           # the bias grows with the distance
    model = make_worker(make, cfg, t, block_size=8, num_blocks=50)
    got = run_portions(model, toks, 0, [200, 150, 38, 1, 1])
    assert rel_err(got[-8:], ref[-8:]) < TOL and rel_err(got, ref) < TOL


def case_values_are_unnormed_keys(make):
    """Key heads and channels of very different size: the scores see normed keys, the values keep their size; norm weights far from
    one on both sides."""
    cfg = config([(attn(heads=4, kv_heads=2, dim=6, window=9, keep=1), dense())])
    t = O.random_tensors(cfg, seed=21, dtype=torch.float32)
    t["l0.mix.k"][:6] *= 50.0
    t["l0.mix.k.b"][3] = 20.0
    t["l0.mix.k.norm"] = torch.tensor([0.1, 2.0, -1.0, 0.5, 3.0, 1.0])
    t["l0.mix.q.norm"] = torch.tensor([1.5, 0.3, 1.0, -2.0, 0.7, 1.0])
    toks = tokens_for(cfg, 25, 21)
    ref = O.forward(cfg, t, toks)
    model = make_worker(make, cfg, t)
    assert rel_err(run_portions(model, toks, 0, [11, 1, 1, 12]), ref) < TOL


def _latent_probe(n, key_pos, H=2, dn=8, dr=4, dv=6, r=8, width=16, vocab=32, scale=0.5, sink=0.0):
    """One latent-attention layer in which every query's unrotated part points along one direction of the latent, which only the
    marked token (token 1) has; the rotated parts are zero."""
    cfg = config([(latent(heads=H, dim=dn, rot_dim=dr, vdim=dv, kv_rank=r, scale=scale), None)], width=width, vocab=vocab, embed_scale=1.0)
    t = O.random_tensors(cfg, seed=12, dtype=torch.float32)
    t["embed"] = torch.randn(vocab, width, generator=torch.Generator().manual_seed(2)) * 0.1
    t["embed"][:, 0] = 1.0
    t["embed"][:, 1] = 0.0
    t["embed"][:, 2] = 1.0
    t["embed"][1, 1], t["embed"][1, 2] = 4.0, 0.0
    q = torch.zeros(H, dn + dr, width); q[:, 0, 0] = 4.0
    dkv = torch.zeros(r + dr, width); dkv[0, 1] = 2.0; dkv[1, 2] = 2.0
    uk = torch.zeros(H, dn, r); uk[:, 0, 0] = 2.0                       # the key's first entry: the marked direction of the latent
    t["l0.mix.q"], t["l0.mix.dkv"], t["l0.mix.uk"] = q.reshape(-1, width), dkv, uk.reshape(-1, r)
    t["l0.mix.dkv.norm"] = torch.ones(r)
    t["l0.mix.sink"] = torch.full((H,), sink)
    t["l0.ls1"] = torch.full((width,), 2.0)
    toks = [2 + (i % (vocab - 2)) for i in range(n)]
    toks[key_pos] = 1
    return cfg, t, toks


def case_far_latent(make):
    """A marked latent hundreds of positions back among rows that all score the same: every later position must still see it."""
    cfg, t, toks = _latent_probe(n=390, key_pos=3)
    ref = O.forward(cfg, t, toks)
    plain = list(toks); plain[3] = 5
    assert rel_err(O.forward(cfg, t, plain)[-1], ref[-1]) > 0.05
    model = make_worker(make, cfg, t, block_size=8, num_blocks=50)
    got = run_portions(model, toks, 0, [200, 150, 38, 1, 1])
    assert rel_err(got[-8:], ref[-8:]) < TOL and rel_err(got, ref) < TOL


def case_sink(make):
    """Sinks from far below to far above the scores, different per head: with a large sink a head's output nearly vanishes, which the
    gate and the output norm then show; the first token (alone with the sink) shows it most."""
    for sinks in ([-20.0, 3.0], [9.0, 2.0], [0.0, 30.0]):
        cfg, t, toks = _latent_probe(n=21, key_pos=4)
        t["l0.mix.sink"] = torch.tensor(sinks)
        ref = O.forward(cfg, t, toks)
        none = dict(t); none["l0.mix.sink"] = torch.full((2,), -1e4)
        assert rel_err(O.forward(cfg, none, toks), ref) > 0.02
        for cuts in ([21], [1] * 21, [2, 3, 1, 15]):
            model = make_worker(make, cfg, t, block_size=8, num_blocks=6)
            assert rel_err(run_portions(model, toks, 1, cuts), ref) < TOL, (sinks, cuts)


def case_first_tokens_and_block_borders(make):
    """The marked row at the first position, at the last slot of a block and at the first slot of the next one; queries right behind
    it, in a prompt and decoded - in both kinds of attention."""
    for key_pos in (0, 7, 8):
        for cfg, t, toks in (_attention_probe(n=20, key_pos=key_pos, window=32, keep=1), _latent_probe(n=20, key_pos=key_pos)):
            ref = O.forward(cfg, t, toks)
            for cuts in ([20], [key_pos + 1, 1, 1, 17 - key_pos], [2] + [1] * 18, [8, 8, 4]):
                model = make_worker(make, cfg, t, block_size=8, num_blocks=6)
                assert rel_err(run_portions(model, toks, 1, cuts), ref) < TOL, (key_pos, cuts)


def case_rotation_far_out(make):
    """Positions far beyond the original context of the ramped frequencies; the rotated parts dominate the scores."""
    cfg = config([(latent(heads=2, dim=2, rot_dim=8, vdim=6, kv_rank=12, base=50.0, scaling=(5.0, 24, 3.0, 0.4), scale=0.6), None)])
    t = O.random_tensors(cfg, seed=13, dtype=torch.float32)
    t["l0.mix.uk"] *= 0.05
    toks = tokens_for(cfg, 150, 13)
    ref = O.forward(cfg, t, toks, dtype=torch.float64)
    for change in ({"factor": 4.0}, {"original": 30}, {"fast": 6.0}, {"slow": 0.2}):
        rot = cfg["layers"][0]["mixer"]["rot"]
        other = {**cfg["layers"][0]["mixer"], "rot": {**rot, "scaling": {**rot["scaling"], **change}}}
        if O.ramped_frequencies(other["rot"]) != O.ramped_frequencies(rot):
            assert rel_err(O.forward({**cfg, "layers": [{**cfg["layers"][0], "mixer": other}]}, t, toks, dtype=torch.float64), ref) > 0.01
    model = make_worker(make, cfg, t, block_size=8, num_blocks=20)
    assert rel_err(run_portions(model, toks, 0, [70, 2, 60, 1, 1, 1, 15]), ref) < TOL


def case_slow_channels_remember(make):
    """Decays so close to one that what the first tokens wrote is still in the state hundreds of tokens later, through portions and
    decoding, beside channels that forget within a token or two (and batches whose decays cannot be folded into the staged vectors)."""
    for tau, slow, fast in ((16.0, 6.0, -90.0), (1.0, 9.0, -12.0)):
        cfg = config([(gla(heads=2, dim=12, vdim=7, tau=tau), None), (gla(heads=3, dim=4, vdim=5, tau=tau), dense())], width=32)
        t = O.random_tensors(cfg, seed=14, dtype=torch.float32)
        for layer, nk in (("l0", 24), ("l1", 12)):
            b = torch.full((nk,), slow)
            b[::3] = fast
            t[f"{layer}.mix.a2.b"] = b
            t[f"{layer}.mix.a2"] *= 0.1
        toks = tokens_for(cfg, 300, 14)
        ref = O.forward(cfg, t, toks, dtype=torch.float64)
        other = list(toks); other[0] = (toks[0] + 1) % cfg["vocab"]; other[1] = (toks[1] + 3) % cfg["vocab"]
        assert rel_err(O.forward(cfg, t, other, dtype=torch.float64)[-1], ref[-1]) > 1e-3     # the start still matters at the end
        model = make_worker(make, cfg, t, block_size=16, num_blocks=20)
        got = run_portions(model, toks, 2, [130, 2, 100, 3, 1, 1] + [1] * 63)
        assert rel_err(got, ref) < TOL and rel_err(got[-1], ref[-1]) < TOL


def case_state_rows_used_again(make):
    """A row whose previous sequence left states of every linear-attention layer: the next sequence in that row starts from nothing,
    also when its first portion is a single token."""
    cfg = config([(gla(), None), (latent(), dense()), (gla(heads=2, dim=17, vdim=4, tau=30.0), dense())])
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
