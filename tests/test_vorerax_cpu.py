"""CPU: the Vorerax worker's host path (registry, config, weight fusions, cache rows, state rows, batch metadata and segments, block / row /
state reuse, the scheduler loop) with the CUDA kernels replaced by the stand-ins of tests/cpu_shim.py, against oracle/vorerax.py."""
import json
import os

import pytest
import torch

import bupozen_cases as B
import vorerax_cases as C
from cpu_shim import product_on_cpu
from oracle import vorerax as O
from test_bupozen_cpu import _make


@pytest.fixture()
def cpu():
    with product_on_cpu():
        yield _make


def test_registry_picks_the_worker_from_the_config():
    import swiftllm_b200
    from swiftllm_b200 import registry
    mc = registry.model_config_from_dict(C.full_config())
    assert isinstance(mc, swiftllm_b200.VoreraxModelConfig) and registry.model_class_for(mc) is swiftllm_b200.VoreraxModel
    assert {"hyper_streams.cu", "delta_rule.cu", "matrix_memory.cu", "scan_ops.cu", "window_attn.cu", "stream_ops.cu"} <= \
        set(swiftllm_b200.VoreraxModel.NATIVE_SOURCES)
    assert "float32" in swiftllm_b200.VoreraxModel.DTYPES


def test_config_geometry_and_constants():
    import swiftllm_b200
    from swiftllm_b200.model_config import DeltaRuleSpec, MatrixMemorySpec, WAVE_BANDS, WindowAttentionSpec
    from swiftllm_b200.worker.kernels.window_attn import shared_row_width
    mc = swiftllm_b200.VoreraxModelConfig(C.full_config())
    # cache rows: [1 / rms (8 entries hold up to four key heads) | keys as projected with their turned entries, rounded up to 8]
    assert mc.cache_slots_per_width == {8 + 32: 1, 8 + 8: 1, 8 + 32: 1} or mc.cache_slots_per_width == {40: 2, 16: 1}
    assert [mc.cache_slot[i] for i in range(7)] == [None, (40, 0), None, (16, 0), None, None, (40, 1)]
    for i in (1, 3, 6):
        m = mc.mixers[i]
        assert m.cache_width == shared_row_width(m.kv_heads, m.dim, m.rot_dims)
    assert mc.get_kvslot_size(torch.bfloat16) == (40 + 16 + 40) * 2
    assert mc.get_state_size(torch.bfloat16) == 4 + 4 * 6 * 10 * 7 + 2 * (60 + 42) * 2 + 4 * 3 * (10 * 6 + 10 + 1) + \
        4 * 2 * (5 * 33 + 5 + 1) + 4 * 4 * 5 * 33 + 4 * (40 + 132) * 2
    a, d, s = mc.mixers[1], mc.mixers[0], mc.mixers[2]
    assert isinstance(a, WindowAttentionSpec) and a.window == 7 and a.shared_kv and a.whole_norm and a.learned_sink and a.gate_per_head
    assert a.rot_scaling == (WAVE_BANDS, 3.0, 40.0, 0.8, 2.5) and a.pair_halves and not a.sink
    assert mc.mixers[6].window == 0 and mc.mixers[6].rot_dims == 0 and mc.mixers[3].rot_scaling is None
    assert isinstance(d, DeltaRuleSpec) and (d.heads, d.kv_heads, d.dim, d.vdim, d.conv) == (6, 3, 10, 7, 3)
    assert isinstance(s, MatrixMemorySpec) and s.gate_cap == 9.0
    f = mc.ffs[0]
    assert (f.activation, f.routing, f.groups, f.keep, f.top) == ("silu_glu", "sigmoid_bias", 3, 2, 2) and mc.ffs[1] is None
    assert mc.ffs[2].groups == 1 and mc.num_streams == 3 and mc.residual_mult == 0.6 and mc.embedding_scale == 1.75
    assert (mc.pair_hash.buckets, mc.pair_hash.mul_prev, mc.pair_hash.mul_cur) == (53, 7, 11)
    plain = swiftllm_b200.VoreraxModelConfig(C.SINGLE["no_streams"])
    assert plain.num_streams == 1 and not plain.hyper
    bad = C.config([(C.attn(), None)])
    bad["layers"][0]["mixer"]["vdim"] = 11                    # the values are the keys
    with pytest.raises(AssertionError):
        swiftllm_b200.VoreraxModelConfig(bad)
    with pytest.raises(AssertionError):                        # three experts do not fit into one group of two
        swiftllm_b200.VoreraxModelConfig(C.config([(C.attn(), C.moe(top=3, keep=1))]))


def test_frequency_bands():
    from swiftllm_b200.model_config import WAVE_BANDS
    from swiftllm_b200.worker.token_model import rotary_frequencies
    for bands in (C.BANDS, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}, {"factor": 2.0, "low": 1.0, "high": 2.0, "original": 6}):
        rot = {"base": 500.0, "dims": 32, "scaling": bands}
        f, amp = rotary_frequencies(500.0, 32, (WAVE_BANDS, bands["factor"], bands["original"], bands["low"], bands["high"]))
        assert amp == 1.0 and f == pytest.approx(O.frequencies(rot), rel=1e-12)


def test_weight_fusions(cpu):
    cfg = C.full_config()
    t = O.random_tensors(cfg, seed=3, dtype=torch.float32)
    w = B.make_worker(cpu, cfg, t).weight.layers
    assert torch.equal(w[0].in_proj, torch.cat([t[f"l0.mix.{k}"] for k in "qkvg"])) and torch.equal(w[0].rate, torch.exp(t["l0.mix.A_log"]))
    assert torch.equal(w[0].gate_proj, torch.cat([t["l0.mix.b"], t["l0.mix.a"]])) and w[0].conv.shape == (30 + 30 + 42, 3)
    assert torch.equal(w[2].gate_proj, torch.cat([t["l2.mix.f"], t["l2.mix.i"]]))
    assert torch.equal(w[0].conn2.share, t["l0.hc2.out"] * 0.6) and torch.equal(w[0].conn1.mix, t["l0.hc1.mix"])


def test_checkpoint_folder_roundtrip(tmp_path, cpu):
    import swiftllm_b200
    from safetensors.torch import save_file
    cfg = C.config([(C.delta(), None), (C.attn(), C.moe()), (C.mlstm(), None)])
    t = O.random_tensors(cfg, seed=9)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in t.items()}, os.path.join(tmp_path, "model.safetensors"))
    ec = swiftllm_b200.EngineConfig(model_path=str(tmp_path), use_dummy=False, block_size=4, gpu_mem_utilization=0.9, num_cpu_blocks=0,
                                    max_seqs_in_block_table=2, max_blocks_per_seq=8, max_batch_size=2, max_tokens_in_batch=64,
                                    dtype="float32")
    m = swiftllm_b200.create_model(ec)
    m.load_weights()
    m.init_kvcache_and_swap(8)
    toks = B.tokens_for(cfg, 9, 9)
    assert B.rel_err(B.run_portions(m, toks, 1, [4, 5]), O.forward(cfg, t, toks)) < B.TOL


@pytest.mark.parametrize("name", sorted(C.SINGLE))
def test_single_mechanisms(cpu, name):
    B.case_whole_prompt(cpu, C.SINGLE[name], n=17)


def test_whole_prompt(cpu):
    B.case_whole_prompt(cpu, C.full_config())


def test_prefill_vs_decode(cpu):
    B.case_prefill_vs_decode(cpu, C.full_config())


def test_portions(cpu):
    B.case_portions(cpu, C.full_config())


def test_mixed_batch(cpu):
    B.case_mixed_batch(cpu, C.full_config())


def test_blocks_and_rows_reused(cpu):
    B.case_blocks_and_rows_reused(cpu, C.full_config())


def test_long_decode(cpu):
    B.case_long_decode(cpu, C.config([(C.attn(window=11), C.moe()), (C.delta(), None), (C.mlstm(), C.moe())]), n=45)


def test_greedy_generation(cpu):
    B.case_greedy_generation(cpu, C.config([(C.delta(), C.moe()), (C.attn(), C.moe()), (C.mlstm(), None)]))


@pytest.mark.parametrize("case", C.PROBES)
def test_probes(cpu, case):
    getattr(C, "case_" + case)(cpu)
