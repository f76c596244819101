"""CPU: the Zuzezen worker's host path (registry, config, weight fusions, cache rows of several widths, state rows, batch metadata and
segments, block / row / state reuse, the scheduler loop) with the CUDA kernels replaced by the stand-ins of tests/cpu_shim.py,
against oracle/zuzezen.py."""
import json
import os

import pytest
import torch

import bupozen_cases as B
import zuzezen_cases as C
from cpu_shim import product_on_cpu
from oracle import zuzezen as O
from test_bupozen_cpu import _make


@pytest.fixture()
def cpu():
    with product_on_cpu():
        yield _make


def test_registry_picks_the_worker_from_the_config():
    import swiftllm_b200
    from swiftllm_b200 import registry
    mc = registry.model_config_from_dict(C.full_config())
    assert isinstance(mc, swiftllm_b200.ZuzezenModelConfig) and registry.model_class_for(mc) is swiftllm_b200.ZuzezenModel
    assert {"gla.cu", "latent_attn.cu", "window_attn.cu", "stream_ops.cu"} <= set(swiftllm_b200.ZuzezenModel.NATIVE_SOURCES)
    assert "float32" in swiftllm_b200.ZuzezenModel.DTYPES


def test_config_geometry_and_constants():
    import swiftllm_b200
    from swiftllm_b200.model_config import GatedLinearAttentionSpec, LatentAttentionSpec, WindowAttentionSpec
    from swiftllm_b200.worker.kernels.window_attn import shared_row_width
    mc = swiftllm_b200.ZuzezenModelConfig(C.full_config())
    # cache rows: [latent | rotated part], [1 / rms (8 entries hold up to four key heads) | keys as projected, rounded up to 8]
    assert mc.cache_slots_per_width == {24 + 6: 1, 8 + 24: 1, 72 + 4: 1, 8 + 8: 1, 8 + 32: 1}
    assert [mc.cache_slot[i] for i in range(7)] == [None, (30, 0), (32, 0), (76, 0), (16, 0), None, (40, 0)]
    for i in (2, 4, 6):
        assert mc.mixers[i].cache_width == shared_row_width(mc.mixers[i].kv_heads, mc.mixers[i].dim)
    assert mc.get_kvslot_size(torch.bfloat16) == (30 + 32 + 76 + 16 + 40) * 2
    assert mc.get_state_size() == 4 * (3 * 10 * 6 + 2 * 5 * 33)
    a, l, g = mc.mixers[2], mc.mixers[1], mc.mixers[5]
    assert isinstance(a, WindowAttentionSpec) and a.window == 7 and a.keep_first == 2 and a.shared_kv and a.distance_bias and a.gate_per_head
    assert a.qk_weight_norm and a.rot_dims == 0 and not a.sink
    assert isinstance(l, LatentAttentionSpec) and l.q_rank == 0 and l.rot_scaling == (3.0, 40.0, 4.0, 0.5) and l.sink and l.gate == "element"
    assert l.window == 0 and l.rot_key == (100.0, 6, (3.0, 40.0, 4.0, 0.5))
    assert isinstance(g, GatedLinearAttentionSpec) and (g.heads, g.dim, g.vdim, g.tau) == (2, 5, 33, 1.0)
    assert mc.ffs[0].activation == "silu_glu" and mc.ffs[0].bias and mc.ffs[1] is None and mc.ffs[2].ff == 17
    assert mc.embedding_scale == 1.75
    plain = swiftllm_b200.ZuzezenModelConfig(C.SINGLE["gla_dense"])
    assert plain.cache_slots_per_width == {}
    bad = C.config([(C.attn(), None)])
    bad["layers"][0]["mixer"]["vdim"] = 11                    # the values are the keys
    with pytest.raises(AssertionError):
        swiftllm_b200.ZuzezenModelConfig(bad)


def test_gains_and_inner_decay_size_come_from_the_checkpoint(cpu):
    """The output norm's 1 + w and the layer scale are one gain; both q / k norm weights are one; the decay projection's inner size
    is whatever the tensors have."""
    for rank in (1, 5, 24):
        cfg = C.config([(C.gla(), C.dense()), (C.attn(), None)])
        t = O.random_tensors(cfg, seed=3, dtype=torch.float32, rank=rank)
        m = B.make_worker(cpu, cfg, t)
        w = m.weight.layers
        assert w[0].a2.shape[1] == rank and w[0].in_proj.shape[0] == 2 * 30 + 2 * 18 + rank
        assert torch.equal(w[0].norm2, (1 + t["l0.norm2"]) * t["l0.ls2"])
        assert torch.equal(w[1].qk_norm, t["l1.mix.q.norm"] * t["l1.mix.k.norm"])
        toks = B.tokens_for(cfg, 12, rank)
        assert B.rel_err(B.run_portions(m, toks, 0, [5, 1, 6]), O.forward(cfg, t, toks)) < B.TOL


def test_checkpoint_folder_roundtrip(tmp_path, cpu):
    import swiftllm_b200
    from safetensors.torch import save_file
    cfg = C.config([(C.gla(), None), (C.latent(), C.dense()), (C.attn(), None)])
    t = O.random_tensors(cfg, seed=9, rank=3)
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
    B.case_long_decode(cpu, C.config([(C.attn(window=11), C.dense()), (C.gla(), None), (C.latent(), C.dense())]), n=45)


def test_greedy_generation(cpu):
    B.case_greedy_generation(cpu, C.config([(C.gla(), C.dense()), (C.attn(), C.dense()), (C.latent(), None)]))


@pytest.mark.parametrize("case", ["window_edges", "kept_keys_far_away", "values_are_unnormed_keys", "far_latent", "sink",
                                  "first_tokens_and_block_borders", "rotation_far_out", "slow_channels_remember", "state_rows_used_again"])
def test_probes(cpu, case):
    getattr(C, "case_" + case)(cpu)
