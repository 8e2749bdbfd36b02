"""Host-side logic of bench.py that needs no GPU: how a fixed job is spread over several GPUs."""
import dataclasses
import importlib
import os
import sys

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from conftest import cg

bench = importlib.import_module("bench")
synth = cg.synth


def test_parallelism_rule():
    small, big, moe = synth.LLAMA_32_1B, synth.LLAMA_3_8B, synth.QWEN3_30B_A3B
    # one GPU: nothing to choose
    assert bench.choose_parallelism("auto", small, 8, 1) == "tp"
    # a model whose decode step is bound by dependent latency keeps whole copies and splits the rows ...
    for world in (2, 4, 8):
        assert bench.choose_parallelism("auto", small, 8, world) == "dp"
    # ... unless the rows do not divide
    assert bench.choose_parallelism("auto", small, 8, 3) == "tp"
    # a model whose weight stream dominates is split
    for world in (2, 4, 8):
        assert bench.choose_parallelism("auto", big, 32, world) == "tp"
    # mixture-of-experts: experts and rows split when both divide
    assert bench.choose_parallelism("auto", moe, 8, 8) == "ep"
    assert bench.choose_parallelism("auto", moe, 8, 3) == "tp"
    # an explicit choice is kept
    for asked in ("tp", "dp", "ep"):
        assert bench.choose_parallelism(asked, small, 8, 2) == asked


def test_workloads_name_known_configurations():
    for name, (cfg_name, batch, prompt, decode) in bench.WORKLOADS.items():
        cfg = getattr(synth, cfg_name)
        assert batch >= 1 and prompt >= 1 and decode >= 1
        assert cfg.num_hidden_layers >= 1 and cfg.vocab_size > 0
        assert bench.dense_params_per_step(cfg) > 0


def test_layered_workloads_count_looped_layers():
    layered = importlib.import_module("catgrad-rs_b200.layered")
    for name, (cfg_name, batch, prompt, decode) in bench.LAYERED_WORKLOADS.items():
        cfg = getattr(layered, cfg_name)
        if not cfg.loop:
            # a layer with another one's weights counts them again
            own = dataclasses.replace(cfg, layers=[dataclasses.replace(L, weights_of=None) for L in cfg.layers])
            assert any(L.weights_of is not None for L in cfg.layers) == (cfg.design is layered.DESIGNS["Regupel"])
            assert bench.layered_step_bytes(own, batch, prompt) == bench.layered_step_bytes(cfg, batch, prompt)
            assert all(v > 0 for v in bench.layered_step_bytes(cfg, batch, prompt).values())
            continue
        once = bench.layered_step_bytes(dataclasses.replace(cfg, loop=None), batch, prompt)
        looped = bench.layered_step_bytes(cfg, batch, prompt)
        assert all(looped[k] > once[k] > 0 for k in once if k != "states" or cfg.recurrent)
    # experts without gates are two matrices each; block-diagonal gates count
    cfg = layered.KIVORAX_W1024
    plain = dataclasses.replace(cfg, layers=[dataclasses.replace(L, experts=None) if L.experts else L for L in cfg.layers])
    a, b = (bench.layered_step_bytes(c, 8, 512)["weights"] for c in (cfg, plain))
    more = sum(4 * 1024 * L.ffn * bench.experts_reached(32, 4, 8) + 2 * 32 * 1024 - 4 * 1024 * L.ffn for L in cfg.layers if L.experts)
    assert abs(a - b - more) < 1
    assert abs(bench.experts_reached(64, 64, 3) - 64) < 1e-9 and abs(bench.experts_reached(64, 1, 1) - 1) < 1e-9
