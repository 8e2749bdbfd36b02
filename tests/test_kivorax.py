"""Decoders of the Kivorax design (sublayers side by side on one norm, a per-layer input for the token,
averages over depth; attention with distance biases, warmed queries and gated values beside Griffin's
recurrent block; the delta rule and gated linear attention with a decay per key channel; dense gelu
feed-forwards with biases and ungated experts) against the plain restatement of its equations in
kivorax_oracle.py: each mechanism alone, whole prompts, portions, decoding through the cache and state,
unequal batches, reused slots, far keys, far memories and extreme decays, and greedy generation through
the decoder's entry points.

Errors are measured as in test_hybrid.py.  In a bf16 context a token whose choice of experts is a close
call may choose otherwise, so such tokens are left out there.
"""
import functools
import importlib
import json
import os
import subprocess

import numpy as np
import pytest

import kivorax_oracle as oracle
from test_hybrid import ROOT, TOL, backends, close, decoder, err, everything, same_up_to_ties, toks  # noqa: F401

cg = importlib.import_module("catgrad-rs_b200")
gpu = pytest.mark.gpu


def par(heads=4, kv_heads=2, dim=24, vdim=20, scale=0.4, temp=(0.4, 10), width=48, blocks=3, conv=4):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        left["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "parallel", "mixer": {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv}}, "mlp": None}


def cdelta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": None}


def gla(heads=3, dim=16, vdim=24, tau=4.0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": None}


def dense(layer, ff=88):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def moe(layer, experts=7, top=3, ff=28):
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}})


def model(layers, width=72, vocab=104, eps=1e-4, scale=2.5, side=12):
    return {"architecture": "Kivorax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "embedding": {"scale": scale},
            "token_side": {"dim": side} if side else None}


def weights(cfg, seed=0, ranks=(10, 14)):
    """Random weights under which every mechanism carries weight: attention scores of a few units, decays
    from one token to hundreds, biases and gains that differ, averages that mix all depths.  The routers
    read mostly the first components of the stream, where a token's embedding holds well separated
    levels that the layers hardly move: few choices are close calls."""
    rng = np.random.default_rng(seed)
    out = {}
    E = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if L["mlp"] and L["mlp"]["kind"] == "moe"] or [0])
    levels = np.array([rng.permutation(np.linspace(-2.5, 2.5, E)) for _ in range(cfg["vocab"])]).reshape(cfg["vocab"], E) / cfg["embedding"]["scale"]
    c = cg.registry.config_from_json(cfg)
    c.ranks = ranks
    for name, shape in c.param_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "A_log":
            w = rng.uniform(-3.0, 1.5, shape)
        elif leaf == "dt_bias":
            w = rng.uniform(-4.0, 0.0, shape)
        elif name.endswith("a2.b"):
            w = rng.uniform(-1.0, 5.0, shape)
        elif leaf == "lam":
            w = rng.uniform(-5.0, -0.5, shape)
        elif name.endswith("ra.b"):
            w = rng.uniform(-4.0, 2.0, shape)
        elif leaf in ("r1", "r2"):
            w = rng.uniform(0.05, 2.0 if leaf == "r1" else 0.5, shape)
        elif leaf == "dwa":
            w = rng.normal(0, 0.25, shape)
            w[-1] += 1.0 - w.sum()
        elif leaf == "b" and not name.endswith(".mix.b"):
            w = rng.normal(0, 0.4, shape)
        elif len(shape) == 1:
            w = 1.0 + rng.normal(0, 0.3, shape)
        elif leaf == "embed" and name == "embed":
            w = rng.normal(0, 0.5, shape)
            w[:, :E] = levels
        elif name == "side.embed":
            w = rng.normal(0, 1.0, shape)
        elif leaf == "router":
            w = rng.normal(0, 0.15 * shape[1] ** -0.5, shape) + np.eye(*shape)
        elif leaf == "conv":
            w = rng.normal(0, shape[1] ** -0.5, shape)
        else:
            w = rng.normal(0, (1.5 if leaf in ("g", "g2", "ra", "ri") else 1.0) * shape[-1] ** -0.5, shape)
            if name.endswith(("left.q", "left.k")):
                w *= np.geomspace(0.3, 2.0, shape[0])[:, None]     # heads differ in size
        if leaf in ("o", "down", "out") or name.endswith(("down.b", "side.norm")):
            w[:E] *= 0.05
        if leaf == "norm1":
            w[:E] = 1.0
        out[name] = cg.synth.bf16_round(np.asarray(w, np.float32))
    return out


def sure(gaps, n):
    """Tokens none of whose expert choices is a close call."""
    return np.min(gaps, axis=0) > 0.05 if gaps else np.ones(n, bool)


def expected(cfg, W, seq, **kw):
    """The oracle's logits and which positions to compare in bf16."""
    gaps = []
    want = oracle.forward(cfg, W, seq, gaps=gaps, **kw)
    return want, sure(gaps, len(seq))


def agrees(got, want, ok, prec):
    ok = np.asarray(ok) if prec == "bf16" else np.ones(len(want), bool)
    assert ok.mean() > 0.25 or len(ok) < 20
    return not ok.any() or close(np.asarray(got)[ok], np.asarray(want)[ok], prec)


MIXED = model([dense(cdelta()), moe(gla()), moe(par()), cdelta(heads=2, kv_heads=2, dim=24, vdim=16, conv=2),
               moe(gla(heads=2, dim=40, vdim=8, tau=16.0), 4, 1, 20), dense(par(heads=6, kv_heads=3, dim=8, vdim=16, width=32, blocks=2, temp=None), 40)])


# ---------------------------------------------------------------------------- configuration (CPU)

def test_config_reader_and_shapes():
    cfg = cg.registry.config_from_json(MIXED)
    assert cfg.rms_norm_eps == 1e-4 and cfg.embed_scale == 2.5 and cfg.token_side == 12 and cfg.recurrent
    assert cfg.design.switches()["parallel_sublayers"] == cfg.design.switches()["depth_average"] == 1
    st = cfg.layers[2].struct(cfg.design)
    right = type(st).from_address(st.beside)
    assert (st.mixer, st.gate, st.dist_bias, st.out_norm, st.q_temp_coef, st.q_temp_every, st.act, st.experts) == (4, 2, 1, 1, 0.4, 10.0, 3, 7)
    assert (right.mixer, right.heads, right.vdim, right.conv) == (8, 3, 16, 4)
    assert cfg.layers[5].struct(cfg.design).q_temp_every == 0
    st = cfg.layers[0].struct(cfg.design)
    assert (st.mixer, st.heads, st.kv_heads, st.dim, st.vdim, st.conv, st.act, st.ffn) == (6, 4, 2, 16, 24, 4, 4, 88)
    st = cfg.layers[4].struct(cfg.design)
    assert (st.mixer, st.tau, st.top_k) == (7, 16.0, 1)
    s = cfg.param_shapes()
    assert s["l0.mix.a2"] == (64, 16) and s["l0.mlp.up.b"] == (88,) and s["l1.mix.a2.b"] == (48,) and s["l2.mix.left.g"] == (80, 72)
    assert s["l2.mix.right.ra"] == (3, 16, 16) and s["l3.dwa"] == (5,) and s["side.embed"] == (104, 72) and s["l5.side.proj"] == (72, 12)
    assert not {"l0.norm2", "l0.mlp.gate", "l1.mlp.e0.gate", "l0.mix.a", "l0.mix.g", "l1.mix.q.conv", "final.norm.b"} & set(s)
    plain = cg.registry.config_from_json(model([gla()], side=0))
    assert plain.token_side == 0 and "side.embed" not in plain.param_shapes()
    with pytest.raises(ValueError):
        cg.registry.config_from_json(model([dict(gla(), type="delta")]))
    with pytest.raises(ValueError):
        L = cg.registry.config_from_json(model([par(width=50, blocks=3)]))
        L.layers[0].struct(L.design)


FAULTS = [(f, par()) for f in ("no_temperature", "late_temperature", "no_distance", "far_by_one", "no_gate", "interleaved_heads", "whole_sum",
                               "taps_reversed", "lost_tail", "lost_state", "gates_transposed", "first_token_special", "no_conv_bias")]
FAULTS += [(f, cdelta()) for f in ("taps_reversed", "lost_tail", "no_silu", "no_unit", "mean_decay", "undecayed_read", "early_read", "lost_state")]
FAULTS += [(f, gla()) for f in ("no_tau", "decays_first", "sigmoid_gate", "lost_state", "no_side", "first_part", "side_of_input", "no_average",
                                "averages_averages")]
FAULTS += [("no_up_bias", dense(gla())), ("no_down_bias", dense(gla())), ("sequential", dense(gla())), ("renormalised", moe(gla()))]


@pytest.mark.parametrize("fault,layer", FAULTS)
def test_planted_mistakes_would_show(fault, layer):
    """The inputs of these tests tell the equations from near misses: with the mistake planted in the
    oracle the logits move by hundreds of times the f32 tolerance."""
    cfg = model([gla(), layer, cdelta()])
    W, seq = weights(cfg), toks(60, 1)
    moved = err(oracle.forward(cfg, W, seq, faults=(fault,)), oracle.forward(cfg, W, seq))
    assert moved > 300 * TOL["f32"], moved


def test_oracle_recurrences_are_decaying_sums():
    """What gated linear attention reads at a token is the decayed sum over all tokens before it, and the
    recurrent block's state is the decayed sum of its gated inputs."""
    rng = np.random.default_rng(0)
    T, W, m = 12, 8, {"heads": 2, "dim": 3, "vdim": 4, "tau": 2.0}
    P = {n: rng.normal(size=(r, W)) for n, r in (("q", 6), ("k", 6), ("v", 8), ("g", 8), ("a1", 5))}
    P |= {"a2": rng.normal(size=(6, 5)), "a2.b": rng.normal(size=6), "norm": np.ones(4), "o": np.eye(8)}
    h = rng.normal(size=(T, W))
    q, k, v = ((h @ P[n].T).reshape(T, 2, -1) for n in "qkv")
    la = np.log(oracle.sigmoid(h @ P["a1"].T @ P["a2"].T + P["a2.b"])).reshape(T, 2, 3) / 2.0
    o = np.array([[sum((q[t, n] * k[s, n] * np.exp(la[s + 1:t + 1, n].sum(0))).sum() * v[s, n] for s in range(t + 1)) for n in range(2)]
                  for t in range(T)]) * 3 ** -0.5
    assert np.allclose(oracle.gla(h, P.__getitem__, m, 1e-6), oracle.rms(o, 1e-6).reshape(T, 8) * oracle.silu(h @ P["g"].T))
    assert [oracle.temperature(p, 1.0, 4) for p in (0, 2, 3, 6, 7)] == [1.0, 1.0, 1 + np.log(2), 1 + np.log(2), 1 + np.log(3)]


# --------------------------------------------------------------------- each mechanism alone (GPU)

ALONE = {
    "parallel": [par()],
    "parallel_no_temperature": [par(temp=None)],
    "parallel_temperature_every_token": [par(temp=(1.5, 1))],
    "parallel_temperature_after_the_end": [par(temp=(2.0, 1000))],
    "parallel_one_head": [par(heads=1, kv_heads=1, dim=8, vdim=8, width=8, blocks=1, conv=1)],
    "parallel_values_wider": [par(dim=32, vdim=64)],
    "parallel_keys_wider": [par(dim=64, vdim=24)],
    "parallel_head_64": [par(dim=64, vdim=64, heads=2, kv_heads=1)],
    "parallel_head_128": [par(heads=4, kv_heads=1, dim=72, vdim=128, width=128, blocks=2)],
    "parallel_head_256": [par(heads=2, kv_heads=1, dim=160, vdim=256, scale=0.1)],
    "parallel_head_300": [par(heads=2, kv_heads=1, dim=300, vdim=12, scale=0.1)],
    "parallel_many_queries_per_key": [par(heads=12, kv_heads=1, dim=16, vdim=16)],
    "parallel_eight_queries_per_key": [par(heads=16, kv_heads=2, dim=16, vdim=24)],
    "parallel_one_block": [par(width=96, blocks=1, conv=2)],
    "parallel_channel_blocks": [par(width=40, blocks=40, conv=3)],
    "parallel_uneven_blocks": [par(width=66, blocks=6, conv=5)],
    "parallel_blocks_of_48": [par(width=144, blocks=3)],
    "parallel_wide_blocks": [par(width=320, blocks=2, conv=6)],
    "delta": [cdelta()],
    "delta_equal_heads": [cdelta(heads=2, kv_heads=2, dim=32, vdim=32, conv=3)],
    "delta_one_head": [cdelta(heads=1, kv_heads=1, dim=8, vdim=40, conv=1)],
    "delta_uneven": [cdelta(heads=6, kv_heads=2, dim=20, vdim=36, conv=5)],
    "delta_odd": [cdelta(heads=3, kv_heads=1, dim=5, vdim=7, conv=2)],
    "delta_48": [cdelta(heads=2, kv_heads=1, dim=48, vdim=80)],
    "delta_64": [cdelta(heads=2, kv_heads=1, dim=64, vdim=96, conv=2)],
    "delta_100": [cdelta(heads=2, kv_heads=2, dim=100, vdim=72)],
    "delta_128": [cdelta(heads=4, kv_heads=2, dim=128, vdim=128)],
    "delta_wide": [cdelta(heads=2, kv_heads=1, dim=136, vdim=144, conv=3)],
    "delta_wide_values": [cdelta(heads=2, kv_heads=1, dim=48, vdim=200)],
    "gla": [gla()],
    "gla_one_head": [gla(heads=1, dim=8, vdim=40, tau=1.0)],
    "gla_odd": [gla(heads=3, dim=5, vdim=7, tau=16.0)],
    "gla_64": [gla(heads=2, dim=64, vdim=64, tau=16.0)],
    "gla_72": [gla(heads=2, dim=72, vdim=136, tau=2.0)],
    "gla_128": [gla(heads=2, dim=128, vdim=128, tau=0.5)],
    "gla_wide": [gla(heads=2, dim=144, vdim=20)],
    "dense": [dense(gla(), 100)],
    "dense_beside_two_mixers": [dense(par(), 44)],
    "experts": [moe(gla())],
    "one_of_many": [moe(cdelta(), 16, 1)],
    "all_experts": [moe(gla(), 5, 5)],
    "single_expert": [moe(par(), 1, 1, 44)],
    "many_experts": [moe(gla(), 40, 4, 12)],
    "seven_layers": [gla(), cdelta(), gla(), par(), gla(), cdelta(), gla()],
    "narrow": [moe(par(heads=1, kv_heads=1, dim=6, vdim=5, width=6, blocks=2), 3, 2, 11), dense(cdelta(heads=3, kv_heads=1, dim=10, vdim=7), 13)],
}


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(backends, name, prec):
    """Residual stream behind every layer and logits at every position, in one portion and cut in ways
    that take the prompt kernels, those of short portions and the decode kernels."""
    cfg = model(ALONE[name], width=44 if name == "narrow" else 72, vocab=101 if name == "narrow" else 104, side=5 if name == "narrow" else 12)
    W, seq = weights(cfg, 3), toks(150, 2, 101)
    layers = []
    want, ok = expected(cfg, W, seq, hooks=lambda i, x: layers.append(x))
    dec = decoder(backends[prec], cfg, W)
    dec.keep_residuals()
    got = everything(dec, seq)
    got_layers = dec.residuals()
    for i, x in enumerate(layers):
        assert agrees(got_layers[i], x, ok, prec), i
    assert agrees(got, want, ok, prec)
    dec.keep_residuals(False)
    for cut in ([129, 10] + [1] * 11, [70, 80], [40, 30, 5, 2, 73]):
        assert agrees(everything(dec, seq, cut), want, ok, prec), cut
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("scale,eps,side,ranks", [(1.0, 1e-6, 0, (1, 1)), (12.0, 1e-2, 8, (24, 16)), (0.25, 0.5, 70, (7, 40)), (3.0, 1e-2, 1, (16, 3))])
def test_constants_and_ranks(backends, scale, eps, side, ranks, prec):
    """The ranks of the low-rank projections follow from the tensors alone."""
    cfg = model([par(), cdelta(), dense(gla())], scale=scale, eps=eps, side=side)
    W, seq = weights(cfg, 4, ranks), toks(70, 3)
    want, ok = expected(cfg, W, seq)
    dec = decoder(backends[prec], cfg, W)
    assert agrees(everything(dec, seq), want, ok, prec)
    assert agrees(everything(dec, seq, [40] + [1] * 30), want, ok, prec)
    dec.close()


@gpu
def test_wide_rows_take_the_persistent_kernels(backends):
    """Sizes at which the projections (gelu among them) and the experts run on the persistent GEMMs."""
    for seed, n, ff in ((6, 600, 256), (7, 1100, 512)):
        cfg = model([moe(par(heads=4, kv_heads=2, dim=64, vdim=128, width=512, blocks=4), 4, 2, ff), dense(gla(heads=8, dim=64, vdim=128), 4096),
                     moe(cdelta(heads=4, kv_heads=2, dim=128, vdim=128), 4, 2, ff)], width=1024, side=128)
        W, seq = weights(cfg, seed, (128, 128)), toks(n, seed)
        want, ok = expected(cfg, W, seq)
        dec = decoder(backends["bf16"], cfg, W, max_seq=1104, max_batch=1)
        assert agrees(everything(dec, seq), want, ok, "bf16")
        dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("layer", [cdelta(dim=64, vdim=32), gla(dim=64, vdim=32, tau=1.0), cdelta(dim=128, vdim=64), gla(heads=2, dim=100, vdim=64, tau=0.25)])
def test_extreme_decays(backends, layer, prec):
    """Channels that forget everything at some tokens and hardly anything at others, beside channels that
    never forget and channels that always do: factors relative to a chunk's start or end alone would
    overflow, or lose what was written behind a strong decay."""
    cfg = model([layer])
    W, seq = weights(cfg, 5), toks(200, 6)
    rng = np.random.default_rng(1)
    b = "l0.mix." + ("dt_bias" if layer["type"] == "channel_delta" else "a2.b")
    sign = 1.0 if layer["type"] == "channel_delta" else -1.0      # large z: strong decay / hardly any
    W[b] = cg.synth.bf16_round((sign * rng.choice([-12.0, -6.0, 0.0, 5.0, 60.0], W[b].shape)).astype(np.float32))
    W["l0.mix.a2"] = cg.synth.bf16_round(W["l0.mix.a2"] * 6.0)
    if "l0.mix.A_log" in W:
        W["l0.mix.A_log"] = np.asarray(rng.choice([-1.0, 1.0, 2.75], W["l0.mix.A_log"].shape), np.float32)
    want = oracle.forward(cfg, W, seq)
    dec = decoder(backends[prec], cfg, W)
    for cut in (None, [64, 64, 72], [100, 3, 60] + [1] * 37):
        got = everything(dec, seq, cut)
        assert np.isfinite(got).all() and close(got, want, prec), cut
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_extreme_gates_of_the_recurrent_block(backends, prec):
    """Decays from exactly 1 (to f32) to exactly 0: sqrt(1 - a^2) from a alone would lose its small values."""
    cfg = model([par(width=64, blocks=4)])
    W, seq = weights(cfg, 6), toks(160, 7)
    rng = np.random.default_rng(2)
    W["l0.mix.right.lam"] = np.asarray(rng.choice([-12.0, -6.0, 0.0, 20.0], 64), np.float32)
    W["l0.mix.right.ra.b"] = np.asarray(rng.choice([-9.0, 0.0, 9.0], (4, 16)), np.float32)
    W["l0.mix.left.out"] *= 0.1
    want = oracle.forward(cfg, W, seq)
    dec = decoder(backends[prec], cfg, W)
    for cut in (None, [100] + [1] * 60, [65, 3, 92]):
        assert close(everything(dec, seq, cut), want, prec), cut
    dec.close()


# -------------------------------------------------------------------- cuts, batches, slots (GPU)

@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("cut", [1, 2, 3, 7, 8, 16, 63, 64, 65, 128, [1, 2, 64, 1, 70, 128]])
def test_portions(backends, cut, prec):
    W, seq = weights(MIXED, 7), toks(300 if cut not in (1, 2) else 140, 4)
    dec = decoder(backends[prec], MIXED, W)
    want, ok = expected(MIXED, W, seq)
    assert agrees(everything(dec, seq, cut + [1] * 400 if isinstance(cut, list) else cut), want, ok, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_unequal_batch(backends, prec):
    """Rows of unequal length as one batch, then decoded together while shorter ones end earlier."""
    W = weights(MIXED, 8)
    seqs = [toks(n, 20 + n) for n in (1, 2, 67, 193, 64, 130, 3, 9, 71)]
    want = [expected(MIXED, W, s) for s in seqs]
    n = len(seqs)
    dec = decoder(backends[prec], MIXED, W, max_batch=n)
    B = backends[prec]
    tail = [0, 1, 9, 5, 3, 7, 1, 8, 6]
    slots = [dec.open_sequence() for _ in seqs]
    at = [len(s) - t for s, t in zip(seqs, tail)]
    ask = [(r, p) for r in range(n) for p in range(0, at[r], 7)]
    got = B.to_numpy(dec.run([(slots[r], seqs[r][:at[r]]) for r in range(n)], ask))
    assert agrees(got, [want[r][0][p] for r, p in ask], [want[r][1][p] for r, p in ask], prec)
    decoded = []
    while True:
        live = [r for r in range(n) if at[r] < len(seqs[r])]
        if not live:
            break
        got = B.to_numpy(dec.run([(slots[r], [seqs[r][at[r]]]) for r in live], [(k, 0) for k in range(len(live))]))
        for k, r in enumerate(live):
            decoded.append((got[k], want[r][0][at[r]], want[r][1][at[r]]))
            at[r] += 1
    assert agrees(*zip(*decoded), prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_mixed_portions_in_one_batch(backends, prec):
    """Rows that start, rows that go on by a portion and rows that go on by one token, together."""
    W, B = weights(MIXED, 12), backends[prec]
    seqs = [toks(n, 60 + n) for n in (90, 141, 77)]
    want = [expected(MIXED, W, s) for s in seqs]
    dec = decoder(B, MIXED, W, max_batch=3)
    slots = [dec.open_sequence() for _ in seqs]
    at, rows = [0, 0, 0], []
    for step in ((50, 0, 0), (1, 100, 0), (1, 1, 76), (37, 3, 1), (1, 37, 0)):
        live = [r for r in range(3) if step[r]]
        got = B.to_numpy(dec.run([(slots[r], seqs[r][at[r]:at[r] + step[r]]) for r in live],
                                 [(k, i) for k, r in enumerate(live) for i in range(step[r])]))
        i = 0
        for r in live:
            rows += [(got[i + j], want[r][0][at[r] + j], want[r][1][at[r] + j]) for j in range(step[r])]
            i += step[r]
            at[r] += step[r]
    assert at == [90, 141, 77] and agrees(*zip(*rows), prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_slots_are_reused_clean(backends, prec):
    W = weights(MIXED, 9)
    dec = decoder(backends[prec], MIXED, W, max_batch=2)
    a, b = toks(90, 40), toks(75, 41)
    other = dec.open_sequence()
    dec.run([(other, toks(33, 42))])
    for seq in (a, b, a[:1], b[:3]):     # all through the one free slot
        want, ok = expected(MIXED, W, seq)
        assert agrees(everything(dec, seq, [len(seq) // 2 or 1] * 3), want, ok, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_places_do_not_matter(backends, prec):
    """A sequence's logits do not depend on its slot or on its neighbours, beyond rounding."""
    W, B = weights(MIXED, 10), backends[prec]
    dec = decoder(B, MIXED, W, max_batch=4)
    seq = toks(100, 50)
    alone, ok = everything(dec, seq), expected(MIXED, W, seq)[1]
    s = [dec.open_sequence() for _ in range(3)]
    got = B.to_numpy(dec.run([(s[2], toks(41, 51)), (s[1], seq), (s[0], toks(170, 52))], [(1, k) for k in range(100)]))
    assert agrees(got, alone, ok, prec)
    dec.close()


def play(dec, seq, how):
    n, s, i = len(seq), dec.open_sequence(), 0
    for k in {"prompt": [n], "decode": [n - 1, 1], "portion": [n - 70, 70], "short": [n - 9, 9]}[how]:
        r = dec.run([(s, seq[i:i + k])], [(0, k - 1)])
        i += k
    dec.close_sequence(s)
    return dec.B.to_numpy(r)[0]


QUIET = range(40)      # tokens between the ones that matter


def telling(cfg, W, values):
    """A vector whose product with the first layer's normed input is values[token], and 0 for quiet tokens."""
    tokens = [t for t in QUIET if t not in values] + list(values)
    h = np.array([oracle.rms(W["embed"][t].astype(np.float64) * cfg["embedding"]["scale"], cfg["norm"]["eps"]) * W["l0.norm1"] for t in tokens])
    return np.linalg.lstsq(h, np.array([float(values.get(t, 0.0)) for t in tokens]), rcond=None)[0]


def rounded(w):
    return cg.synth.bf16_round(np.asarray(w, np.float32))


@functools.lru_cache(maxsize=None)
def far_keys(dim, vdim, slope):
    """A model, its weights and (distance, tokens, the oracle's last logits): the last token looks for one key,
    which stands out at every distance of interest: near, at the borders of key tiles, at the start.  A
    nearer token with the same key and another value competes with it by the distance alone."""
    cfg = model([par(heads=2, kv_heads=1, dim=dim, vdim=vdim, scale=1.0, temp=(0.3, 100), width=8, blocks=2)], side=0)
    W, n, p, rng = weights(cfg, 11), 450, "l0.mix.left.", np.random.default_rng(5)
    asks, sought, rival = 103, 102, 101
    k = rng.normal(size=dim)
    W[p + "k"] = rounded(np.outer(k, telling(cfg, W, {sought: 1, rival: 1, asks: 0})))
    W[p + "q"] = rounded(np.outer(np.concatenate([k, k]) * 14.0 / (k @ k), telling(cfg, W, {asks: 1, sought: 0, rival: 0})))
    W[p + "r1"], W[p + "r2"] = np.asarray([slope, 0.3 * slope], np.float32), np.asarray([0.3, 0.05], np.float32)
    W["l0.mix.right.out"] *= 0.1
    cases = []
    for back in (1, 2, 31, 32, 63, 64, 65, 127, 128, 129, 300, 449):
        seq = np.random.default_rng(back).integers(0, len(QUIET), n)
        seq[n - 1], seq[n - 1 - back] = asks, sought
        if back > 64:
            seq[n - 1 - back // 4] = rival
        want = oracle.forward(cfg, W, seq)[-1]
        swapped = seq.copy()
        swapped[n - 1 - back] = 0
        assert err(oracle.forward(cfg, W, swapped)[-1], want) > TOL["bf16"]
        if back > 64:
            assert err(oracle.forward(cfg, W, seq, faults=("no_distance",))[-1], want) > 300 * TOL["f32"]
        cases.append((back, seq, want))
    return cfg, W, cases


FAR = [(24, 20, 1.0), (64, 64, 0.2), (64, 128, 1.5), (128, 128, 1.0), (96, 256, 0.7), (300, 40, 1.0)]


@pytest.mark.parametrize("sizes", FAR)
def test_far_keys_decide(sizes):
    far_keys(*sizes)


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("sizes", FAR)
def test_far_keys(backends, sizes, prec):
    cfg, W, cases = far_keys(*sizes)
    dec = decoder(backends[prec], cfg, W)
    for back, seq, want in cases:
        for how in ("prompt", "decode", "portion", "short"):
            assert close(play(dec, seq, how), want, prec), (back, how)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_steep_distance_biases(backends, prec):
    """Biases of tens of units between neighbouring tokens and across a tile."""
    cfg = model([par(heads=3, kv_heads=1, dim=64, vdim=64), par(heads=3, kv_heads=3, dim=24, vdim=100)])
    W, seq = weights(cfg, 12), toks(330, 8)
    for l in (0, 1):
        W[f"l{l}.mix.left.r1"], W[f"l{l}.mix.left.r2"] = np.asarray([8.0, 0.01, 3.0], np.float32), np.asarray([4.0, 0.001, 10.0], np.float32)
    want = oracle.forward(cfg, W, seq)
    dec = decoder(backends[prec], cfg, W)
    assert close(everything(dec, seq), want, prec)
    assert close(everything(dec, seq, [200, 100] + [1] * 30), want, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("layer", [cdelta(heads=2, kv_heads=1, dim=32, vdim=32), gla(heads=2, dim=32, vdim=32), par(heads=1, kv_heads=1, width=32, blocks=2)])
def test_states_remember_far_tokens(backends, layer, prec):
    """A recurrence that forgets little: one large write, hundreds of tokens of small ones, then the read;
    across portions and chunks."""
    cfg = model([layer], side=0)
    W = weights(cfg, 21)
    kind, m = layer["type"], "l0.mix."
    seq = np.random.default_rng(4).integers(0, len(QUIET), 500)
    loud = telling(cfg, W, {102: 1.0})
    if kind == "channel_delta":
        W[m + "A_log"], W[m + "dt_bias"] = np.full(2, -4.0, np.float32), np.full(64, -4.0, np.float32)
        W[m + "b"] = rounded(np.tile(telling(cfg, W, {t: 4.0 if t == 102 else -7.0 for t in [*QUIET, 102]}), (2, 1)))
    elif kind == "gla":
        W[m + "a2.b"] = np.full(64, 9.0, np.float32)
        W[m + "a2"] = rounded(0.1 * W[m + "a2"])
        W[m + "k"] = rounded(0.1 * W[m + "k"] + np.outer(np.ones(64), loud))
    else:
        W[m + "right.lam"] = np.full(32, -8.0, np.float32)
        W[m + "right.x"] = rounded(0.02 * W[m + "right.x"] + 5.0 * np.outer(np.ones(32), loud))
        W[m + "right.x.b"] *= 0.0
        W[m + "right.conv.b"] *= 0.0
        W[m + "left.out"] = rounded(0.05 * W[m + "left.out"])
    seq[3], seq[499] = 102, 103
    other = seq.copy()
    other[3] = 5
    want = oracle.forward(cfg, W, seq)
    moved = err(oracle.forward(cfg, W, other)[-1], want[-1])
    assert moved > TOL["bf16"], moved
    dec = decoder(backends[prec], cfg, W)
    for cut in (None, 64, [100, 5, 7, 64, 1, 1, 200, 121, 1], [2] + [1] * 3 + [495]):
        got = everything(dec, seq.tolist(), cut)
        assert close(got, want, prec) and close(got[-1], want[-1], prec), cut
    dec.close()


@gpu
def test_residual_stream_of_a_bf16_context(backends):
    """A stream far larger than what the layers add: rounded to bf16 the additions would be lost."""
    cfg = model([gla(), moe(cdelta()), par()], scale=256.0)
    W = weights(cfg, 13)
    for i in range(3):
        W[f"l{i}.dwa"] = np.asarray([0.0] * (i + 1) + [1.0], np.float32)
    seq, layers, gaps = toks(80, 70), [], []
    oracle.forward(cfg, W, seq, hooks=lambda i, x: layers.append(x), gaps=gaps)
    ok = sure(gaps, 80)
    dec = decoder(backends["bf16"], cfg, W)
    dec.keep_residuals()
    everything(dec, seq)
    got = dec.residuals().astype(np.float64)
    assert agrees((got[-1] - got[0])[ok], (layers[-1] - layers[0])[ok], ok[ok], "bf16")
    dec.close()


# ------------------------------------------------------------------ generation and serving (GPU)

def greedy(cfg, W, prompt, n):
    """n + 1 greedy tokens of the oracle and the margins of its picks (0 at a close choice of experts)."""
    seq, out, margin = list(prompt), [], []
    for _ in range(n + 1):
        lg, ok = expected(cfg, W, seq)
        top = np.sort(lg[-1])
        out.append(int(lg[-1].argmax()))
        margin.append(float(top[-1] - top[-2]) / float(np.sqrt((lg[-1] ** 2).mean())) if ok[-1] else 0.0)
        seq.append(out[-1])
    return out, margin


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_greedy_generation(backends, prec):
    """cg_decoder_generate (captured decode graph), generate_batch and DecoderLM give the oracle's tokens."""
    B, W = backends[prec], weights(MIXED, 14)
    dec = decoder(B, MIXED, W, max_seq=96, max_batch=3)
    prompts = [toks(n, 80 + n) for n in (5, 37, 18)]
    ref = [greedy(MIXED, W, p, 12) for p in prompts]
    tol = 6 * TOL[prec]
    out = dec.generate_batch(prompts, 12)
    for r in range(3):
        assert same_up_to_ties(out[r], *ref[r], tol), r
    eq = dec.generate(np.asarray([prompts[1], prompts[1]]), 12)
    assert same_up_to_ties(eq[0], *ref[1], tol) and (eq[0] == eq[1]).all()
    # teacher-forced steps pick the same tokens as the captured graph replayed them
    dec.reset()
    dec.prefill(B.from_numpy(np.asarray([prompts[1]], dtype=np.uint32)))
    for t in eq[0][:12]:
        dec.step_with(B.from_numpy(np.asarray([t], dtype=np.uint32)))
    assert (dec.tokens()[0] == eq[0]).all()
    dec.reset()
    lm = cg.serve.DecoderLM(dec)
    first = [next(lm.complete(prompts[2]))]
    first += [next(lm) for _ in range(6)]
    assert same_up_to_ties(first, *ref[2], tol)
    # another context: a state cannot go back, so it starts again
    other = prompts[2][:11] + prompts[0]
    again = next(lm.complete(other))
    assert dec.position()[0] == len(other) and not dec.keeps_prefix
    assert same_up_to_ties([again], *greedy(MIXED, W, other, 0), tol)
    dec.close()


@gpu
def test_long_decoding(backends):
    """300 decode steps through the captured graph against one pass over the generated tokens."""
    B, W = backends["bf16"], weights(MIXED, 15)
    dec = decoder(B, MIXED, W, max_seq=400, max_batch=2)
    prompts = [toks(50, 90), toks(9, 91)]
    out = dec.generate_batch(prompts, 300)
    for p, o in zip(prompts, out):
        lg, ok = expected(MIXED, W, list(p) + o[:-1].tolist())
        lg, ok = lg[len(p) - 1:], ok[len(p) - 1:]
        top = np.sort(lg, axis=1)
        clear = ok & ((top[:, -1] - top[:, -2]) / np.sqrt((lg ** 2).mean()) > 6 * TOL["bf16"])
        assert clear.mean() > 0.1 and (lg.argmax(1)[clear] == o[clear]).all()
    dec.close()


@gpu
def test_prefill_append_and_prompt_portions(backends):
    """The equal-length entry points, with a workspace so small that the prompt runs in portions."""
    B, W = backends["f32"], weights(MIXED, 16)
    dec = decoder(B, MIXED, W, max_batch=2)
    ids = np.asarray([toks(230, 95), toks(230, 96)], dtype=np.uint32)
    want = [oracle.forward(MIXED, W, r) for r in ids]
    for chunk in (8192, 128, 200):
        B.set_option("prefill_chunk", chunk)
        lg = B.to_numpy(dec.prefill(B.from_numpy(ids[:, :200]), want_logits=True))
        assert all(close(lg[r], want[r][199], "f32") for r in range(2)), chunk
        lg = B.to_numpy(dec.append(B.from_numpy(ids[:, 200:]), want_logits=True))
        assert all(close(lg[r], want[r][229], "f32") for r in range(2)), chunk
    B.set_option("prefill_chunk", 8192)
    with pytest.raises(cg.BackendPanic):
        dec.truncate(181)
    dec.close()


@gpu
def test_bad_models_are_errors(backends):
    B, W = backends["bf16"], weights(MIXED, 17)
    for name in ("l1.mlp.e3.up", "l0.mlp.up.b", "l2.mix.right.ra", "l2.mix.left.out", "l0.mix.g1", "l3.dwa", "side.embed", "l4.side.norm", "l1.mix.a2.b"):
        bad = dict(W)
        del bad[name]
        with pytest.raises(cg.BackendPanic):
            decoder(B, MIXED, bad)
    bad = dict(W)
    bad["l0.mix.a2"] = bad["l0.mix.a2"][:, :-1]      # not the rank of a1
    with pytest.raises(cg.BackendPanic):
        decoder(B, MIXED, bad)
    for layer in (par(heads=3, kv_heads=2), gla(tau=0.0), cdelta(heads=3, kv_heads=2), cdelta(conv=0), moe(gla(), 4, 5)):
        with pytest.raises(cg.BackendPanic):
            cg.Decoder(B, cg.registry.config_from_json(model([layer])), max_seq=16, max_batch=1)


@gpu
@pytest.mark.parametrize("dtype,prec", [("float32", "f32"), ("bfloat16", "bf16")])
def test_trace_run_replays_a_trace(tmp_path, dtype, prec):
    """bin/trace_run on a checkpoint folder: unequal requests in one batch, then decoded together."""
    if not __import__("torch").cuda.is_available():
        pytest.skip("no CUDA device")
    W = weights(MIXED, 18)
    (tmp_path / "config.json").write_text(json.dumps(MIXED))
    cg.safetensors_io.write(str(tmp_path / "model.safetensors"), W.items())
    seqs = {"a": toks(40, 97), "b": toks(71, 98)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seqs["a"][:38], "want": [37, 0]}, {"id": "b", "tokens": seqs["b"][:69], "want": [5]}],
              "end": []},
             {"step": 1, "entries": [{"id": k, "tokens": [seqs[k][n]], "want": []} for k, n in (("a", 38), ("b", 69))], "end": []},
             {"step": 2, "entries": [{"id": k, "tokens": [seqs[k][n]], "want": [0]} for k, n in (("a", 39), ("b", 70))], "end": ["a", "b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens",
                        "111"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = {k: expected(MIXED, W, s) for k, s in seqs.items()}
    got = np.concatenate([np.fromfile(tmp_path / "0.f32", "<f4").reshape(3, -1), np.fromfile(tmp_path / "2.f32", "<f4").reshape(2, -1)])
    places = [("a", 37), ("a", 0), ("b", 5), ("a", 39), ("b", 70)]
    assert agrees(got, [want[k][0][i] for k, i in places], [want[k][1][i] for k, i in places], prec)
