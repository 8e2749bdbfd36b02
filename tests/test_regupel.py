"""Decoders of the Regupel design (layer norms behind the sublayers; gated, per-head normed window
attention with a sink; window attention with kept first tokens beside lightning attention;
sigmoid-routed experts with weighted inputs and a shared expert; layers with another one's weights)
against the plain restatement of its equations in regupel_oracle.py: each mechanism alone, whole prompts,
portions, decoding through the cache and state, unequal batches, reused slots, edges of windows and of
the kept tokens, and greedy generation through the decoder's entry points.

Errors are measured as in test_hybrid.py.  In a bf16 context a token whose choice of experts is a close
call may choose otherwise, so such tokens are left out there.
"""
import importlib
import json
import os
import subprocess

import numpy as np
import pytest

import regupel_oracle as oracle
from test_hybrid import ROOT, TOL, backends, close, decoder, err, everything, same_up_to_ties, toks  # noqa: F401

cg = importlib.import_module("catgrad-rs_b200")
gpu = pytest.mark.gpu
SCALING = {"factor": 6.0, "low": 1.0, "high": 5.0, "original": 300}


def att(heads=4, kv_heads=2, dim=24, vdim=20, window=20, rot=16, base=5000.0, scale=1.4, scaling=SCALING):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
         "mask": {"size": window} if window else None, "rot": {"base": base, "dims": rot, "scaling": scaling} if rot else None}
    return {"type": "attention", "mixer": m, "mlp": None}


def par(heads=4, kv_heads=2, dim=24, vdim=20, window=20, kept=5, scale=0.3, rheads=3, rdim=16, rvdim=12, decay=None, left=0.7, right=1.2):
    decay = decay or [1.0 - 2.0 ** -(0.5 + 8.0 * h / max(rheads - 1, 1)) for h in range(rheads)]
    m = {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                  "mask": {"size": window, "keep_first": kept} if window else None},
         "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay}, "left_scale": left, "right_scale": right}
    return {"type": "parallel", "mixer": m, "mlp": None}


def moe(layer, experts=7, top=3, ff=28, shared=36):
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top},
                            "shared": {"ff": shared} if shared else None})


def model(layers, width=72, vocab=104, eps=1e-4, scale=2.5, mult=0.8, logit_scale=0.6):
    return {"architecture": "Regupel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "residual_mult": mult,
            "embedding": {"scale": scale}, "logit_scale": logit_scale}


def again(layer, of):
    return dict(layer, weights_of=of)


def weights(cfg, seed=0):
    """Random weights under which every mechanism carries weight: attention scores of a few units, sinks
    worth several keys, gates and routers away from one half, biases and gains that differ.  The routers
    read mostly the first components of the stream, where a token's embedding holds well separated levels
    that the layers hardly move: few choices are close calls, whose other outcome the following
    tokens would see."""
    rng = np.random.default_rng(seed)
    out = {}
    E = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if L["mlp"]] or [0])
    levels = np.array([rng.permutation(np.linspace(-2.5, 2.5, E)) for _ in range(cfg["vocab"])]).reshape(cfg["vocab"], E) / cfg["embedding"]["scale"]
    for name, shape in cg.registry.config_from_json(cfg).param_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "sink":
            w = rng.normal(2.0, 1.0, shape)
        elif leaf == "b":
            w = rng.normal(0, 0.4, shape)
        elif len(shape) == 1:
            w = 1.0 + rng.normal(0, 0.3, shape)
        elif leaf == "embed":
            w = rng.normal(0, 0.5, shape)
            w[:, :E] = levels
        elif leaf == "router":
            w = rng.normal(0, 0.15 * shape[1] ** -0.5, shape) + np.eye(*shape)
        elif name.endswith("mix.g"):
            w = rng.normal(0, 1.5 * shape[1] ** -0.5, shape)
        else:
            w = rng.normal(0, shape[1] ** -0.5, shape)
            if leaf in ("q", "k"):
                w *= np.geomspace(0.3, 2.0, shape[0])[:, None]     # heads differ in size
        if name.startswith("l") and ".norm" in name and ".mix." not in name:
            w[:E] *= 0.05
        out[name] = cg.synth.bf16_round(np.asarray(w, np.float32))
    return out


def sure(gaps, n):
    """Tokens none of whose expert choices is a close call."""
    return np.min(gaps, axis=0) > 0.02 if gaps else np.ones(n, bool)


def expected(cfg, W, seq, **kw):
    """The oracle's logits and which positions to compare in bf16."""
    gaps = []
    want = oracle.forward(cfg, W, seq, gaps=gaps, **kw)
    return want, sure(gaps, len(seq))


def agrees(got, want, ok, prec):
    ok = np.asarray(ok) if prec == "bf16" else np.ones(len(want), bool)
    assert ok.mean() > 0.25 or len(ok) < 20
    return not ok.any() or close(np.asarray(got)[ok], np.asarray(want)[ok], prec)


MIXED = model([moe(par(), shared=0), moe(att(heads=2, kv_heads=1, dim=16, vdim=32, window=33, rot=4)),
               par(heads=6, kv_heads=3, dim=8, vdim=16, window=9, kept=3, rheads=2, rdim=24, rvdim=40),
               again(moe(att(heads=2, kv_heads=1, dim=16, vdim=32, window=33, rot=4)), 1), moe(par(window=40, kept=70, rheads=5), 4, 1, 20)])


# ---------------------------------------------------------------------------- configuration (CPU)

def test_config_reader_and_shapes():
    cfg = cg.registry.config_from_json(MIXED)
    assert cfg.rms_norm_eps == 1e-4 and cfg.embed_scale == 2.5 and cfg.residual_mult == 0.8 and cfg.logit_scale == 0.6 and cfg.recurrent
    assert not cg.registry.config_from_json(model([att()])).recurrent
    assert [cfg.owner(i) for i in range(5)] == [0, 1, 2, 1, 4] and cfg.layer_runs() == list(range(5))
    st = cfg.layers[1].struct(cfg.design)
    assert (st.mixer, st.qk_norm, st.sink, st.gate, st.rot_half, st.window, st.keep_first) == (4, 2, 1, 1, 1, 33, 0)
    assert (st.experts, st.top_k, st.scoring, st.weigh_input, st.correction, st.shared_ffn, st.weights_of) == (7, 3, 1, 1, 0, 36, 0)
    assert (st.rot_factor, st.rot_low, st.rot_high, st.rot_original) == (6.0, 1.0, 5.0, 300.0)
    assert cfg.layers[3].struct(cfg.design).weights_of == 2
    st = cfg.layers[2].struct(cfg.design)
    right = type(st).from_address(st.beside)
    assert (st.mixer, st.qk_norm, st.sink, st.gate, st.keep_first, st.ffn, right.mixer, right.heads, right.dim) == (4, 1, 0, 0, 3, 0, 5, 2, 24)
    assert (st.out_scale, right.out_scale) == (0.7, 1.2)
    assert np.ctypeslib.as_array((np.ctypeslib.ctypes.c_double * 2).from_address(right.decay)).tolist() == MIXED["layers"][2]["mixer"]["right"]["decay"]
    s = cfg.param_shapes()
    assert s["l0.mix.left.v"] == (40, 72) and s["l0.mix.right.g"] == (36, 72) and s["l0.mix.right.o"] == (72, 36) and s["l1.mix.g"] == (2, 72)
    assert s["l1.mlp.shared.down"] == (72, 36) and s["l4.mlp.e3.up"] == (20, 72) and s["l1.norm2.b"] == s["final.norm.b"] == (72,)
    assert not any(k.startswith("l3.") for k in s) and not {"head", "l0.mlp.shared.up", "l2.norm2", "l0.norm1b", "l1.mlp.correction"} & set(s)
    for bad in (dict(att(), type="delta"), dict(att(), mlp={"kind": "dense", "ff": 8})):
        with pytest.raises(ValueError):
            cg.registry.config_from_json(model([bad]))
    with pytest.raises(ValueError):
        L = cg.registry.config_from_json(model([par(rheads=3, decay=[0.5, 0.9])]))
        L.layers[0].struct(L.design)


def test_struct_mirror_matches_the_header():
    import re
    text = open(os.path.join(ROOT, "include", "catgrad_cuda.h")).read()
    body = text[text.index("typedef struct cg_layer_config {"):text.index("} cg_layer_config;")]
    body = re.sub(r"/\*.*?\*/", "", body, flags=re.S).split("{", 1)[1]
    kinds = {"int32_t": 4, "double": 8, "const double*": 8, "const struct cg_layer_config*": 8}
    fields = []
    for stmt in body.split(";"):
        m = re.match(r"\s*((?:const )?(?:struct )?\w+\s*\*?)\s*(.+)", stmt.strip().replace("\n", " "))
        if m:
            kind = re.sub(r"\s+\*", "*", m.group(1).strip())
            fields += [(n.strip(), kinds[kind]) for n in m.group(2).split(",")]
    mirror = importlib.import_module("catgrad-rs_b200.layered").LayerStruct._fields_
    assert fields == [(n, np.ctypeslib.ctypes.sizeof(t)) for n, t in mirror]


FAULTS = [(f, att()) for f in ("wide", "narrow", "no_sink", "late_start", "neighbours", "unscaled", "no_head_norm", "no_gate", "pre_norm",
                               "uncentred", "no_bias", "no_mult")]
FAULTS += [(f, par()) for f in ("no_first", "more_first", "fewer_first", "narrow", "norm_per_head", "swapped_scales", "lost_state", "no_silu",
                                "decays_first", "norm_per_value_head", "silu_gate")]
FAULTS += [(f, moe(att())) for f in ("renormalised", "weighted_output", "no_shared")]


@pytest.mark.parametrize("fault,layer", FAULTS)
def test_planted_mistakes_would_show(fault, layer):
    """The inputs of these tests tell the equations from near misses: with the mistake planted in the
    oracle the logits move by hundreds of times the f32 tolerance."""
    cfg = model([layer, att(window=0)])
    W, seq = weights(cfg), toks(60, 1)
    moved = err(oracle.forward(cfg, W, seq, faults=(fault,)), oracle.forward(cfg, W, seq))
    assert moved > 1000 * TOL["f32"], moved


def test_oracle_masks_and_frequencies():
    mask = {"size": 3, "keep_first": 2}
    assert [oracle.visible(i, mask).tolist() for i in (0, 2, 4, 9)] == [[0], [0, 1, 2], [0, 1, 2, 3, 4], [0, 1, 7, 8, 9]]
    assert oracle.visible(2, {"size": 1, "keep_first": 9}).tolist() == [0, 1, 2] and oracle.visible(5, {"size": 1}).tolist() == [5]
    rot = {"base": 10000.0, "dims": 32, "scaling": SCALING}
    f, g = oracle.frequencies(rot), oracle.frequencies(dict(rot, scaling=None))
    ratio, turns = g / f, 300 * g / (2 * np.pi)
    assert np.allclose(ratio[turns > 5], 1) and np.allclose(ratio[turns < 1], 6)
    between = ratio[(turns > 1) & (turns < 5)]
    assert len(between) and (between > 1).all() and (between < 6).all()


def test_recurrence_oracle_is_a_decaying_sum():
    """The state read at a token is the decayed sum over all tokens before it."""
    rng = np.random.default_rng(0)
    m = {"heads": 2, "dim": 3, "vdim": 4, "decay": [0.5, 0.9]}
    T, W = 12, 8
    P = {n: rng.normal(size=(r, W)) for n, r in (("q", 6), ("k", 6), ("v", 8), ("g", 8))}
    P["o"], P["norm"] = np.eye(8), np.ones(8)
    h = rng.normal(size=(T, W))
    got = oracle.lightning(h, P.__getitem__, m, 1e-6)
    q, k, v = (oracle.silu(h @ P[n].T).reshape(T, 2, -1) for n in "qkv")
    o = np.array([[sum(m["decay"][n] ** (t - s) * (q[t, n] @ k[s, n]) * v[s, n] for s in range(t + 1)) for n in range(2)] for t in range(T)])
    assert np.allclose(got, oracle.rms(o.reshape(T, 8), 1e-6) * oracle.sigmoid(h @ P["g"].T))


# --------------------------------------------------------------------- each mechanism alone (GPU)

ALONE = {
    "attention": [att()],
    "attention_no_window": [att(window=0)],
    "attention_window_1": [att(window=1)],
    "attention_window_64": [att(dim=64, vdim=64, window=64, rot=64)],
    "attention_window_beyond": [att(window=1000)],
    "attention_no_rotation": [att(rot=0)],
    "attention_two_rotated": [att(rot=2)],
    "attention_unscaled_rotation": [att(scaling=None)],
    "attention_one_head": [att(heads=1, kv_heads=1, dim=8, vdim=8, rot=8)],
    "attention_many_queries_per_key": [att(heads=12, kv_heads=1, dim=16, vdim=16, window=40)],
    "attention_eight_queries_per_key": [att(heads=16, kv_heads=2, dim=16, vdim=24, window=40)],
    "attention_head_100": [att(heads=3, kv_heads=3, dim=100, vdim=36, window=50, rot=98)],
    "attention_head_128": [att(heads=4, kv_heads=1, dim=128, vdim=96, window=70, rot=64)],
    "attention_head_256": [att(heads=2, kv_heads=1, dim=160, vdim=256, window=70, rot=20)],
    "attention_head_300": [att(heads=2, kv_heads=1, dim=300, vdim=12, window=30, rot=300)],
    "parallel": [par()],
    "parallel_no_window": [par(window=0)],
    "parallel_nothing_kept": [par(kept=0)],
    "parallel_one_kept": [par(kept=1, window=1)],
    "parallel_kept_beyond_the_window": [par(kept=33, window=7)],
    "parallel_kept_64": [par(dim=64, vdim=64, kept=64, window=16, heads=6, kv_heads=2)],
    "parallel_kept_65": [par(dim=64, vdim=48, kept=65, window=20)],
    "parallel_head_128": [par(dim=128, vdim=64, kept=4, window=30, rdim=128, rvdim=128)],
    "parallel_head_256": [par(heads=2, kv_heads=1, dim=200, vdim=160, kept=40, window=50, rdim=100, rvdim=72)],
    "parallel_head_300": [par(heads=2, kv_heads=1, dim=300, vdim=10, kept=6, window=11)],
    "parallel_many_queries_per_key": [par(heads=10, kv_heads=1, kept=6, window=11)],
    "parallel_one_recurrent_head": [par(rheads=1, rdim=5, rvdim=3, decay=[0.8])],
    "parallel_wide_recurrence": [par(rheads=2, rdim=144, rvdim=20)],
    "parallel_wide_values": [par(rheads=2, rdim=48, rvdim=200)],
    "parallel_decays": [par(rheads=5, rdim=32, rvdim=32, decay=[0.0, 1.0, 1e-3, 0.9999, 0.5])],
    "parallel_scales": [par(left=-1.7, right=0.05), par(left=0.02, right=3.0)],
    "experts": [moe(att())],
    "one_of_many": [moe(att(), 16, 1)],
    "all_experts": [moe(att(), 5, 5)],
    "single_expert": [moe(att(), 1, 1, 44, 20)],
    "many_experts": [moe(par(), 40, 4, 12, 100)],
    "no_shared_expert": [moe(att(), shared=0)],
    "shared_weights": [moe(par()), att(), again(moe(par()), 0), again(att(), 1), again(moe(par()), 0)],
    "weights_of_a_later_layer": [again(moe(att()), 1), moe(att())],
    "narrow": [moe(par(heads=1, kv_heads=1, dim=6, vdim=5, window=9, kept=2, rheads=1, rdim=3, rvdim=7), 3, 2, 11, 13),
               att(heads=3, kv_heads=1, dim=10, vdim=7, rot=6)],
}


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(backends, name, prec):
    """Residual stream after every layer and logits at every position, in one portion and cut in ways
    that take the prompt kernels, those of short portions and the decode kernels."""
    cfg = model(ALONE[name], width=44 if name == "narrow" else 72, vocab=101 if name == "narrow" else 104)
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
@pytest.mark.parametrize("mult,scale,logit_scale,eps", [(1.0, 1.0, 1.0, 1e-6), (0.3, 12.0, 0.1, 1e-2), (2.0, 0.25, 7.0, 0.5)])
def test_constants(backends, mult, scale, logit_scale, eps, prec):
    cfg = model([moe(par()), att()], mult=mult, scale=scale, logit_scale=logit_scale, eps=eps)
    W, seq = weights(cfg, 4), toks(70, 3)
    want, ok = expected(cfg, W, seq)
    dec = decoder(backends[prec], cfg, W)
    assert agrees(everything(dec, seq), want, ok, prec)
    assert agrees(everything(dec, seq, [40] + [1] * 30), want, ok, prec)
    dec.close()


@gpu
def test_wide_rows_take_the_persistent_kernels(backends):
    """Sizes at which the projections (silu among them) and the experts run on the persistent GEMMs."""
    for seed, n, ff in ((6, 600, 256), (7, 1100, 512)):
        cfg = model([moe(par(heads=4, kv_heads=2, dim=64, vdim=64, window=100, kept=20, rheads=8, rdim=128, rvdim=128), 4, 2, ff, 2048),
                     att(heads=2, kv_heads=1, dim=64, vdim=64, window=90, rot=32)], width=1024)
        W, seq = weights(cfg, seed), toks(n, seed)
        want, ok = expected(cfg, W, seq)
        dec = decoder(backends["bf16"], cfg, W, max_seq=1104, max_batch=1)
        assert agrees(everything(dec, seq), want, ok, "bf16")
        dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_strong_and_weak_sinks(backends, prec):
    """Sinks from nothing to nearly everything, and beyond what an exponential can hold."""
    cfg = model([att(heads=4, kv_heads=1, dim=64, vdim=64, window=50)])
    W, seq = weights(cfg, 8), toks(140, 5)
    for sink in ((-200.0, -5.0, 0.0, 4.0), (8.0, 3.0, 100.0, -100.0)):
        W["l0.mix.sink"] = np.asarray(sink, np.float32)
        want = oracle.forward(cfg, W, seq)
        dec = decoder(backends[prec], cfg, W)
        assert close(everything(dec, seq), want, prec), sink
        assert close(everything(dec, seq, [100] + [1] * 40), want, prec), sink
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
    seqs = [toks(n, 20 + n) for n in (1, 2, 67, 193, 64, 130)]
    want = [expected(MIXED, W, s) for s in seqs]
    dec = decoder(backends[prec], MIXED, W, max_batch=6)
    B = backends[prec]
    tail = [0, 1, 9, 5, 3, 7]
    slots = [dec.open_sequence() for _ in seqs]
    at = [len(s) - t for s, t in zip(seqs, tail)]
    ask = [(r, p) for r in range(6) for p in range(0, at[r], 7)]
    got = B.to_numpy(dec.run([(slots[r], seqs[r][:at[r]]) for r in range(6)], ask))
    assert agrees(got, [want[r][0][p] for r, p in ask], [want[r][1][p] for r, p in ask], prec)
    decoded = []
    while True:
        live = [r for r in range(6) if at[r] < len(seqs[r])]
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


def seeking_model(layer, side, n_heads, dim, sink=None):
    """One layer in which the queries of token 103 look for the keys of token 102 alone, which stand out
    wherever they are visible."""
    cfg = model([layer])
    W, eps = weights(cfg, 11), cfg["norm"]["eps"]
    asks, sought, p = 103, 102, f"l0.mix.{side}"
    h = {t: W["embed"][t].astype(np.float64) * cfg["embedding"]["scale"] for t in (asks, sought)}
    k = W[p + "k"].astype(np.float64) @ h[sought]
    W[p + "q"] = cg.synth.bf16_round(np.concatenate([np.outer(k * 3.0 / (k @ k) ** 0.5, h[asks] / (h[asks] @ h[asks]))] * n_heads).astype(np.float32))
    if sink is None:
        k = oracle.rms(k, eps) * W[p + "k.norm"]
        W[p + "q"] = cg.synth.bf16_round(np.concatenate([np.outer(k / (k @ k), h[asks] / (h[asks] @ h[asks]))] * n_heads).astype(np.float32))
        W[p + "q.norm"] = np.full(n_heads * dim, 30.0 / dim ** 0.5 / np.sqrt(np.mean(k * k)), np.float32)
    else:
        W[p + "sink"] = np.full(n_heads, sink, np.float32)
    return cfg, W, asks, sought


def play(dec, seq, how):
    n, s, i = len(seq), dec.open_sequence(), 0
    for k in {"prompt": [n], "decode": [n - 1, 1], "portion": [n - 70, 70], "short": [n - 9, 9]}[how]:
        r = dec.run([(s, seq[i:i + k])], [(0, k - 1)])
        i += k
    dec.close_sequence(s)
    return dec.B.to_numpy(r)[0]


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("how", ["prompt", "decode", "portion", "short"])
@pytest.mark.parametrize("window,dim", [(0, 64), (2, 24), (40, 64), (63, 64), (64, 128), (65, 64), (128, 128), (129, 64), (200, 256), (300, 72)])
def test_far_keys_and_window_edges(backends, window, dim, how, prec):
    """Gated attention: the one key that stands out, at every distance of interest: near, at the borders of
    key tiles, and just inside and just outside the window."""
    cfg, W, asks, sought = seeking_model(att(heads=2, kv_heads=1, dim=dim, vdim=dim, window=window, rot=0, scale=30.0 / dim), "", 2, dim, 12.0)
    n = 450
    backs = (1, 63, 64, 65, 127, 128, 300, 449) if not window else sorted({max(window - 2, 1), window - 1, window, window + 1} - {0})
    dec = decoder(backends[prec], cfg, W)
    for back in backs:
        seq = np.random.default_rng(back).integers(0, 102, n)
        seq[n - 1], seq[n - 1 - back] = asks, sought
        short = slice(-1 - (window or n) - 2, None)   # (no rotation: only the window counts)
        want = oracle.forward(cfg, W, seq[short])[-1]
        swapped = seq.copy()
        swapped[n - 1 - back] = 0
        moved = err(oracle.forward(cfg, W, swapped[short])[-1], want)
        assert moved > 4 * TOL["bf16"] if not window or back < window else moved == 0   # inside it decides, outside it does not exist
        assert close(play(dec, seq, how), want, prec), back
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("how", ["prompt", "decode", "portion", "short"])
@pytest.mark.parametrize("window,kept,dim", [(5, 1, 64), (40, 20, 24), (64, 64, 64), (63, 65, 128), (130, 63, 64), (20, 128, 64), (70, 129, 128),
                                             (50, 30, 256), (33, 200, 64), (50, 10, 300)])
def test_first_tokens_and_window_edges(backends, window, kept, dim, how, prec):
    """Windows with kept first tokens: the key that stands out among the first ones kept, just past them,
    and at both sides of the window's edge."""
    layer = par(heads=2, kv_heads=1, dim=dim, vdim=dim, window=window, kept=kept, scale=1.0, left=1.5, right=0.1)
    cfg, W, asks, sought = seeking_model(layer, "left.", 2, dim)
    n = 420
    dec = decoder(backends[prec], cfg, W)
    for at in sorted({0, kept // 2, kept - 1, kept, kept + 1, n - 1 - window, n - window, n - 2}):
        seq = np.random.default_rng(at).integers(0, 102, n)
        seq[n - 1], seq[at] = asks, sought
        want = oracle.forward(cfg, W, seq)[-1]
        hidden = oracle.forward(cfg, W, seq, faults=("no_first",))[-1]
        if at < kept and at <= n - 1 - window:
            assert err(hidden, want) > 4 * TOL["bf16"]       # seen only because it is kept
        elif kept <= at <= n - 1 - window:
            more = oracle.forward(cfg, W, seq, faults=("more_first",) if at == kept else ("wide",))[-1]
            assert at not in (kept, n - 1 - window) or err(more, want) > 4 * TOL["bf16"]   # one more token would show
        assert close(play(dec, seq, how), want, prec), at
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_window_passes_over_decoded_tokens(backends, prec):
    """The sought token itself is decoded, and leaves the window while others are decoded; the same at a
    kept place stays."""
    layer = par(heads=2, kv_heads=1, dim=64, vdim=64, window=23, kept=4, scale=1.0, left=1.5, right=0.1)
    cfg, W, asks, sought = seeking_model(layer, "left.", 2, 64)
    for place in (50, 3):
        seq = np.random.default_rng(3).integers(0, 102, 90)
        seq[place] = sought
        seq[51:] = asks                       # every later token asks: 22 of them still see place 50
        want = oracle.forward(cfg, W, seq)
        assert place == 3 or err(want[72], want[73]) > 4 * TOL["bf16"]
        dec = decoder(backends[prec], cfg, W)
        assert close(everything(dec, seq.tolist(), [45] + [1] * 45), want, prec)
        dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_state_remembers_far_tokens(backends, prec):
    """A recurrence that forgets little: one large write, hundreds of tokens of small ones, then the read;
    across portions and chunks."""
    cfg = model([par(rheads=2, rdim=32, rvdim=32, decay=[0.9999, 0.99], left=0.05, right=2.0)])
    W = weights(cfg, 21)
    W["embed"][:100] *= 0.05                    # the tokens between write and read little
    W["embed"] = cg.synth.bf16_round(W["embed"])
    seq = np.random.default_rng(4).integers(0, 100, 500)
    seq[3], seq[499] = 102, 103
    other = seq.copy()
    other[3] = 5
    want = oracle.forward(cfg, W, seq)
    assert err(oracle.forward(cfg, W, other)[-1], want[-1]) > 2 * TOL["bf16"]
    dec = decoder(backends[prec], cfg, W)
    for cut in (None, 64, [100, 5, 7, 64, 1, 1, 200, 121, 1], [2] + [1] * 3 + [495]):
        got = everything(dec, seq.tolist(), cut)
        assert close(got, want, prec) and close(got[-1], want[-1], prec), cut
    dec.close()


@gpu
def test_residual_stream_and_inputs_of_experts_in_a_bf16_context(backends):
    """A stream far larger than what the layers add: rounded to bf16 the additions would be lost."""
    cfg = model([att(), moe(att()), par()], scale=256.0, mult=0.05)
    W = weights(cfg, 13)
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
    again_ = next(lm.complete(other))
    assert dec.position()[0] == len(other) and not dec.keeps_prefix
    assert same_up_to_ties([again_], *greedy(MIXED, W, other, 0), tol)
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
    for name in ("l1.mlp.e3.up", "l0.norm1.b", "l0.mix.right.g", "l1.mlp.shared.up", "l1.mix.sink"):
        bad = dict(W)
        del bad[name]
        with pytest.raises(cg.BackendPanic):
            decoder(B, MIXED, bad)
    for layer in (att(heads=3, kv_heads=2), att(rot=30), att(rot=5), moe(att(), 4, 5), par(rheads=1, decay=[1.5]), again(att(), 0)):
        cfg = model([layer])
        with pytest.raises(cg.BackendPanic):
            cg.Decoder(B, cg.registry.config_from_json(cfg), max_seq=16, max_batch=1)


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
