"""Decoders of the Segedra design (windowed attention with a sink, hyper-connected streams, experts with
corrected routing, squared-relu feed-forwards, loops) against the plain restatement of its equations
in segedra_oracle.py: each mechanism alone, whole prompts, portions, decoding through the cache,
unequal batches, reused slots, window edges, and greedy generation through the decoder's entry points.

Errors are measured as in test_hybrid.py.  In a bf16 context a token whose choice of experts is a close
call may choose otherwise, so such tokens are left out there.
"""
import importlib
import json
import os
import subprocess

import numpy as np
import pytest

import segedra_oracle as oracle
from test_hybrid import ROOT, TOL, backends, close, decoder, err, everything, same_up_to_ties, toks  # noqa: F401

cg = importlib.import_module("catgrad-rs_b200")
gpu = pytest.mark.gpu


def att(heads=4, kv_heads=2, dim=24, vdim=20, window=20, rot=16, base=5000.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
         "mask": {"size": window} if window else None, "rot": {"base": base, "dims": rot} if rot else None}
    return {"type": "attention", "mixer": m, "mlp": None}


def dense(layer, ff=88):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def moe(layer, experts=7, top=3, ff=28, limit=0.9, scale=1.7):
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}})


def model(layers, width=72, vocab=104, loop=None, eps=1e-4, streams=3, scale=2.5):
    return {"architecture": "Segedra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "loop": loop,
            "streams": streams, "embedding": {"scale": scale}}


def weights(cfg, seed=0):
    """Random weights under which every mechanism carries weight: attention scores of a few units, sinks
    worth several keys, streams that differ, experts that reach their limits, corrections that
    change the choice."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in cg.registry.config_from_json(cfg).param_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        if ".hc" in name:
            s = cfg["streams"]
            w = {"in": rng.uniform(0.2, 0.5, shape) + 0.8 * (np.arange(s) == s - 1) if leaf == "in" else 0, "out": rng.uniform(0.2, 1.4, shape),
                 "mix": np.eye(s) * 0.7 + rng.uniform(-0.2, 0.2, (s, s)) + 0.9 * np.tri(s, k=-1) if leaf == "mix" else 0}[leaf]
        elif leaf == "sink":
            w = rng.normal(2.0, 1.0, shape)
        elif leaf == "correction":
            w = rng.normal(0, 0.3, shape)
        elif name.endswith((".q.norm", ".k.norm")):
            w = 1.3 + rng.normal(0, 0.3, shape)
        elif leaf.startswith("norm"):
            w = rng.normal(0, 0.3, shape)
        elif leaf == "embed":
            w = rng.normal(0, 0.5, shape)
        elif leaf == "router":
            w = rng.normal(0, 2.0 * shape[1] ** -0.5, shape)
        else:
            w = rng.normal(0, shape[1] ** -0.5, shape)
            if name.endswith((".mix.q", ".mix.k")):
                w *= np.geomspace(0.2, 2.5, shape[0])[:, None]     # heads differ in size
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


MIXED = model([dense(att()), att(heads=2, kv_heads=1, dim=16, vdim=32, window=33, rot=4), moe(att(window=0)),
               moe(att(heads=6, kv_heads=6, dim=8, vdim=8, window=5, rot=8), 4, 1, 20)],
              loop={"start": 1, "stop": 3, "times": 2})


# ---------------------------------------------------------------------------- configuration (CPU)

def test_config_reader_and_shapes():
    cfg = cg.registry.config_from_json(MIXED)
    assert cfg.layer_runs() == oracle.layer_runs(MIXED) == [0, 1, 2, 1, 2, 3]
    assert cfg.rms_norm_eps == 1e-4 and cfg.streams == 3 and cfg.embed_scale == 2.5 and not cfg.recurrent
    assert [L.window for L in cfg.layers] == [20, 33, 0, 5] and [L.rotated for L in cfg.layers] == [16, 4, 16, 8]
    assert cfg.layers[1].ffn == 0 and cfg.layers[0].experts is None and cfg.layers[2].experts.top == 3
    st = cfg.layers[2].struct(cfg.design)
    assert (st.mixer, st.act, st.experts, st.top_k, st.qk_norm, st.sink) == (4, 2, 7, 3, 1, 1) and abs(st.act_limit - 0.9) < 1e-12
    s = cfg.param_shapes()
    assert s["l0.mix.v"] == (40, 72) and s["l0.mix.o"] == (72, 80) and s["l2.mlp.e6.down"] == (72, 28) and s["l1.hc1.mix"] == (3, 3)
    assert "head" not in s and "l0.mlp.gate" not in s and "l1.norm2" not in s and "l1.hc2.in" not in s
    with pytest.raises(ValueError):
        cg.registry.config_from_json(model([dict(att(), type="delta")]))
    with pytest.raises(ValueError):
        cg.registry.config_from_json(model([dict(att(), mlp={"kind": "unheard of"})]))


@pytest.mark.parametrize("fault,layer", [
    ("wide", att()), ("narrow", att()), ("no_sink", att()), ("late_start", att()), ("norm_per_head", att()),
    ("transposed_mix", att()), ("no_correction", moe(att())), ("corrected_weights", moe(att())), ("renormalised", moe(att()))])
def test_planted_mistakes_would_show(fault, layer):
    """The inputs of these tests tell the equations from near misses: with the mistake planted in the
    oracle the logits move by thousands of times the f32 tolerance, and by more than twice the bf16 one."""
    cfg = model([layer, att(window=0)])
    W, seq = weights(cfg), toks(60, 1)
    moved = err(oracle.forward(cfg, W, seq, faults=(fault,)), oracle.forward(cfg, W, seq))
    assert moved > 2 * TOL["bf16"]


def test_rotation_oracle_preserves_relative_angles():
    rng = np.random.default_rng(0)
    q, k = rng.normal(size=16), rng.normal(size=16)
    dots = [oracle.rotate(q, p + 5, 1000.0, 10) @ oracle.rotate(k, p, 1000.0, 10) for p in (0, 3, 70)]
    assert np.allclose(dots, dots[0])


def test_window_oracle():
    assert [oracle.visible(i, {"size": 3}) for i in range(5)] == [0, 0, 0, 1, 2]
    assert oracle.visible(9, {"size": 1}) == 9 and oracle.visible(9, None) == 0


# --------------------------------------------------------------------- each mechanism alone (GPU)

ALONE = {
    "attention": [att()],
    "no_window": [att(window=0)],
    "window_1": [att(window=1)],
    "window_2": [att(window=2)],
    "window_64": [att(dim=64, vdim=64, window=64, rot=64)],
    "window_65": [att(dim=64, vdim=48, window=65, rot=32)],
    "window_beyond": [att(window=1000)],
    "one_head": [att(heads=1, kv_heads=1, dim=8, vdim=8, rot=2)],
    "no_rotation": [att(rot=0)],
    "many_queries_per_key": [att(heads=12, kv_heads=1, dim=16, vdim=16, window=40)],
    "eight_queries_per_key": [att(heads=16, kv_heads=2, dim=16, vdim=24, window=40)],
    "head_100": [att(heads=3, kv_heads=3, dim=100, vdim=36, window=50, rot=98, scale=0.2)],
    "head_128": [att(heads=4, kv_heads=1, dim=128, vdim=128, window=70, rot=64)],
    "head_256": [att(heads=2, kv_heads=1, dim=160, vdim=256, window=70, rot=20)],
    "head_300": [att(heads=2, kv_heads=1, dim=300, vdim=12, window=30, rot=300)],
    "dense": [dense(att())],
    "experts": [moe(att())],
    "one_of_many": [moe(att(), 16, 1)],
    "all_experts": [moe(att(), 5, 5, limit=0.4)],
    "single_expert": [moe(att(), 1, 1, 44, limit=5.0, scale=0.6)],
    "many_experts": [moe(att(), 40, 4, 12, limit=2.0, scale=3.0)],
    "narrow": [dense(att(heads=1, kv_heads=1, dim=6, vdim=5, rot=2), 13), moe(att(heads=3, kv_heads=1, dim=10, vdim=7, rot=6), 3, 2, 11)],
}


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(backends, name, prec):
    """Residual stream after every layer and logits at every position, in one portion and cut in ways
    that take the prompt kernels and the decode kernels."""
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
    assert agrees(everything(dec, seq, [139] + [1] * 11), want, ok, prec)
    assert agrees(everything(dec, seq, [70, 80]), want, ok, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("streams", [0, 1, 2, 4, 5, 9])
def test_streams(backends, streams, prec):
    cfg = model([dense(att()), moe(att(window=9))], streams=streams, scale=1.0 if streams == 1 else 3.0)
    W, seq = weights(cfg, 4), toks(70, 3)
    want, ok = expected(cfg, W, seq)
    dec = decoder(backends[prec], cfg, W)
    assert agrees(everything(dec, seq), want, ok, prec)
    assert agrees(everything(dec, seq, [40] + [1] * 30), want, ok, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 2), (1, 2, 4), (2, 3, 2)])
def test_loops(backends, loop, prec):
    cfg = model([att(), dense(att(window=7)), moe(att(window=30))], loop=loop and dict(zip(("start", "stop", "times"), loop)))
    W, seq = weights(cfg, 5), toks(60, 3)
    dec = decoder(backends[prec], cfg, W)
    want, ok = expected(cfg, W, seq)
    assert agrees(everything(dec, seq), want, ok, prec)
    assert agrees(everything(dec, seq, [49] + [1] * 11), want, ok, prec)
    dec.close()


@gpu
def test_wide_rows_take_the_persistent_kernels(backends):
    """Sizes at which the projections, the squared relu and the experts run on the persistent GEMMs."""
    for seed, n, ff in ((6, 600, 9216), (7, 1100, 8192)):
        cfg = model([dense(att(heads=2, kv_heads=1, dim=64, vdim=64, window=100, rot=32), ff), moe(att(window=10), 4, 2, 256)], width=1024, streams=2)
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
    for sink in ((-200.0, -5.0, 0.0, 4.0), (8.0, 3.0, 100.0, -100.0), (12.0, 12.0, 12.0, 12.0)):
        W["l0.mix.sink"] = np.asarray(sink, np.float32)
        want = oracle.forward(cfg, W, seq)
        dec = decoder(backends[prec], cfg, W)
        assert close(everything(dec, seq), want, prec), sink
        assert close(everything(dec, seq, [100] + [1] * 40), want, prec), sink
        dec.close()


# -------------------------------------------------------------------- cuts, batches, slots (GPU)

@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("cut", [1, 2, 3, 16, 63, 64, 65, 128, [1, 2, 64, 1, 70, 128]])
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


def seeking_model(window, dim, heads=2):
    """One layer without rotation whose queries of token 103 look for token 102 alone: its key stands
    out wherever it is visible."""
    cfg = model([att(heads=heads, kv_heads=1, dim=dim, vdim=dim, window=window, rot=0, scale=1.0)], streams=2)
    W, eps = weights(cfg, 11), cfg["norm"]["eps"]
    asks, sought = 103, 102
    h = {t: oracle.norm(W["embed"][t].astype(np.float64) * cfg["embedding"]["scale"] * W["l0.hc1.in"].sum(), W["l0.norm1"], eps)
         for t in (asks, sought)}
    k = oracle.rms(W["l0.mix.k"] @ h[sought], eps) * W["l0.mix.k.norm"]
    W["l0.mix.q"] = cg.synth.bf16_round(np.concatenate([np.outer(k / (k @ k), h[asks] / (h[asks] @ h[asks]))] * heads).astype(np.float32))
    W["l0.mix.q.norm"] = np.full(heads * dim, 30.0 / dim ** 0.5 / np.sqrt(np.mean(k * k)), np.float32)
    W["l0.mix.sink"] = np.full(heads, 12.0, np.float32)
    return cfg, W, asks, sought


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("how", ["prompt", "decode", "portion"])
@pytest.mark.parametrize("window,dim", [(0, 64), (1, 64), (2, 24), (40, 64), (63, 64), (64, 128), (65, 64), (127, 64), (128, 128), (129, 64),
                                        (200, 256), (300, 72), (385, 128)])
def test_far_keys_and_window_edges(backends, window, dim, how, prec):
    """The one key that stands out, at every distance of interest: near, at the borders of key tiles, and
    just inside and just outside the window."""
    cfg, W, asks, sought = seeking_model(window, dim)
    n = 520
    backs = (1, 63, 64, 65, 127, 128, 300, 511, 519) if not window else sorted({max(window - 2, 1), window - 1, window, window + 1} - {0})
    dec = decoder(backends[prec], cfg, W)
    got, want = [], []
    for back in backs:
        seq = np.random.default_rng(back).integers(0, 102, n)
        seq[n - 1], seq[n - 1 - back] = asks, sought
        want.append(oracle.forward(cfg, W, seq[-1 - (window or n) - 2:])[-1])   # (no rotation: only the window counts)
        swapped = seq.copy()
        swapped[n - 1 - back] = 0
        moved = err(oracle.forward(cfg, W, swapped[-1 - (window or n) - 2:])[-1], want[-1])
        assert moved > 4 * TOL["bf16"] if not window or back < window else moved == 0   # inside it decides, outside it does not exist
        s, i = dec.open_sequence(), 0
        for k in {"prompt": [n], "decode": [n - 1, 1], "portion": [n - 70, 70]}[how]:
            r = dec.run([(s, seq[i:i + k])], [(0, k - 1)])
            i += k
        got.append(dec.B.to_numpy(r)[0])
        dec.close_sequence(s)
    for back, g, w in zip(backs, got, want):
        assert close(g, w, prec), back
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_window_passes_over_decoded_tokens(backends, prec):
    """The sought token itself is decoded, and leaves the window while others are decoded."""
    cfg, W, asks, sought = seeking_model(23, 64)
    rng = np.random.default_rng(3)
    seq = rng.integers(0, 102, 90)
    seq[50] = sought
    seq[51:] = asks                       # every later token asks: 22 of them still see it
    want = oracle.forward(cfg, W, seq)
    assert err(want[72], want[73]) > 4 * TOL["bf16"]
    dec = decoder(backends[prec], cfg, W)
    assert close(everything(dec, seq.tolist(), [45] + [1] * 45), want, prec)
    dec.close()


@gpu
def test_residual_streams_are_f32_in_a_bf16_context(backends):
    """Streams far larger than what the layers add: rounded to bf16 the additions would be lost."""
    cfg = model([att(), dense(att()), att()], scale=256.0, streams=2)
    W = weights(cfg, 13)
    for k in W:
        if k.endswith(".mix") and ".hc" in k:
            W[k] = np.eye(2, dtype=np.float32)
    seq, layers = toks(80, 70), []
    oracle.forward(cfg, W, seq, hooks=lambda i, x: layers.append(x))
    dec = decoder(backends["bf16"], cfg, W)
    dec.keep_residuals()
    everything(dec, seq)
    got = dec.residuals().astype(np.float64)
    assert err(got[-1] - got[0], layers[-1] - layers[0]) < 4e-2
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
    # another context keeps the common prefix: the cached keys of what follows are written over
    other = prompts[2][:11] + prompts[0]
    again = next(lm.complete(other))
    assert dec.position()[0] == len(other)
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
def test_prefill_append_truncate_and_prompt_portions(backends):
    """The equal-length entry points, with a workspace so small that the prompt runs in portions, and
    going back to an earlier position."""
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
        dec.truncate(101)
        assert dec.position()[0] == 101
        lg = B.to_numpy(dec.append(B.from_numpy(ids[:, 101:180]), want_logits=True))
        assert all(close(lg[r], want[r][179], "f32") for r in range(2)), chunk
    B.set_option("prefill_chunk", 8192)
    with pytest.raises(cg.BackendPanic):
        dec.truncate(181)
    dec.close()


@gpu
def test_bad_models_are_errors(backends):
    B, W = backends["bf16"], weights(MIXED, 17)
    bad = dict(W)
    del bad["l2.mlp.e3.up"]
    with pytest.raises(cg.BackendPanic):
        decoder(B, MIXED, bad)
    for layer in (att(heads=3, kv_heads=2), att(rot=30), att(rot=5), moe(att(), 4, 5), moe(att(), limit=0.0)):
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


# ------------------------------------------------------- the attention kernels by themselves (GPU)

@gpu
@pytest.mark.parametrize("S,d,window", [(64, 64, 1), (130, 64, 64), (300, 128, 127), (300, 64, 128), (513, 128, 129), (200, 256, 50), (40, 64, 9),
                                        (260, 128, 1000)])
def test_fused_attention_windows(backends, S, d, window):
    B = backends["bf16"]
    rng = np.random.default_rng(S + window)
    q, k, v = (cg.synth.bf16_round(rng.normal(0, 1, (2, n, S, d)).astype(np.float32)) for n in (4, 2, 2))
    got = B.to_numpy(B.fused_attention(B.from_numpy(q), B.from_numpy(k), B.from_numpy(v), window=window))
    i, j = np.arange(S)[:, None], np.arange(S)[None]
    s = np.einsum("bhid,bhjd->bhij", q.astype(np.float64), np.repeat(k, 2, 1).astype(np.float64)) / d ** 0.5
    s[:, :, (j > i) | (i - j >= window)] = -np.inf
    p = np.exp(s - s.max(-1, keepdims=True))
    want = np.einsum("bhij,bhjd->bhid", p / p.sum(-1, keepdims=True), np.repeat(v, 2, 1).astype(np.float64))
    assert err(got, want) < 2e-2
