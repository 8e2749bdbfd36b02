"""Decoders built layer by layer (the Ralapel design) against the plain restatement of its equations
in hybrid_oracle.py: each mechanism alone, whole prompts, portions, decoding through the cache and
state, unequal batches, reused slots, loops, and greedy generation through the decoder's entry points.

Errors are root mean squares over the vocabulary (or the width), relative to those of the expected
values.  The f32 context has to agree to a few 1e-5, the bf16 context to the size its roundings have.
"""
import importlib
import json
import subprocess
import sys
import os

import numpy as np
import pytest

import hybrid_oracle as oracle

cg = importlib.import_module("catgrad-rs_b200")
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
gpu = pytest.mark.gpu
TOL = {"f32": 3e-5, "bf16": 4e-2}


def latent(heads=3, dim=24, rot_dim=8, vdim=20, kv_rank=40, base=10000.0, scale=None):
    return {"type": "latent_attention", "mlp": None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"type": "delta", "mlp": None, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def ssd(heads=4, groups=2, state=16, vdim=24, norm_groups=2, conv=4):
    return {"type": "mamba2", "mlp": None,
            "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "norm_groups": norm_groups, "conv": conv}}


def with_ff(layer, ff=88):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def model(layers, width=72, vocab=104, loop=None, eps=1e-5):
    return {"architecture": "Ralapel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "loop": loop}


def weights(cfg, seed=0):
    """Random weights under which every mechanism carries weight: unit-scale products, attention
    scores of a few units (a far key can win), decays from one token to hundreds."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in cg.registry.config_from_json(cfg).param_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "A_log":
            w = rng.uniform(-2.5, 1.5, shape)
        elif leaf == "dt_bias":
            w = rng.uniform(-4.0, 0.0, shape)
        elif name.endswith("conv.b"):
            w = rng.normal(0, 0.2, shape)
        elif name.endswith("conv"):
            w = rng.normal(0, shape[1] ** -0.5, shape)
        elif leaf in ("norm1b", "norm2b"):
            w = 0.4 + rng.normal(0, 0.1, shape)      # keeps the roundings of a looped model from growing
        elif len(shape) == 1:
            w = 1.0 + rng.normal(0, 0.2, shape)
        elif leaf == "embed":
            w = rng.normal(0, 1.0, shape)
        else:
            w = rng.normal(0, (2.0 if leaf in ("q", "dkv") else 1.0) * shape[1] ** -0.5, shape)
        out[name] = cg.synth.bf16_round(w.astype(np.float32))
    return out


@pytest.fixture(scope="module")
def backends():
    if not __import__("torch").cuda.is_available():
        pytest.skip("no CUDA device")
    return {"f32": cg.CudaBackend(0, cg.PREC_F32), "bf16": cg.CudaBackend(0, cg.PREC_BF16)}


def decoder(B, cfg, W, max_seq=640, max_batch=4):
    dec = cg.Decoder(B, cg.registry.config_from_json(cfg), max_seq=max_seq, max_batch=max_batch)
    dec.load(W.items())
    return dec


def err(got, want):
    """Largest per-position error of got [.., n] against want, relative to want's overall size."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.sqrt(((got - want) ** 2).mean(-1)).max() / np.sqrt((want ** 2).mean()))


def close(got, want, prec):
    """f32: every position.  bf16: a recurrence's read-out is normed, so a position whose read-out
    happens to be small shows its roundings enlarged; one in ten may, up to five times."""
    got, want = np.atleast_2d(np.asarray(got, np.float64)), np.atleast_2d(np.asarray(want, np.float64))
    e = np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
    if os.environ.get("HYBRID_ERRORS"):
        print(prec, len(e), "median %.2e, 0.9 quantile %.2e, largest %.2e" % (np.median(e), np.quantile(e, 0.9), e.max()))
    if prec == "f32":
        return e.max() < TOL["f32"]
    return np.quantile(e, 0.9) < TOL["bf16"] and e.max() < 5 * TOL["bf16"]


def toks(n, seed, vocab=104):
    return np.random.default_rng(1000 + seed).integers(0, vocab, n).tolist()


def everything(dec, seq, cut=None):
    """Logits at every position of one sequence, run in portions of `cut` tokens (None: at once)."""
    s = dec.open_sequence()
    out, i = [], 0
    cuts = cut if isinstance(cut, list) else [cut or len(seq)] * len(seq)
    for n in cuts:
        part = seq[i:i + n]
        if not part:
            break
        out.append(dec.B.to_numpy(dec.run([(s, part)], [(0, k) for k in range(len(part))])))
        i += len(part)
    dec.close_sequence(s)
    return np.concatenate(out)


MIXED = model([delta(heads=2, kv_heads=1, dim=24, vdim=16, conv=2), ssd(), with_ff(latent()), with_ff(delta(), 40), latent(heads=2, dim=16)],
              loop={"start": 2, "stop": 4, "times": 2})


# ---------------------------------------------------------------------------- configuration (CPU)

def test_config_reader_and_shapes():
    cfg = cg.registry.config_from_json(MIXED)
    assert cfg.layer_runs() == [i for i, _ in oracle.layer_runs(MIXED)] == [0, 1, 2, 3, 2, 3, 4]
    assert cfg.rms_norm_eps == 1e-5 and cfg.layers[2].ffn == 88 and cfg.layers[0].ffn == 0
    s = cfg.param_shapes()
    assert s["l1.mix.in"] == (4 * 24 * 2 + 2 * 2 * 16 + 4, 72) and s["l2.mix.dkv"] == (48, 72) and s["loop.in"] == (72, 144)
    plain = cg.registry.config_from_json(model([delta()]))
    assert plain.loop is None and "loop.in" not in plain.param_shapes()
    with pytest.raises(ValueError):
        cg.registry.config_from_json({"architecture": "nothing like it"})
    with pytest.raises(ValueError):
        cg.registry.config_from_json(model([dict(delta(), type="unheard of")]))


def test_registry_reads_other_families():
    c = cg.registry.config_from_json({"architectures": ["LlamaForCausalLM"], "hidden_size": 64, "intermediate_size": 128, "num_hidden_layers": 2,
                                      "num_attention_heads": 4, "num_key_value_heads": 2, "vocab_size": 100, "rms_norm_eps": 1e-5})
    assert c.arch == "llama" and c.head_dim == 16


@pytest.mark.parametrize("fault,mixer", [("drop_first", latent()), ("skip_self", latent()), ("read_first", delta())])
def test_planted_mistakes_would_show(fault, mixer):
    """The inputs of these tests tell the equations from near misses: with the mistake planted in the
    oracle the logits move by far more than any tolerance used here."""
    cfg = model([mixer])
    W, seq = weights(cfg), toks(60, 1)
    good, bad = oracle.forward(cfg, W, seq), oracle.forward(cfg, W, seq, faults=(fault,))
    assert err(bad, good) > 5 * TOL["bf16"]


def test_rotation_oracle_preserves_relative_angles():
    rng = np.random.default_rng(0)
    q, k = rng.normal(size=16), rng.normal(size=16)
    dots = [oracle.rotate_pairs(q, p + 5, 1000.0) @ oracle.rotate_pairs(k, p, 1000.0) for p in (0, 3, 70)]
    assert np.allclose(dots, dots[0])


# --------------------------------------------------------------------- each mechanism alone (GPU)

ALONE = {
    "latent": [latent()],
    "latent_one_head": [latent(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, base=77.0)],
    "latent_uneven": [latent(heads=5, dim=20, rot_dim=6, vdim=36, kv_rank=27, scale=0.31)],
    "latent_128": [latent(heads=2, dim=64, rot_dim=32, vdim=100, kv_rank=96)],
    "latent_192": [latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=136)],
    "latent_wide_values": [latent(heads=2, dim=16, rot_dim=16, vdim=264, kv_rank=64)],
    "delta": [delta()],
    "delta_equal_heads": [delta(heads=2, kv_heads=2, dim=32, vdim=32, conv=3)],
    "delta_one_head": [delta(heads=1, kv_heads=1, dim=8, vdim=40, conv=1)],
    "delta_uneven": [delta(heads=6, kv_heads=2, dim=20, vdim=36, conv=5)],
    "delta_128": [delta(heads=4, kv_heads=2, dim=128, vdim=128)],
    "delta_64": [delta(heads=2, kv_heads=1, dim=64, vdim=96, conv=2)],
    "ssd": [ssd()],
    "ssd_one_group": [ssd(heads=3, groups=1, state=24, vdim=16, norm_groups=1, conv=2)],
    "ssd_groups": [ssd(heads=6, groups=3, state=12, vdim=20, norm_groups=6, conv=5)],
    "ssd_128": [ssd(heads=4, groups=1, state=128, vdim=64, norm_groups=1)],
    "ssd_no_conv": [ssd(heads=2, groups=2, state=32, vdim=48, norm_groups=4, conv=1)],
    # beyond what the tensor-core kernels take
    "latent_rank_600": [latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=600)],
    "delta_wide": [delta(heads=2, kv_heads=1, dim=136, vdim=144, conv=3)],
    "ssd_wide": [ssd(heads=2, groups=1, state=144, vdim=136, norm_groups=2, conv=6)],
    "feed_forward": [with_ff(ssd(heads=1, groups=1, state=8, vdim=8, norm_groups=1), 44)],
    "narrow": [with_ff(latent(heads=1, dim=6, rot_dim=2, vdim=5, kv_rank=11), 13), delta(heads=3, kv_heads=1, dim=5, vdim=7)],
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
    want = oracle.forward(cfg, W, seq, hooks=lambda kind, i, x: layers.append(x))
    dec = decoder(backends[prec], cfg, W)
    dec.keep_residuals()
    got = everything(dec, seq)
    got_layers = dec.residuals()
    for i, x in enumerate(layers):
        assert close(got_layers[i], x, prec), i
    assert close(got, want, prec)
    dec.keep_residuals(False)
    assert close(everything(dec, seq, [139] + [1] * 11), want, prec)
    assert close(everything(dec, seq, [70, 80]), want, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 2), (1, 2, 4), (2, 3, 2)])
def test_loops(backends, loop, prec):
    cfg = model([delta(), with_ff(latent()), ssd()], loop=loop and dict(zip(("start", "stop", "times"), loop)))
    W, seq = weights(cfg, 5), toks(40, 3)
    dec = decoder(backends[prec], cfg, W)
    want = oracle.forward(cfg, W, seq)
    assert close(everything(dec, seq), want, prec)
    assert close(everything(dec, seq, [33, 1, 1, 1, 1, 1, 1, 1]), want, prec)
    dec.close()


# -------------------------------------------------------------------- cuts, batches, slots (GPU)

@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("cut", [1, 2, 3, 16, 63, 64, 65, 128, [1, 2, 64, 1, 70, 128]])
def test_portions(backends, cut, prec):
    W, seq = weights(MIXED, 7), toks(300 if cut not in (1, 2) else 140, 4)
    dec = decoder(backends[prec], MIXED, W)
    want = oracle.forward(MIXED, W, seq)
    assert close(everything(dec, seq, cut + [1] * 400 if isinstance(cut, list) else cut), want, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_unequal_batch(backends, prec):
    """Rows of unequal length as one batch, then decoded together while shorter ones end earlier."""
    W = weights(MIXED, 8)
    seqs = [toks(n, 20 + n) for n in (1, 2, 67, 193, 64, 130)]
    want = [oracle.forward(MIXED, W, s) for s in seqs]
    dec = decoder(backends[prec], MIXED, W, max_batch=6)
    B = backends[prec]
    tail = [0, 1, 9, 5, 3, 7]
    slots = [dec.open_sequence() for _ in seqs]
    at = [len(s) - t for s, t in zip(seqs, tail)]
    ask = [(r, p) for r in range(6) for p in range(0, at[r], 7)]
    got = B.to_numpy(dec.run([(slots[r], seqs[r][:at[r]]) for r in range(6)], ask))
    assert close(got, [want[r][p] for r, p in ask], prec)
    decoded = []
    while True:
        live = [r for r in range(6) if at[r] < len(seqs[r])]
        if not live:
            break
        got = B.to_numpy(dec.run([(slots[r], [seqs[r][at[r]]]) for r in live], [(k, 0) for k in range(len(live))]))
        for k, r in enumerate(live):
            decoded.append((got[k], want[r][at[r]]))
            at[r] += 1
    assert close(*zip(*decoded), prec)
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
        assert close(everything(dec, seq, [len(seq) // 2 or 1] * 3), oracle.forward(MIXED, W, seq), prec)
    with pytest.raises(cg.BackendPanic):
        s = dec.open_sequence()
        dec.open_sequence()
    dec.close_sequence(s)
    with pytest.raises(cg.BackendPanic):
        dec.run([(s, [1])])              # closed
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_places_do_not_matter(backends, prec):
    """A sequence's logits do not depend on its slot or on its neighbours, beyond rounding."""
    W, B = weights(MIXED, 10), backends[prec]
    dec = decoder(B, MIXED, W, max_batch=4)
    seq = toks(100, 50)
    alone = everything(dec, seq)
    s = [dec.open_sequence() for _ in range(3)]
    got = B.to_numpy(dec.run([(s[2], toks(41, 51)), (s[1], seq), (s[0], toks(170, 52))], [(1, k) for k in range(100)]))
    assert close(got, alone, prec)
    dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
@pytest.mark.parametrize("how", ["prompt", "decode"])
def test_far_keys(backends, how, prec):
    """One key stands out: the last token's query is made to look for one other token, which stands
    1 to 519 places back and nowhere else."""
    lay = latent(heads=2, dim=32, rot_dim=4, vdim=32, kv_rank=64, base=1e6, scale=1.0)
    cfg = model([lay])
    W = weights(cfg, 11)
    n, asks, sought, eps = 520, 103, 102, cfg["norm"]["eps"]
    h = {t: oracle.rms(oracle.rms(W["embed"][t].astype(np.float64), eps) * W["embed.norm"], eps) * W["l0.norm1"] for t in (asks, sought)}
    c = oracle.rms(W["l0.mix.dkv"][:64] @ h[sought], eps) * W["l0.mix.dkv.norm"]
    for i in range(2):
        k = W["l0.mix.uk"][i * 32:(i + 1) * 32] @ c
        W["l0.mix.q"][i * 36:i * 36 + 32] = np.outer(40 * k / (k @ k), h[asks] / (h[asks] @ h[asks]))
    W["l0.mix.q"] = cg.synth.bf16_round(W["l0.mix.q"])
    for back in (1, 63, 64, 65, 127, 128, 300, 511, 519):
        seq = np.random.default_rng(back).integers(0, 102, n)
        seq[n - 1], seq[n - 1 - back] = asks, sought
        want = oracle.forward(cfg, W, seq)[-1]
        swapped = seq.copy()
        swapped[n - 1 - back] = 0
        assert err(oracle.forward(cfg, W, swapped)[-1], want) > 3 * TOL["bf16"]   # the far key decides
        dec = decoder(backends[prec], cfg, W)
        cuts = [n] if how == "prompt" else [n - 1, 1]
        s = dec.open_sequence()
        i = 0
        for k in cuts:
            got = dec.B.to_numpy(dec.run([(s, seq[i:i + k])], [(0, k - 1)]))[0]
            i += k
        assert close(got, want, prec), back
        dec.close()


@gpu
@pytest.mark.parametrize("prec", ["f32", "bf16"])
def test_long_memory_of_the_recurrences(backends, prec):
    """Slow decays: the first tokens still show in the state after hundreds of others."""
    cfg = model([delta(heads=2, kv_heads=1, dim=48, vdim=32), ssd(heads=2, groups=1, state=48, vdim=32, norm_groups=1)])
    W = weights(cfg, 12)
    for k in W:
        if k.endswith("A_log"):
            W[k] = np.full_like(W[k], -6.0)
        if k == "l0.mix.b":
            W[k] = W[k] * 0.25
    seq = toks(420, 60)
    want = oracle.forward(cfg, W, seq)
    changed = oracle.forward(cfg, W, [(t + 1) % 104 for t in seq[:8]] + seq[8:])
    assert err(changed[-40:], want[-40:]) > 2e-3
    dec = decoder(backends[prec], cfg, W)
    assert close(everything(dec, seq), want, prec)
    assert close(everything(dec, seq, [200, 150] + [1] * 70), want, prec)
    dec.close()


@gpu
def test_residual_stream_is_f32_in_a_bf16_context(backends):
    """A residual stream far larger than what the layers add: rounded to bf16 the additions would be lost."""
    cfg = model([delta(), ssd(), with_ff(latent())])
    W = weights(cfg, 13)
    W["embed.norm"] = W["embed.norm"] * 256.0
    for k in W:
        if k.endswith("norm1b") or k.endswith("norm2b"):
            W[k] = W[k] * 0.5
    seq, layers = toks(80, 70), []
    oracle.forward(cfg, W, seq, hooks=lambda kind, i, x: layers.append(x))
    dec = decoder(backends["bf16"], cfg, W)
    dec.keep_residuals()
    everything(dec, seq)
    got = dec.residuals().astype(np.float64)
    assert err(got[-1] - got[0], layers[-1] - layers[0]) < 4e-2
    dec.close()


# ------------------------------------------------------------------ generation and serving (GPU)

def greedy(cfg, W, prompt, n):
    """n + 1 greedy tokens of the oracle and the margins of its picks."""
    seq, out, margin = list(prompt), [], []
    for _ in range(n + 1):
        lg = oracle.forward(cfg, W, seq)[-1]
        top = np.sort(lg)
        out.append(int(lg.argmax()))
        margin.append(float(top[-1] - top[-2]) / float(np.sqrt((lg ** 2).mean())))
        seq.append(out[-1])
    return out, margin


def same_up_to_ties(got, want, margin, tol):
    for g, w, m in zip(got, want, margin):
        if g != w:
            return m < tol     # from a near tie on the sequences may differ
    return True


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
    # a context that extends the old one keeps the state; one that does not starts again
    again = [next(lm.complete(prompts[2] + first[:7] + [3])), next(lm.complete(prompts[0]))]
    assert same_up_to_ties(again[1:], *ref[0], tol)
    dec.close()


@gpu
def test_long_decoding(backends):
    """300 decode steps through the captured graph against one pass over the generated tokens."""
    B, W = backends["bf16"], weights(MIXED, 15)
    dec = decoder(B, MIXED, W, max_seq=400, max_batch=2)
    prompts = [toks(50, 90), toks(9, 91)]
    out = dec.generate_batch(prompts, 300)
    for p, o in zip(prompts, out):
        lg = oracle.forward(MIXED, W, list(p) + o[:-1].tolist())[len(p) - 1:]
        top = np.sort(lg, axis=1)
        sure = (top[:, -1] - top[:, -2]) / np.sqrt((lg ** 2).mean()) > 6 * TOL["bf16"]
        assert sure.mean() > 0.2 and (lg.argmax(1)[sure] == o[sure]).all()
    dec.close()


@gpu
def test_prefill_append_and_prompt_portions(backends):
    """The equal-length entry points, with a workspace so small that the prompt runs in portions."""
    B, W = backends["bf16"], weights(MIXED, 16)
    dec = decoder(B, MIXED, W, max_batch=2)
    ids = np.asarray([toks(230, 95), toks(230, 96)], dtype=np.uint32)
    want = [oracle.forward(MIXED, W, r) for r in ids]
    for chunk in (8192, 128, 200):
        B.set_option("prefill_chunk", chunk)
        lg = B.to_numpy(dec.prefill(B.from_numpy(ids[:, :200]), want_logits=True))
        assert all(close(lg[r], want[r][199], "bf16") for r in range(2)), chunk
        lg = B.to_numpy(dec.append(B.from_numpy(ids[:, 200:]), want_logits=True))
        assert all(close(lg[r], want[r][229], "bf16") for r in range(2)), chunk
        assert dec.position()[0] == 230
    B.set_option("prefill_chunk", 8192)
    with pytest.raises(cg.BackendPanic):
        dec.truncate(100)
    dec.truncate(230)
    dec.close()


@gpu
def test_bad_input_is_an_error_not_a_fault(backends):
    B, W = backends["bf16"], weights(MIXED, 17)
    dec = decoder(B, MIXED, W, max_seq=32, max_batch=2)
    s = dec.open_sequence()
    with pytest.raises(cg.BackendPanic):
        dec.run([(s, toks(33, 1))])
    with pytest.raises(cg.BackendPanic):
        dec.run([(s, toks(3, 1))], [(0, 5)])
    with pytest.raises(cg.BackendPanic):
        dec.run([(s, [1]), (s, [2])])
    dec.close()
    bad = dict(W)
    del bad["l3.mix.k.conv"]
    with pytest.raises(cg.BackendPanic):
        decoder(B, MIXED, bad)


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
    want = {k: oracle.forward(MIXED, W, s) for k, s in seqs.items()}
    got0 = np.fromfile(tmp_path / "0.f32", "<f4").reshape(3, -1)
    got2 = np.fromfile(tmp_path / "2.f32", "<f4").reshape(2, -1)
    assert not (tmp_path / "1.f32").exists()
    assert close(np.concatenate([got0, got2]), [want["a"][37], want["a"][0], want["b"][5], want["a"][39], want["b"][70]], prec)
