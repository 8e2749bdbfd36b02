"""A plain, slow restatement of the Segedra equations in numpy float64, one function per mechanism.

tests/test_segedra.py compares the library with it.  It shares no code with the library: sequences are
run one at a time, attention one query at a time, experts one token at a time, and nothing is fused,
batched, grouped or cached.  A checkpoint is a dict name -> array, a configuration is the parsed
config.json.

`hooks` (optional) receives (run index, sum of the streams [T, width]) after every layer run; `gaps`, a
list, receives per routed layer run how far each token's last chosen expert is ahead of the next [T].
`faults` lets a test plant a mistake here, on the CPU, to see that its inputs would show it.
"""
from __future__ import annotations

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """RMS norm with the gain 1 + w."""
    return rms(x, eps) * (1.0 + w)


def rotate(x, pos, base, dims):
    """Components (2i, 2i + 1) of the first `dims` of x [..., d] turn by pos * base^(-2i / dims)."""
    out = x.copy()
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def sink_softmax(s, sink):
    """exp(s_j) / (sum_j exp(s_j) + exp(sink)); sink None: plain."""
    top = s.max() if sink is None else max(s.max(), sink)
    e = np.exp(s - top)
    return e / (e.sum() + (0.0 if sink is None else np.exp(sink - top)))


def visible(i, mask, faults=()):
    """First position that position i sees."""
    if not mask or not mask.get("size"):
        return 0
    size = mask["size"] + ("wide" in faults) - ("narrow" in faults)
    return max(0, i - size + 1)


def attention(h, P, m, eps, faults=()):
    """h [T, width]; P(name) gives a tensor of the mixer."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = h @ P("q").T, h @ P("k").T, (h @ P("v").T).reshape(T, G, dv)
    if "norm_per_head" in faults:
        q = rms(q.reshape(T, H, d), eps).reshape(T, H * d) * P("q.norm")
    else:
        q = rms(q, eps) * P("q.norm")
    k = rms(k, eps) * P("k.norm")
    q, k = q.reshape(T, H, d), k.reshape(T, G, d)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    late = 1 if "late_start" in faults else 0
    q = np.stack([rotate(q[t], t + late, rot["base"], rot["dims"]) for t in range(T)])
    k = np.stack([rotate(k[t], t, rot["base"], rot["dims"]) for t in range(T)])
    sink = P("sink")
    out = np.empty((T, H, dv))
    for t in range(T):
        lo = visible(t, m.get("mask"), faults)
        for n in range(H):
            g = n // (H // G)
            w = sink_softmax(k[lo:t + 1, g] @ q[t, n] * m["scale"], None if "no_sink" in faults else sink[n])
            out[t, n] = w @ v[lo:t + 1, g]
    return out.reshape(T, H * dv) @ P("o").T


def squared_relu_mlp(h, P):
    return (np.maximum(h @ P("up").T, 0.0) ** 2) @ P("down").T


def expert(h, gate, up, down, limit):
    """Bounded gated unit: the gate from above, the linear part on both sides and shifted by one."""
    g = np.minimum(gate @ h, limit)
    u = np.clip(up @ h, -limit, limit)
    return down @ (g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0))


def route(h, router, correction, top, scale, faults=()):
    """(expert, weight) pairs of one token: chosen by corrected scores, weighted by plain ones."""
    z = router @ h
    s = np.exp(z - z.max())
    s /= s.sum()
    choice = s if "no_correction" in faults else s + correction
    chosen = np.argsort(-choice, kind="stable")[:top]
    w = (choice if "corrected_weights" in faults else s)[chosen] * scale
    if "renormalised" in faults:
        w = w / s[chosen].sum()
    return list(zip(chosen.tolist(), w))


def choice_gap(h, router, correction, top):
    """How far the last chosen expert's corrected score is ahead of the next one's."""
    z = router @ h
    s = np.exp(z - z.max())
    c = np.sort(s / s.sum() + correction)[::-1]
    return c[top - 1] - c[top] if top < len(c) else np.inf


def experts_mlp(h, P, m, faults=(), gaps=None):
    out = np.zeros_like(h)
    r = m["router"]
    if gaps is not None:
        gaps.append(np.array([choice_gap(t, P("router"), P("correction"), r["top"]) for t in h]))
    for t in range(h.shape[0]):
        for e, w in route(h[t], P("router"), P("correction"), r["top"], r["scale"], faults):
            out[t] += w * expert(h[t], P(f"e{e}.gate"), P(f"e{e}.up"), P(f"e{e}.down"), m["expert"]["limit"])
    return out


def streams_in(x, w):
    """x [s, T, width] -> one row per token."""
    return np.einsum("s,stw->tw", w, x)


def streams_out(x, y, mix, out, faults=()):
    """mix[from, to]."""
    if "transposed_mix" in faults:
        mix = mix.T
    return np.einsum("st,snw->tnw", mix, x) + out[:, None, None] * y


def layer_runs(cfg):
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


def forward(cfg, W, tokens, hooks=None, faults=(), gaps=None):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x0 = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    plain = not cfg["streams"]               # no streams: a residual sum
    x = np.stack([x0] * (cfg["streams"] or 1))
    for run, i in enumerate(layer_runs(cfg)):
        L, l = cfg["layers"][i], f"l{i}."

        def sublayer(x, q, f):
            if plain:
                return x + f(norm(x[0], W[f"{l}norm{q}"], eps))
            y = f(norm(streams_in(x, W[f"{l}hc{q}.in"]), W[f"{l}norm{q}"], eps))
            return streams_out(x, y, W[f"{l}hc{q}.mix"], W[f"{l}hc{q}.out"], faults)

        x = sublayer(x, 1, lambda h: attention(h, lambda n: W[f"{l}mix.{n}"], L["mixer"], eps, faults))
        m = L["mlp"]
        if m and m["kind"] == "dense":
            x = sublayer(x, 2, lambda h: squared_relu_mlp(h, lambda n: W[f"{l}mlp.{n}"]))
        elif m:
            x = sublayer(x, 2, lambda h: experts_mlp(h, lambda n: W[f"{l}mlp.{n}"], m, faults, gaps))
        if hooks:
            hooks(run, x.sum(0))
    return norm(x.sum(0), W["final.norm"], eps) @ W["embed"].T
