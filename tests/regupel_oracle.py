"""A plain, slow restatement of the Regupel equations in numpy float64, one function per mechanism.

tests/test_regupel.py compares the library with it.  It shares no code with the library: sequences are
run one at a time, attention one query at a time, the recurrence one token at a time, experts one token
at a time, and nothing is fused, batched, grouped, chunked or cached.  A checkpoint is a dict name ->
array, a configuration is the parsed config.json.

`hooks` (optional) receives (run index, residual stream [T, width]) after every layer run; `gaps`, a
list, receives per routed layer run how far each token's last chosen expert is ahead of the next [T].
`faults` lets a test plant a mistake here, on the CPU, to see that its inputs would show it.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps, faults=()):
    d = x - (0.0 if "uncentred" in faults else x.mean(axis=-1, keepdims=True))
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w + (0.0 if "no_bias" in faults else b)


def frequencies(rot, faults=()):
    """Angular frequency of each rotated pair, with the wavelength-dependent stretching of long contexts."""
    n = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * np.arange(n // 2) / n)
    s = rot.get("scaling")
    if not s or "unscaled" in faults:
        return f
    out = []
    for fi in f:
        wave = 2.0 * np.pi / fi
        short, long = s["original"] / s["high"], s["original"] / s["low"]
        if wave < short:
            out.append(fi)
        elif wave > long:
            out.append(fi / s["factor"])
        else:
            t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - t) * fi / s["factor"] + t * fi)
    return np.array(out)


def rotate(x, pos, freqs, faults=()):
    """Components (i, i + n) of x [..., d] turn by pos * freqs[i], n the number of frequencies."""
    n = len(freqs)
    out = x.copy()
    for i in range(n):
        a = pos * freqs[i]
        iu, iv = (2 * i, 2 * i + 1) if "neighbours" in faults else (i, i + n)
        u, v = x[..., iu], x[..., iv]
        out[..., iu] = u * np.cos(a) - v * np.sin(a)
        out[..., iv] = v * np.cos(a) + u * np.sin(a)
    return out


def visible(i, mask, faults=()):
    """Positions that position i sees."""
    j = np.arange(i + 1)
    if not mask or not mask.get("size"):
        return j
    size = mask["size"] + ("wide" in faults) - ("narrow" in faults)
    keep = mask.get("keep_first") or 0
    keep = 0 if "no_first" in faults else keep + ("more_first" in faults) - ("fewer_first" in faults)
    return j[(i - j < size) | (j < keep)]


def sink_softmax(s, sink):
    """exp(s_j) / (sum_j exp(s_j) + exp(sink)); sink None: plain."""
    top = s.max() if sink is None else max(s.max(), sink)
    e = np.exp(s - top)
    return e / (e.sum() + (0.0 if sink is None else np.exp(sink - top)))


def attend(q, k, v, m, sink, faults=()):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv], one query at a time."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.empty((T, H, v.shape[2]))
    for t in range(T):
        j = visible(t, m.get("mask"), faults)
        for n in range(H):
            g = n // (H // G)
            w = sink_softmax(k[j, g] @ q[t, n] * m["scale"], None if sink is None else sink[n])
            out[t, n] = w @ v[j, g]
    return out


def attention(h, P, m, eps, faults=()):
    """Rotated, per-head normed attention with a sink and a gate per head; P(name) gives a tensor."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ P("q").T).reshape(T, H, d), (h @ P("k").T).reshape(T, G, d), (h @ P("v").T).reshape(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        f = frequencies(rot, faults)
        late = 1 if "late_start" in faults else 0
        q = np.stack([rotate(q[t], t + late, f, faults) for t in range(T)])
        k = np.stack([rotate(k[t], t, f, faults) for t in range(T)])
    if "no_head_norm" not in faults:
        q, k = rms(q, eps), rms(k, eps)
    out = attend(q, k, v, m, None if "no_sink" in faults else P("sink"), faults)
    if "no_gate" not in faults:
        out = out * sigmoid(h @ P("g").T)[:, :, None]
    return out.reshape(T, H * dv) @ P("o").T


def normed_attention(h, P, m, eps, faults=()):
    """Unrotated attention with norms over all query and over all key heads, first tokens kept."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = h @ P("q").T, h @ P("k").T, (h @ P("v").T).reshape(T, G, dv)
    if "norm_per_head" in faults:
        q = rms(q.reshape(T, H, d), eps).reshape(T, H * d) * P("q.norm")
    else:
        q = rms(q, eps) * P("q.norm")
    k = rms(k, eps) * P("k.norm")
    out = attend(q.reshape(T, H, d), k.reshape(T, G, d), v, m, None, faults)
    return out.reshape(T, H * dv) @ P("o").T


def lightning(h, P, m, eps, faults=()):
    """S <- decay S + k v^T, read by q, one token at a time."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    act = (lambda z: z) if "no_silu" in faults else silu
    q, k = act(h @ P("q").T).reshape(T, H, d), act(h @ P("k").T).reshape(T, H, d)
    v = act(h @ P("v").T).reshape(T, H, dv)
    S = np.zeros((H, d, dv))
    out = np.empty((T, H, dv))
    for t in range(T):
        if "lost_state" in faults and t == T // 2:
            S[:] = 0.0
        for n in range(H):
            new = np.outer(k[t, n], v[t, n])
            S[n] = m["decay"][n] * (S[n] + new) if "decays_first" in faults else m["decay"][n] * S[n] + new
            out[t, n] = S[n].T @ q[t, n]
    o = out.reshape(T, H * dv)
    if "norm_per_value_head" in faults:
        o = rms(out, eps).reshape(T, H * dv) * P("norm")
    else:
        o = rms(o, eps) * P("norm")
    g = h @ P("g").T
    return (o * (silu(g) if "silu_gate" in faults else sigmoid(g))) @ P("o").T


def parallel(h, P, m, eps, faults=()):
    left = normed_attention(h, lambda n: P("left." + n), m["left"], eps, faults)
    right = lightning(h, lambda n: P("right." + n), m["right"], eps, faults)
    ls, rs = m["left_scale"], m["right_scale"]
    if "swapped_scales" in faults:
        ls, rs = rs, ls
    return ls * left + rs * right


def gated_mlp(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, top, faults=()):
    """(expert, weight) pairs of one token."""
    s = sigmoid(router @ h)
    chosen = np.argsort(-s, kind="stable")[:top]
    w = s[chosen]
    if "renormalised" in faults:
        w = w / w.sum()
    return list(zip(chosen.tolist(), w))


def choice_gap(h, router, top):
    """How far the last chosen expert's score is ahead of the next one's."""
    c = np.sort(sigmoid(router @ h))[::-1]
    return c[top - 1] - c[top] if top < len(c) else np.inf


def experts_mlp(h, P, m, faults=(), gaps=None):
    r = m["router"]
    out = np.zeros_like(h)
    if m.get("shared") and "no_shared" not in faults:
        out = out + gated_mlp(h, P("shared.gate"), P("shared.up"), P("shared.down"))
    if gaps is not None:
        gaps.append(np.array([choice_gap(t, P("router"), r["top"]) for t in h]))
    for t in range(h.shape[0]):
        for e, w in route(h[t], P("router"), r["top"], faults):
            mats = P(f"e{e}.gate"), P(f"e{e}.up"), P(f"e{e}.down")
            out[t] += w * gated_mlp(h[t], *mats) if "weighted_output" in faults else gated_mlp(w * h[t], *mats)
    return out


def forward(cfg, W, tokens, hooks=None, faults=(), gaps=None):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps, mult = cfg["norm"]["eps"], 1.0 if "no_mult" in faults else cfg["residual_mult"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for run, L in enumerate(cfg["layers"]):
        i = L.get("weights_of", run)
        l = f"l{i}."
        mixer = {"attention": attention, "parallel": parallel}[L["type"]]

        def sublayer(x, q, f):
            n = f"{l}norm{q}"
            if "pre_norm" in faults:
                return x + mult * f(layer_norm(x, W[n], W[n + ".b"], eps))
            return x + mult * layer_norm(f(x), W[n], W[n + ".b"], eps, faults)

        x = sublayer(x, 1, lambda h: mixer(h, lambda n: W[f"{l}mix.{n}"], L["mixer"], eps, faults))
        if L["mlp"]:
            x = sublayer(x, 2, lambda h: experts_mlp(h, lambda n: W[f"{l}mlp.{n}"], L["mlp"], faults, gaps))
        if hooks:
            hooks(run, x)
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["embed"].T * cfg["logit_scale"]
