"""A plain, slow restatement of the Kivorax equations in numpy float64, one function per mechanism.

tests/test_kivorax.py compares the library with it.  It shares no code with the library: sequences are
run one at a time, attention one query at a time, the recurrences and convolutions one token at a time,
experts one token at a time, and nothing is fused, batched, grouped, chunked or cached.  A checkpoint
is a dict name -> array, a configuration is the parsed config.json.

`hooks` (optional) receives (layer, the residual stream [T, width] behind it); `gaps`, a list,
receives per routed layer how far each token's last chosen expert is ahead of the next [T].
`faults` lets a test plant a mistake here, on the CPU, to see that its inputs would show it.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def short_conv(x, taps, bias=0.0, faults=()):
    """Every channel's weighted sum of its last inputs, the newest under the last tap."""
    n = taps.shape[1]
    if "taps_reversed" in faults:
        taps = taps[:, ::-1]
    out = np.zeros_like(x)
    for t in range(len(x)):
        for j in range(n):
            if t - j >= 0 and not ("lost_tail" in faults and t - j < len(x) // 2 <= t):
                out[t] += taps[:, n - 1 - j] * x[t - j]
    return out + bias


def temperature(p, coef, every, faults=()):
    if "no_temperature" in faults:
        return 1.0
    return 1.0 + coef * np.log(np.floor((p + ("late_temperature" not in faults)) / every) + 1.0)


def biased_attention(h, P, m, faults=()):
    """Causal attention whose scores lose r1 ln(1 + r2 distance), queries warmed with the position, the
    heads' outputs gated element by element."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ P("q").T).reshape(T, H, d), (h @ P("k").T).reshape(T, G, d), (h @ P("v").T).reshape(T, G, dv)
    t = m.get("q_temp")
    out = np.empty((T, H, dv))
    for i in range(T):
        f = temperature(i, t["coef"], t["every"], faults) if t else 1.0
        for n in range(H):
            g = n % G if "interleaved_heads" in faults else n // (H // G)
            dist = i - np.arange(i + 1) + ("far_by_one" in faults)
            s = k[:i + 1, g] @ q[i, n] * (f * m["scale"])
            if "no_distance" not in faults:
                s = s - P("r1")[n] * np.log(1.0 + P("r2")[n] * dist)
            w = np.exp(s - s.max())
            out[i, n] = w / w.sum() @ v[:i + 1, g]
    out = out.reshape(T, H * dv)
    if "no_gate" not in faults:
        out = out * sigmoid(h @ P("g").T)
    return out @ P("o").T


def gated_lru(h, P, m, faults=()):
    """Griffin's recurrent block: a gated diagonal recurrence behind a short convolution, times a gelu branch."""
    T, w = h.shape[0], m["width"]
    y = gelu(h @ P("y").T + P("y.b"))
    u = short_conv(h @ P("x").T + P("x.b"), P("conv"), 0.0 if "no_conv_bias" in faults else P("conv.b"), faults)
    S, out, n = np.zeros(w), np.empty((T, w)), w // m["blocks"]
    for t in range(T):
        r, i = np.empty(w), np.empty(w)
        for b in range(m["blocks"]):
            part = slice(b * n, (b + 1) * n)
            A, I = P("ra")[b], P("ri")[b]
            if "gates_transposed" in faults:
                A, I = A.T, I.T
            r[part] = sigmoid(A @ u[t, part] + P("ra.b")[b])
            i[part] = sigmoid(I @ u[t, part] + P("ri.b")[b])
        log_a = -8.0 * r * softplus(P("lam"))
        a = np.exp(log_a)
        keep = 1.0 if "first_token_special" in faults and t == 0 else np.sqrt(1.0 - a * a)
        if "lost_state" in faults and t == T // 2:
            S = np.zeros(w)
        S = a * S + keep * i * u[t]
        out[t] = S * y[t]
    return out @ P("o").T


def parallel(h, P, m, eps, faults=()):
    left = rms(biased_attention(h, lambda n: P("left." + n), m["left"], faults), eps) * P("left.out")
    right = rms(gated_lru(h, lambda n: P("right." + n), m["right"], faults), eps) * P("right.out")
    return (1.0 if "whole_sum" in faults else 0.5) * (left + right)


def channel_delta(h, P, m, eps, faults=()):
    """The delta rule with a decay per head and key channel, one token at a time."""
    T = h.shape[0]
    H, K, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(n):
        x = short_conv(h @ P(n).T, P(n + ".conv"), 0.0, faults)
        return x if "no_silu" in faults else silu(x)

    q, k, v = branch("q").reshape(T, K, d), branch("k").reshape(T, K, d), branch("v").reshape(T, H, dv)
    if "no_unit" not in faults:
        q, k = (x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6) for x in (q, k))
    q = q * d ** -0.5
    beta = sigmoid(h @ P("b").T)
    z = h @ P("a1").T @ P("a2").T + P("dt_bias")
    g = np.exp(-np.exp(P("A_log"))[None, :, None] * softplus(z).reshape(T, H, d))
    S, out = np.zeros((H, d, dv)), np.empty((T, H, dv))
    for t in range(T):
        if "lost_state" in faults and t == T // 2:
            S[:] = 0.0
        for n in range(H):
            e = n // (H // K)
            decay = np.full(d, g[t, n].mean()) if "mean_decay" in faults else g[t, n]
            old = S[n].copy()
            S[n] = decay[:, None] * S[n]
            u = beta[t, n] * (v[t, n] - (old if "undecayed_read" in faults else S[n]).T @ k[t, e])
            read = S[n].copy()
            S[n] = S[n] + np.outer(k[t, e], u)
            out[t, n] = (read if "early_read" in faults else S[n]).T @ q[t, e]
    o = rms(out, eps) * P("norm") * sigmoid(h @ P("g1").T @ P("g2").T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ P("o").T


def gla(h, P, m, eps, faults=()):
    """Gated linear attention: a decay per head and key channel, one token at a time."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ P(n).T).reshape(T, H, -1) for n in "qkv")
    q = q * d ** -0.5
    alpha = sigmoid(h @ P("a1").T @ P("a2").T + P("a2.b")) ** (1.0 if "no_tau" in faults else 1.0 / m["tau"])
    alpha = alpha.reshape(T, H, d)
    S, out = np.zeros((H, d, dv)), np.empty((T, H, dv))
    for t in range(T):
        if "lost_state" in faults and t == T // 2:
            S[:] = 0.0
        for n in range(H):
            new = np.outer(k[t, n], v[t, n])
            S[n] = alpha[t, n][:, None] * (S[n] + new) if "decays_first" in faults else alpha[t, n][:, None] * S[n] + new
            out[t, n] = S[n].T @ q[t, n]
    o = (rms(out, eps) * P("norm")).reshape(T, H * dv)
    g = h @ P("g").T
    return (o * (sigmoid(g) if "sigmoid_gate" in faults else silu(g))) @ P("o").T


def dense_mlp(h, P, faults=()):
    z = h @ P("up").T + (0.0 if "no_up_bias" in faults else P("up.b"))
    return gelu(z) @ P("down").T + (0.0 if "no_down_bias" in faults else P("down.b"))


def expert(h, up, down):
    return (np.maximum(h @ up.T, 0.0) ** 2) @ down.T


def scores(h, router):
    z = router @ h
    e = np.exp(z - z.max())
    return e / e.sum()


def route(h, router, top, faults=()):
    """(expert, weight) pairs of one token."""
    s = scores(h, router)
    chosen = np.argsort(-s, kind="stable")[:top]
    w = s[chosen]
    return list(zip(chosen.tolist(), w / w.sum() if "renormalised" in faults else w))


def choice_gap(h, router, top):
    """How far the logit of the last chosen expert is ahead of the next one's."""
    c = np.sort(router @ h)[::-1]
    return c[top - 1] - c[top] if top < len(c) else np.inf


def experts_mlp(h, P, m, faults=(), gaps=None):
    top = m["router"]["top"]
    if gaps is not None:
        gaps.append(np.array([choice_gap(t, P("router"), top) for t in h]))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in route(h[t], P("router"), top, faults):
            out[t] += w * expert(h[t], P(f"e{e}.up"), P(f"e{e}.down"))
    return out


def token_input(x, e, P, eps):
    """What a layer adds for the token itself: e is the layer's part of the token's side embedding."""
    return rms((gelu(x @ P("gate").T) * e) @ P("proj").T, eps) * P("norm")


def forward(cfg, W, tokens, hooks=None, faults=(), gaps=None):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps, tokens = cfg["norm"]["eps"], np.asarray(tokens)
    side = cfg.get("token_side")
    x = W["embed"][tokens] * cfg["embedding"]["scale"]
    results = [x]
    for i, L in enumerate(cfg["layers"]):
        P = lambda n, l=f"l{i}.": W[l + n]
        h = rms(x, eps) * P("norm1")
        mixer = {"parallel": parallel, "channel_delta": channel_delta, "gla": gla}[L["type"]]
        mixed = mixer(h, lambda n: P("mix." + n), L["mixer"], eps, faults)
        fed = 0.0
        if L["mlp"]:
            hf = rms(x + mixed, eps) * P("norm1") if "sequential" in faults else h
            mlp = lambda n: P("mlp." + n)
            fed = dense_mlp(hf, mlp, faults) if L["mlp"]["kind"] == "dense" else experts_mlp(hf, mlp, L["mlp"], faults, gaps)
        before = x
        x = x + (mixed + fed)
        if side and "no_side" not in faults:
            n = side["dim"]
            at = 0 if "first_part" in faults else i
            e = W["side.embed"][tokens][:, at * n:(at + 1) * n]
            x = x + token_input(before if "side_of_input" in faults else x, e, lambda n: P("side." + n), eps)
        results.append(x)
        if "no_average" not in faults:
            if "averages_averages" in faults:
                results[-1] = x = sum(w * r for w, r in zip(P("dwa"), results))
            else:
                x = sum(w * r for w, r in zip(P("dwa"), results))
        if hooks:
            hooks(i, x)
    return rms(x, eps) * W["final.norm"] @ W["head"].T
