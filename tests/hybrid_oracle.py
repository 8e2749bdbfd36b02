"""A plain, slow restatement of the Ralapel equations in numpy float64, one function per mechanism.

tests/test_hybrid.py compares the library with it.  It shares no code with the library: sequences are run
one at a time, recurrences one token at a time, attention one query at a time, and nothing is
fused, chunked, absorbed or cached.  A checkpoint is a dict name -> float array, a configuration
is the parsed config.json.

`hooks` (optional) receives ("layer", run index, residual stream [T, width]) after every layer run.
`faults` lets a test plant a mistake here, on the CPU, to see that its inputs would show it.
"""
from __future__ import annotations

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(x, pos, base):
    """Neighbouring components (2i, 2i + 1) of x [..., d] turn by pos * base^(-2i/d)."""
    d = x.shape[-1]
    out = np.empty_like(x)
    for i in range(d // 2):
        a = pos * base ** (-2.0 * i / d)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def causal_conv(x, w, bias=None):
    """y[t, c] = sum_j w[c, taps - 1 - j] x[t - j, c] (+ bias[c]); nothing before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            if t - j >= 0:
                y[t] += w[:, taps - 1 - j] * x[t - j]
    return y if bias is None else y + bias


def latent_attention(h, P, m, eps, faults=()):
    """h [T, width]; P(name) gives a tensor of the mixer."""
    T = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = (h @ P("q").T).reshape(T, H, d + r)
    down = h @ P("dkv").T
    c = rms(down[:, :R], eps) * P("dkv.norm")
    k_rot = np.stack([rotate_pairs(down[t, R:], t, base) for t in range(T)])
    k = (c @ P("uk").T).reshape(T, H, d)
    v = (c @ P("uv").T).reshape(T, H, dv)
    out = np.empty((T, H, dv))
    for t in range(T):
        q_rot = rotate_pairs(q[t, :, d:], t, base)
        lo = 0
        hi = t if ("skip_self" in faults and t > 0) else t + 1
        if "drop_first" in faults and t > 0:
            lo = 1
        s = (np.einsum("hd,jhd->hj", q[t, :, :d], k[lo:hi]) + q_rot @ k_rot[lo:hi].T) * m["scale"]
        s = np.exp(s - s.max(axis=1, keepdims=True))
        s /= s.sum(axis=1, keepdims=True)
        out[t] = np.einsum("hj,jhd->hd", s, v[lo:hi])
    return out.reshape(T, H * dv) @ P("o").T


def delta(h, P, m, eps, faults=()):
    T = h.shape[0]
    H, K, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def unit(x):
        return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)

    q = silu(causal_conv(h @ P("q").T, P("q.conv"))).reshape(T, K, d)
    k = silu(causal_conv(h @ P("k").T, P("k.conv"))).reshape(T, K, d)
    v = silu(causal_conv(h @ P("v").T, P("v.conv"))).reshape(T, H, dv)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = sigmoid(h @ P("b").T)
    g = np.exp(-np.exp(P("A_log")) * softplus(h @ P("a").T + P("dt_bias")))
    gate = silu(h @ P("g").T).reshape(T, H, dv)
    S = np.zeros((H, d, dv))
    out = np.empty((T, H, dv))
    for t in range(T):
        for n in range(H):
            kk, qq = k[t, n // (H // K)], q[t, n // (H // K)]
            if "read_first" in faults:
                o_early = S[n].T @ qq
            S[n] = g[t, n] * S[n]
            u = beta[t, n] * (v[t, n] - S[n].T @ kk)
            S[n] = S[n] + np.outer(kk, u)
            out[t, n] = o_early if "read_first" in faults else S[n].T @ qq
    return (rms(out, eps) * P("norm") * gate).reshape(T, H * dv) @ P("o").T


def mamba2(h, P, m, eps, faults=()):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = np.split(h @ P("in").T, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = silu(causal_conv(xbc, P("conv"), P("conv.b")))
    x = xbc[:, :inner].reshape(T, H, dv)
    Bm = xbc[:, inner:inner + G * N].reshape(T, G, N)
    Cm = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + P("dt_bias"))
    S = np.zeros((H, N, dv))
    y = np.empty((T, H, dv))
    for t in range(T):
        for n in range(H):
            g = n // (H // G)
            S[n] = np.exp(-np.exp(P("A_log")[n]) * dt[t, n]) * S[n] + dt[t, n] * np.outer(Bm[t, g], x[t, n])
            y[t, n] = S[n].T @ Cm[t, g] + P("D")[n] * x[t, n]
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.reshape(T, m["norm_groups"], inner // m["norm_groups"]), eps).reshape(T, inner) * P("norm")
    return y @ P("o").T


def dense_mlp(h, P):
    return (gelu_tanh(h @ P("gate").T) * (h @ P("up").T)) @ P("down").T


MIXERS = {"latent_attention": latent_attention, "delta": delta, "mamba2": mamba2}


def layer_runs(cfg):
    """[(layer, starts a pass)] in the order they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    a, b, times = lp["start"], lp["stop"], lp["times"]
    runs = [(i, False) for i in range(a)]
    for _ in range(times):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg, W, tokens, hooks=None, faults=()):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = rms(W["embed"][np.asarray(tokens)], eps) * W["embed.norm"]
    x0 = x
    for run, (i, starts_pass) in enumerate(layer_runs(cfg)):
        L = cfg["layers"][i]
        if starts_pass:
            x = np.concatenate([x, x0], axis=1) @ W["loop.in"].T
        mix = MIXERS[L["type"]](rms(x, eps) * W[f"l{i}.norm1"], lambda n: W[f"l{i}.mix.{n}"], L["mixer"], eps, faults)
        x = x + rms(mix, eps) * W[f"l{i}.norm1b"]
        if L["mlp"]:
            ff = dense_mlp(rms(x, eps) * W[f"l{i}.norm2"], lambda n: W[f"l{i}.mlp.{n}"])
            x = x + rms(ff, eps) * W[f"l{i}.norm2b"]
        if hooks:
            hooks("layer", run, x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T
