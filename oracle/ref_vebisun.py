"""Plain CPU restatement of the Vebisun decoder: one function per mechanism, float64 (or any numpy dtype), whole sequence
at once, no cache, no kernels.  Test infrastructure only; it shares nothing with the product path.

Notation: T tokens, W model width, per head key size D and value size E, heads H, kv heads G.
"""
from __future__ import annotations

import math

import numpy as np


def layer_norm(x, w, b, eps):
    mu = x.mean(-1, keepdims=True)
    dev = x - mu
    return dev / np.sqrt((dev * dev).mean(-1, keepdims=True) + eps) * w + b


def short_conv(u, w):
    """u [T, C], w [C, n]: y[t, c] = sum_j w[c, j] u[t - (n - 1) + j, c], zero before the first token."""
    T, n = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for j in range(n):
        lag = n - 1 - j
        if lag < T:
            y[lag:] += w[:, j] * u[:T - lag]
    return y


def rotary_frequencies(base, dims, scaling=None):
    """f_i = base^(-2i / dims), i < dims / 2; with ``scaling`` {factor, low, high, original} frequencies whose wavelength is
    long against the original context are divided by the factor, with a linear blend in between."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            wl = 2.0 * math.pi / f
            fac, lo, hi, orig = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            if wl > orig / lo:
                f = f / fac
            elif not wl < orig / hi:
                s = (orig / wl - lo) / (hi - lo)
                f = (1.0 - s) * f / fac + s * f
        out.append(f)
    return np.array(out, dtype=np.float64)


def rotate_interleaved(x, positions, freqs):
    """x [T, heads, D]: dimensions (2i, 2i + 1) turn by position * freqs[i]; dimensions past 2 len(freqs) stay."""
    y = x.copy()
    for t, p in enumerate(positions):
        for i, f in enumerate(freqs):
            c, s = math.cos(float(p) * f), math.sin(float(p) * f)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            y[t, :, 2 * i], y[t, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def windowed_attention(q, k, v, scale, softcap=None, window=None):
    """q [T, H, D], k [T, G, D], v [T, G, E]; query i sees keys j with 0 <= i - j < window."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            j0 = 0 if window is None else max(0, i - window + 1)
            s = (k[j0:i + 1, g] @ q[i, h]) * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[j0:i + 1, g]
    return out


def route(z, top, groups=1, keep=1):
    """Router logits z [E] -> (expert indices by falling score, their softmax scores)."""
    e = np.exp(z - z.max())
    s = e / e.sum()
    per = len(s) // groups
    best = np.argsort([-s[g * per:(g + 1) * per].max() for g in range(groups)], kind="stable")[:keep]
    allowed = [g * per + i for g in best for i in range(per)]
    chosen = sorted(allowed, key=lambda i: (-s[i], i))[:top]
    return chosen, s[chosen]


def silu(z):
    return z / (1.0 + np.exp(-z))


def moe(h, router, gates, ups, downs, top, groups=1, keep=1):
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(*route(router @ h[t], top, groups, keep)):
            out[t] += s * (downs[e] @ (silu(gates[e] @ h[t]) * (ups[e] @ h[t])))
    return out


def mixer(W, p, h, m, positions):
    """The attention mixer of one layer; W maps tensor names to arrays, p is the layer's prefix, m its config."""
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    qkv = []
    for n in "qkv":
        u = h @ W[f"{p}.mix.{n}"].T
        if m.get("conv"):
            u = short_conv(u, W[f"{p}.mix.{n}.conv"])
        qkv.append(u)
    T = h.shape[0]
    q, k, v = qkv[0].reshape(T, H, D), qkv[1].reshape(T, G, D), qkv[2].reshape(T, G, E)
    if m.get("rot"):
        f = rotary_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
        q, k = rotate_interleaved(q, positions, f), rotate_interleaved(k, positions, f)
    a = windowed_attention(q, k, v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    return a.reshape(T, H * E) @ W[f"{p}.mix.o"].T


def layer_runs(cfg):
    """(layer index, embedding output added first?) in execution order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, False) for i in range(a)]
    for t in range(times):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg, W, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence; ``trace`` (a list) receives the residual stream after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]

    def norm(name, x):
        return layer_norm(x, W[name], W[name + ".b"], eps)

    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    x0 = x.copy()
    pos = np.arange(len(tokens))
    for i, again in layer_runs(cfg):
        if again:
            x = x + x0
        L, p = cfg["layers"][i], f"l{i}"
        x = x + m * norm(p + ".norm1b", mixer(W, p, norm(p + ".norm1", x), L["mixer"], pos))
        if L.get("mlp"):
            r = L["mlp"]["router"]
            E = r["experts"]
            grp = r.get("groups") or {"count": 1, "keep": 1}
            y = moe(norm(p + ".norm2", x), W[p + ".mlp.router"], *[[W[f"{p}.mlp.e{e}.{n}"] for e in range(E)] for n in ("gate", "up", "down")],
                    r["top"], grp["count"], grp["keep"])
            x = x + m * norm(p + ".norm2b", y)
        if trace is not None:
            trace.append(x.copy())
    return norm("final.norm", x) @ W["head"].T
