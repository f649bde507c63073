"""Plain CPU restatement of the Fimadra decoder: one function per mechanism, float64 (or any numpy dtype), whole sequence
at once, no cache, no kernels.  Test infrastructure only; it shares nothing with the product path.

``store`` stands for the rounding of activations where a 16-bit implementation stores them (projections, normed rows, what attention and
memory give, sublayer outputs); left out, nothing is rounded.  Scores, norms, gates, the memory and the residual sum never are.

Notation: T tokens, W model width, per head key size D and value size E, heads H, kv heads G, latent size R.
"""
from __future__ import annotations

import math

import numpy as np


def exact(x):
    return x


def bf16(x):
    """To the nearest bfloat16 (ties to even), as float64."""
    u = np.asarray(x, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32).astype(np.float64)


def rms(x, eps):
    """Rows of x over their root mean square."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def half_frequencies(base, dims):
    return np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)


def rotate_halves(x, positions, freqs):
    """x [T, heads, D]: dimensions (i, i + n) turn by position * freqs[i], n = len(freqs); dimensions past 2 n stay."""
    n, y = len(freqs), x.copy()
    for t, p in enumerate(positions):
        for i, f in enumerate(freqs):
            c, s = math.cos(float(p) * f), math.sin(float(p) * f)
            u, v = x[t, :, i], x[t, :, i + n]
            y[t, :, i], y[t, :, i + n] = u * c - v * s, v * c + u * s
    return y


def first_visible(i, chunk=None):
    """First key that the query at position i sees: the start of its chunk, or of the sequence."""
    return 0 if not chunk else i - i % chunk


def softmax_attention(q, k, v, scale, chunk=None):
    """q [T, H, D], k [T, G, D], v [T, G, E]; causal, inside chunks of `chunk` positions when that is given."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            j0 = first_visible(i, chunk)
            s = (k[j0:i + 1, g] @ q[i, h]) * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[j0:i + 1, g]
    return out


def attention_mixer(W, p, h, m, eps, positions, store=exact):
    H, D, E = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (store(h @ W[f"{p}.mix.{n}"].T).reshape(T, -1, d) for n, d in (("q", D), ("k", D), ("v", E)))
    if m.get("rot"):
        f = half_frequencies(m["rot"]["base"], m["rot"]["dims"])
        q, k = rotate_halves(q, positions, f), rotate_halves(k, positions, f)
    a = store(softmax_attention(store(rms(q, eps)), store(rms(k, eps)), v, m["scale"], (m.get("mask") or {}).get("size")))
    return a.reshape(T, H * E) @ W[p + ".mix.o"].T


def latent_mixer(W, p, h, m, eps, store=exact):
    H, D, E = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    cq, c = (store(rms(store(h @ W[f"{p}.mix.{n}"].T), eps) * W[f"{p}.mix.{n}.norm"]) for n in ("dq", "dkv"))
    q = store(cq @ W[p + ".mix.uq"].T).reshape(T, H, D)
    k = store(c @ W[p + ".mix.uk"].T).reshape(T, H, D)
    v = store(c @ W[p + ".mix.uv"].T).reshape(T, H, E)
    return store(softmax_attention(q, k, v, m["scale"])).reshape(T, H * E) @ W[p + ".mix.o"].T


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def matrix_memory(q, k, v, i_log, f_log, trace=None):
    """q, k [T, H, D] (q scaled), v [T, H, E], log gates [T, H] -> [T, H, E], token by token.  ``trace`` (a list) receives
    (S, n, m) after every token."""
    T, H, D = q.shape
    out = np.zeros(v.shape, dtype=q.dtype)
    S, n, m = np.zeros((H, D, v.shape[2]), q.dtype), np.zeros((H, D), q.dtype), np.zeros(H, q.dtype)
    for t in range(T):
        for h in range(H):
            top = max(f_log[t, h] + m[h], i_log[t, h])
            keep, take = np.exp(f_log[t, h] + m[h] - top), np.exp(i_log[t, h] - top)
            S[h] = keep * S[h] + take * np.outer(k[t, h], v[t, h])
            n[h] = keep * n[h] + take * k[t, h]
            m[h] = top
            out[t, h] = (S[h].T @ q[t, h]) / (max(abs(n[h] @ q[t, h]), np.exp(-top)) + 1e-6)
        if trace is not None:
            trace.append((S.copy(), n.copy(), m.copy()))
    return out


def mlstm_mixer(W, p, h, m, eps, store=exact):
    H, D, E, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    T = h.shape[0]
    q, k, v, z = (store(h @ W[f"{p}.mix.{n}"].T) for n in "qkvg")
    q, k, v = q.reshape(T, H, D) * D ** -0.5, k.reshape(T, H, D), v.reshape(T, H, E)
    i_log = soft_cap(h @ W[p + ".mix.i"].T + W[p + ".mix.i.b"], cap)
    f_log = log_sigmoid(soft_cap(h @ W[p + ".mix.f"].T + W[p + ".mix.f.b"], cap))
    o = rms(matrix_memory(q, k, v, i_log, f_log), eps).reshape(T, H * E) * W[p + ".mix.norm"]
    return store(o / (1.0 + np.exp(-z))) @ W[p + ".mix.o"].T


def mixer(W, p, h, entry, eps, store=exact):
    m, kind = entry["mixer"], entry["type"]
    if kind == "attention":
        return attention_mixer(W, p, h, m, eps, np.arange(h.shape[0]), store)
    if kind == "latent_attention":
        return latent_mixer(W, p, h, m, eps, store)
    assert kind == "mlstm", kind
    return mlstm_mixer(W, p, h, m, eps, store)


def square_relu(z):
    return np.maximum(z, 0.0) ** 2


def forward(cfg, W, tokens, trace=None, store=exact):
    """Logits [T, vocab] of a whole sequence; ``trace`` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)].copy()
    for l, entry in enumerate(cfg["layers"]):
        p = f"l{l}"
        x = x + store(mixer(W, p, store(rms(x, eps) * W[p + ".norm1"]), entry, eps, store))
        if entry.get("mlp"):
            x = x + store(store(square_relu(store(rms(x, eps) * W[p + ".norm2"]) @ W[p + ".mlp.up"].T)) @ W[p + ".mlp.down"].T)
        if trace is not None:
            trace.append(x.copy())
    return store(rms(x, eps) * W["final.norm"]) @ W["head"].T * cfg["logit_scale"]
