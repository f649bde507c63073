"""Plain CPU restatement of the Fimadra decoder: one function per mechanism, float64 (or any numpy dtype), whole sequence
at once, no cache, no kernels.  Test infrastructure only; it shares nothing with the product path.

Notation: T tokens, W model width, per head key size D and value size E, heads H, kv heads G, latent size R.
"""
from __future__ import annotations

import math

import numpy as np


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


def attention_mixer(W, p, h, m, eps, positions):
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ W[p + ".mix.q"].T).reshape(T, H, D)
    k = (h @ W[p + ".mix.k"].T).reshape(T, G, D)
    v = (h @ W[p + ".mix.v"].T).reshape(T, G, E)
    if m.get("rot"):
        f = half_frequencies(m["rot"]["base"], m["rot"]["dims"])
        q, k = rotate_halves(q, positions, f), rotate_halves(k, positions, f)
    a = softmax_attention(rms(q, eps), rms(k, eps), v, m["scale"], (m.get("mask") or {}).get("size"))
    return a.reshape(T, H * E) @ W[p + ".mix.o"].T


def latent_mixer(W, p, h, m, eps):
    H, D, E = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    cq = rms(h @ W[p + ".mix.dq"].T, eps) * W[p + ".mix.dq.norm"]
    c = rms(h @ W[p + ".mix.dkv"].T, eps) * W[p + ".mix.dkv.norm"]
    q = (cq @ W[p + ".mix.uq"].T).reshape(T, H, D)
    k = (c @ W[p + ".mix.uk"].T).reshape(T, H, D)
    v = (c @ W[p + ".mix.uv"].T).reshape(T, H, E)
    return softmax_attention(q, k, v, m["scale"]).reshape(T, H * E) @ W[p + ".mix.o"].T


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


def mlstm_mixer(W, p, h, m, eps):
    H, D, E, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    T = h.shape[0]
    q = (h @ W[p + ".mix.q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ W[p + ".mix.k"].T).reshape(T, H, D)
    v = (h @ W[p + ".mix.v"].T).reshape(T, H, E)
    i_log = soft_cap(h @ W[p + ".mix.i"].T + W[p + ".mix.i.b"], cap)
    f_log = log_sigmoid(soft_cap(h @ W[p + ".mix.f"].T + W[p + ".mix.f.b"], cap))
    o = rms(matrix_memory(q, k, v, i_log, f_log), eps).reshape(T, H * E) * W[p + ".mix.norm"]
    return (o / (1.0 + np.exp(-(h @ W[p + ".mix.g"].T)))) @ W[p + ".mix.o"].T


def mixer(W, p, h, entry, eps):
    m, kind = entry["mixer"], entry["type"]
    if kind == "attention":
        return attention_mixer(W, p, h, m, eps, np.arange(h.shape[0]))
    if kind == "latent_attention":
        return latent_mixer(W, p, h, m, eps)
    assert kind == "mlstm", kind
    return mlstm_mixer(W, p, h, m, eps)


def square_relu(z):
    return np.maximum(z, 0.0) ** 2


def forward(cfg, W, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence; ``trace`` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)].copy()
    for l, entry in enumerate(cfg["layers"]):
        p = f"l{l}"
        x = x + mixer(W, p, rms(x, eps) * W[p + ".norm1"], entry, eps)
        if entry.get("mlp"):
            x = x + square_relu((rms(x, eps) * W[p + ".norm2"]) @ W[p + ".mlp.up"].T) @ W[p + ".mlp.down"].T
        if trace is not None:
            trace.append(x.copy())
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T * cfg["logit_scale"]
