"""Small random Vebisun models for the tests: configurations, weights, and what the oracle needs of them."""
import numpy as np
import torch


def layer(heads, kv_heads, dim, vdim, window, conv, rot, softcap=15.0, scale=None, moe=None):
    e = {"type": "attention",
         "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rot": rot, "softcap": softcap,
                   "scale": scale if scale is not None else dim ** -0.5, "mask": {"size": window}},
         "mlp": None}
    if moe:
        ff, experts, top, count, keep = moe
        e["mlp"] = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}
    return e


def rot(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def config(width, vocab, layers, loop=None, embed=2.0, mult=0.7, eps=1e-5):
    return {"architecture": "Vebisun", "width": width, "vocab": vocab, "layers": layers, "loop": loop, "embedding": {"scale": embed},
            "residual_mult": mult, "norm": {"eps": eps}}


def mixed():
    """Layers of different sizes, none of which the tuned attention kernels take; one without a feed-forward, a loop of two."""
    return config(72, 101, [
        layer(6, 2, 24, 40, 19, 3, rot(8, 500.0, (8.0, 1.0, 4.0, 64.0)), moe=(24, 6, 2, 3, 1)),
        layer(4, 4, 12, 12, 33, 2, rot(12), softcap=4.0, moe=(16, 4, 3, 1, 1)),
        layer(3, 1, 32, 16, 7, 5, rot(6, 100.0)),
        layer(2, 2, 16, 24, 50, 1, rot(16, 1e6), moe=(40, 9, 1, 3, 1)),
    ], loop={"start": 1, "stop": 3, "times": 2})


def even_group():
    """Head size 64, two query heads per kv head."""
    return config(128, 160, [layer(4, 2, 64, 64, 50, 4, rot(32, 1e4, (4.0, 1.0, 4.0, 128.0)), moe=(48, 8, 2, 4, 2)),
                             layer(8, 2, 64, 64, 131, 3, rot(64), moe=(32, 8, 3, 2, 1))],
                  loop={"start": 0, "stop": 1, "times": 3}, embed=1.0, mult=0.8, eps=1e-6)


def odd_group():
    """Head size 128, three query heads per kv head, no loop."""
    return config(96, 90, [layer(3, 1, 128, 128, 140, 2, rot(16), softcap=30.0, moe=(64, 5, 2, 1, 1)),
                           layer(6, 2, 128, 128, 16, 4, rot(128, 1e5), moe=(16, 12, 4, 6, 3))], mult=0.7, embed=1.0)


def all_chosen(cfg, experts=3):
    """The same model with few experts that every token uses: no choice that 16-bit rounding could tip, so that 16-bit logits can be
    held to a tight limit."""
    for e in cfg["layers"]:
        if e["mlp"]:
            e["mlp"]["router"].update(experts=experts, top=experts, groups={"count": 1, "keep": 1})
    return cfg


ALL = {"mixed": mixed, "even_group": even_group, "odd_group": odd_group}


def weights(cfg, seed=0, sharp=3.0):
    """Random bf16 tensors under their checkpoint names.  ``sharp`` scales the query projections so that attention concentrates on
    few keys: a single wrong key then shows in the logits."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, gain=1.0):
        return (torch.randn(*shape, generator=g) * gain * shape[-1] ** -0.5).bfloat16()

    W, out = cfg["width"], {}

    def norm(name):
        out[name] = (1.0 + 0.2 * torch.randn(W, generator=g)).bfloat16()
        out[name + ".b"] = (0.2 * torch.randn(W, generator=g)).bfloat16()

    out["embed"] = torch.randn(cfg["vocab"], W, generator=g).bfloat16()
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if e["mlp"] else ()):
            norm(p + n)
        rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
        for n, r in rows.items():
            out[p + "mix." + n] = mat(r, W, gain=sharp if n == "q" else 1.0)
            taps = torch.randn(r, m["conv"], generator=g) * 0.4
            taps[:, -1] += 1.0
            out[p + f"mix.{n}.conv"] = taps.bfloat16()
        out[p + "mix.o"] = mat(W, m["heads"] * m["vdim"])
        if e["mlp"]:
            ff, E = e["mlp"]["expert"]["ff"], e["mlp"]["router"]["experts"]
            for j in range(E):
                out[p + f"mlp.e{j}.gate"], out[p + f"mlp.e{j}.up"] = mat(ff, W), mat(ff, W)
                out[p + f"mlp.e{j}.down"] = mat(W, ff)
            out[p + "mlp.router"] = mat(E, W, gain=2.0)
    norm("final.norm")
    out["head"] = mat(cfg["vocab"], W)
    return out


def as_numpy(state):
    return {k: v.double().numpy() for k, v in state.items()}


def rel_error(got, want):
    """Root mean square of the difference per row (its mean taken off) over the spread of the reference."""
    d = np.asarray(got, np.float64) - np.asarray(want, np.float64)
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.asarray(want, np.float64).std()
