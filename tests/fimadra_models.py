"""Small random Fimadra models for the tests: configurations and weights."""
import torch


def attention(heads, kv_heads, dim, vdim, chunk, rot, base=1e4, scale=1.0, ff=None):
    """q and k are normed per head, so ``scale`` alone sets how far attention concentrates."""
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base},
                                           "scale": scale, "mask": {"size": chunk}}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, vdim, q_rank, kv_rank, scale=None, ff=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "scale": scale if scale is not None else dim ** -0.5}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mlstm(heads, dim, vdim, cap, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, logit_scale=0.6, eps=1e-5):
    return {"architecture": "Fimadra", "width": width, "vocab": vocab, "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}}


def mixed():
    """Every kind of layer, with and without a feed-forward; sizes that no tensor-core attention takes."""
    return config(72, 101, [latent(3, 20, 28, 36, 24, ff=56), attention(6, 2, 24, 40, 37, 16, 500.0), mlstm(3, 20, 28, 9.0, ff=40),
                            attention(4, 4, 12, 20, 50, 12, scale=0.7, ff=30), latent(2, 16, 8, 12, 40)])


def odd():
    """Sizes that nothing divides evenly, one head here and there, a long memory, a large eps."""
    return config(50, 67, [mlstm(1, 70, 33, 4.0), attention(3, 1, 14, 9, 3, 6, 100.0, ff=27), latent(1, 7, 5, 11, 13, ff=9), mlstm(5, 6, 10, 30.0),
                           attention(2, 2, 10, 6, 1000, 10)], logit_scale=1.0, eps=1e-2)


def chunkwise():
    """The tensor-core kernels with heads of 64: tuned attention, latents expanded for prompts, matrix memory in chunks."""
    return config(128, 160, [mlstm(4, 32, 40, 12.0), attention(4, 2, 64, 64, 100, 32, scale=0.3, ff=96), latent(4, 64, 64, 64, 128, ff=48), mlstm(2, 64, 96, 15.0)],
                  logit_scale=2.0, eps=1e-6)


def wide():
    """Heads of 128, two head groups over the latents, memories of 128 and 256 rows."""
    return config(96, 90, [latent(18, 128, 128, 40, 256), mlstm(2, 128, 64, 7.0, ff=64), attention(3, 1, 128, 128, 130, 64, 1e5, scale=0.2),
                           mlstm(1, 200, 40, 15.0), latent(5, 64, 64, 24, 512, ff=32), attention(6, 2, 64, 64, 16, 64, scale=0.25)])


ALL = {"mixed": mixed, "odd": odd, "chunkwise": chunkwise, "wide": wide}


def weights(cfg, seed=0):
    """Random bf16 tensors under their checkpoint names.  Latent queries are scaled up so that attention concentrates on few keys, and
    forget gates lean to keeping, so that a lost state or a wrong key shows in the logits."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, gain=1.0):
        return (torch.randn(*shape, generator=g) * gain * shape[-1] ** -0.5).bfloat16()

    def vec(n, mean=1.0, spread=0.2):
        return (mean + spread * torch.randn(n, generator=g)).bfloat16()

    W = cfg["width"]
    out = {"embed": torch.randn(cfg["vocab"], W, generator=g).bfloat16(), "head": mat(cfg["vocab"], W), "final.norm": vec(W)}
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}.mix."
        H, D, E = m["heads"], m["dim"], m["vdim"]
        out[f"l{i}.norm1"] = vec(W)
        out[p + "o"] = mat(W, H * E)
        if e["type"] == "latent_attention":
            Q, R = m["q_rank"], m["kv_rank"]
            out.update({p + "dq": mat(Q, W), p + "dq.norm": vec(Q), p + "uq": mat(H * D, Q, gain=3.0), p + "dkv": mat(R, W), p + "dkv.norm": vec(R),
                        p + "uk": mat(H * D, R), p + "uv": mat(H * E, R)})
        else:
            G = m.get("kv_heads", H)
            out.update({p + "q": mat(H * D, W), p + "k": mat(G * D, W), p + "v": mat(G * E, W)})
        if e["type"] == "mlstm":
            out.update({p + "g": mat(H * E, W), p + "norm": vec(H * E), p + "i": mat(H, W, gain=2.0), p + "i.b": vec(H, 0.0, 1.0), p + "f": mat(H, W),
                        p + "f.b": vec(H, 4.0, 1.0)})
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            out.update({f"l{i}.norm2": vec(W), f"l{i}.mlp.up": mat(ff, W), f"l{i}.mlp.down": mat(W, ff)})
    return out
