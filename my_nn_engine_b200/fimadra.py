"""The Fimadra decoder: how its config.json and tensor names map to a block decoder (block_decoder.py).

Pre-normed layers (norms by root mean square) of three kinds in any order: grouped-query attention inside fixed chunks of positions,
with q and k rotated by halves and normed per head; attention through latents, without positions; and matrix memory with exponential
gates (mLSTM).  A layer may have a dense feed-forward with a squared ReLU.  The logits are scaled."""
from __future__ import annotations

from typing import Dict

import torch

from .block_decoder import BlockDecoder, BlockLayer, BlockModelSpec, Rotary
from .checkpoint import CheckpointError

ARCHITECTURE = "Fimadra"


def _layer(i: int, entry: dict) -> BlockLayer:
    kind, m = entry.get("type"), entry["mixer"]
    if kind == "attention":
        rot = m.get("rot")
        layer = BlockLayer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                           chunk=int((m.get("mask") or {}).get("size") or 0), rotary=Rotary(float(rot["base"]), int(rot["dims"])) if rot else None,
                           rot_halves=True, qk_norm=True)
    elif kind == "latent_attention":
        layer = BlockLayer(mixer=kind, heads=m["heads"], kv_heads=m["heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                           q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]))
    elif kind == "mlstm":
        layer = BlockLayer(mixer=kind, heads=m["heads"], kv_heads=m["heads"], dim=m["dim"], vdim=m["vdim"], scale=1.0, gate_cap=float(m["gate_cap"]))
    else:
        raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
    mlp = entry.get("mlp")
    if mlp:
        if mlp.get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        layer.dense_ff, layer.ff_act = int(mlp["ff"]), "square_relu"
    return layer


def spec_from_config(cfg: dict) -> BlockModelSpec:
    return BlockModelSpec(hidden=cfg["width"], vocab=cfg["vocab"], layers=[_layer(i, e) for i, e in enumerate(cfg["layers"])],
                          norm_eps=float(cfg["norm"]["eps"]), rms_norm=True, post_norm=False, logit_scale=float(cfg["logit_scale"]))


def weights_from_state(spec: BlockModelSpec, state: Dict[str, torch.Tensor]) -> dict:
    """The checkpoint's tensors in the layout BlockDecoder takes; every shape is checked against the configuration."""

    def get(name, *shape):
        t = state.get(name)
        if t is None:
            raise CheckpointError(f"tensor {name} is missing")
        if tuple(t.shape) != shape:
            raise CheckpointError(f"tensor {name} has shape {tuple(t.shape)}, the configuration says {shape}")
        return t

    W, out = spec.hidden, []
    for i, L in enumerate(spec.layers):
        p, H = f"l{i}.mix.", L.heads
        w = {"norm1": (get(f"l{i}.norm1", W), None), "o": get(p + "o", W, H * L.vdim), "conv": None}
        if L.mixer == "latent_attention":
            rows = {"dq": L.q_rank, "dkv": L.kv_rank}
            w.update(q_norm=get(p + "dq.norm", L.q_rank), kv_norm=get(p + "dkv.norm", L.kv_rank), uq=get(p + "uq", H * L.dim, L.q_rank),
                     uk=get(p + "uk", H * L.dim, L.kv_rank), uv=get(p + "uv", H * L.vdim, L.kv_rank))
        elif L.mixer == "mlstm":
            rows = {"q": H * L.dim, "k": H * L.dim, "v": H * L.vdim, "g": H * L.vdim, "i": H, "f": H}
            w.update(head_norm=get(p + "norm", H * L.vdim), gate_bias=torch.cat([get(p + "i.b", H), get(p + "f.b", H)], 0))
        else:
            rows = {"q": H * L.dim, "k": L.kv_heads * L.dim, "v": L.kv_heads * L.vdim}
        w["qkv"] = torch.cat([get(p + n, r, W) for n, r in rows.items()], 0)
        if L.dense_ff:
            w.update(norm2=(get(f"l{i}.norm2", W), None), up=get(f"l{i}.mlp.up", L.dense_ff, W), down=get(f"l{i}.mlp.down", W, L.dense_ff))
        out.append(w)
    return {"embed": get("embed", spec.vocab, W), "layers": out, "final_norm": (get("final.norm", W), None), "head": get("head", spec.vocab, W)}


def build(cfg: dict, state: Dict[str, torch.Tensor], **kwargs) -> BlockDecoder:
    spec = spec_from_config(cfg)
    return BlockDecoder(spec, weights_from_state(spec, state), **kwargs)
