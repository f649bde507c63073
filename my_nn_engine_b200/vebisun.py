"""The Vebisun decoder: how its config.json and tensor names map to a block decoder (block_decoder.py).

Every layer is sandwich-normed (a layer norm before and after each sublayer, residual multiplied by a constant): attention with
short causal convolutions on q, k and v, interleaved rotation of part of each head, capped scores and a sliding window, then a
mixture of SiLU-gated experts chosen from the best expert groups.  A range of layers may be run several times in a row; the
embedding output is added again before each repetition."""
from __future__ import annotations

from typing import Dict

import torch

from .block_decoder import BlockDecoder, BlockLayer, BlockModelSpec, Rotary, RotaryScaling
from .checkpoint import CheckpointError

ARCHITECTURE = "Vebisun"


def _layer(i: int, entry: dict) -> BlockLayer:
    if entry.get("type") != "attention":
        raise ValueError(f"layer {i}: unknown mixer type {entry.get('type')!r}")
    m = entry["mixer"]
    rot = m.get("rot")
    rotary = None
    if rot:
        sc = rot.get("scaling")
        rotary = Rotary(float(rot["base"]), int(rot["dims"]),
                        RotaryScaling(float(sc["factor"]), float(sc["low"]), float(sc["high"]), float(sc["original"])) if sc else None)
    mask = m.get("mask") or {}
    layer = BlockLayer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                       softcap=float(m.get("softcap") or 0.0), window=int(mask.get("size") or 0), conv_taps=int(m.get("conv") or 0), rotary=rotary)
    mlp = entry.get("mlp")
    if mlp:
        if mlp.get("kind") != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        r = mlp["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        layer.experts, layer.top, layer.expert_ff = int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"])
        layer.groups, layer.groups_keep = int(groups["count"]), int(groups["keep"])
    return layer


def spec_from_config(cfg: dict) -> BlockModelSpec:
    loop = cfg.get("loop")
    return BlockModelSpec(hidden=cfg["width"], vocab=cfg["vocab"], layers=[_layer(i, e) for i, e in enumerate(cfg["layers"])],
                          norm_eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]),
                          residual_mult=float(cfg["residual_mult"]),
                          loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop and int(loop["times"]) > 1 else None)


def weights_from_state(spec: BlockModelSpec, state: Dict[str, torch.Tensor]) -> dict:
    """The checkpoint's tensors in the layout BlockDecoder takes; every shape is checked against the configuration."""

    def get(name, *shape):
        t = state.get(name)
        if t is None:
            raise CheckpointError(f"tensor {name} is missing")
        if tuple(t.shape) != shape:
            raise CheckpointError(f"tensor {name} has shape {tuple(t.shape)}, the configuration says {shape}")
        return t

    def norm(name):
        return get(name, spec.hidden), get(name + ".b", spec.hidden)

    H, out = spec.hidden, []
    for i, L in enumerate(spec.layers):
        p = f"l{i}."
        rows = {"q": L.heads * L.dim, "k": L.kv_heads * L.dim, "v": L.kv_heads * L.vdim}
        w = {"norm1": norm(p + "norm1"), "norm1b": norm(p + "norm1b"),
             "qkv": torch.cat([get(p + "mix." + n, r, H) for n, r in rows.items()], 0),
             "conv": torch.cat([get(p + f"mix.{n}.conv", r, L.conv_taps) for n, r in rows.items()], 0) if L.conv_taps else None,
             "o": get(p + "mix.o", H, L.heads * L.vdim)}
        if L.experts:
            e = [f"{p}mlp.e{j}." for j in range(L.experts)]
            w.update(norm2=norm(p + "norm2"), norm2b=norm(p + "norm2b"), router=get(p + "mlp.router", L.experts, H),
                     gate_up=torch.stack([torch.cat([get(n + "gate", L.expert_ff, H), get(n + "up", L.expert_ff, H)], 0) for n in e], 0),
                     down=torch.stack([get(n + "down", H, L.expert_ff) for n in e], 0))
        out.append(w)
    return {"embed": get("embed", spec.vocab, H), "layers": out, "final_norm": norm("final.norm"), "head": get("head", spec.vocab, H)}


def build(cfg: dict, state: Dict[str, torch.Tensor], **kwargs) -> BlockDecoder:
    spec = spec_from_config(cfg)
    return BlockDecoder(spec, weights_from_state(spec, state), **kwargs)
