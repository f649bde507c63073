"""Model families by config.json: which class serves a model directory, and how its weights are read.

``load_model(dir, ...)`` is the one way from a directory to a resident model; the generation command and the trace runner both use
it.  A family registers a predicate over the parsed config.json and a builder ``(model_dir, cfg, **options) -> model``; the model
steps through the common interface of ``DeviceModel`` (decoder.py).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, List

from . import fimadra, vebisun
from .checkpoint import load_model_dir, load_weights_dir
from .decoder import DecoderModel


@dataclass
class Family:
    name: str
    matches: Callable[[dict], bool]
    build: Callable[..., object]  # (model_dir, cfg, **options)
    dtypes: tuple = ("bf16", "f16", "f32")


def _is_llama(cfg: dict) -> bool:
    return cfg.get("model_type") == "llama" or "LlamaForCausalLM" in (cfg.get("architectures") or ())


def _build_llama(model_dir, cfg, **options):
    cfg, state = load_model_dir(model_dir)
    return DecoderModel(cfg, state, **options)


def _is_vebisun(cfg: dict) -> bool:
    return cfg.get("architecture") == vebisun.ARCHITECTURE


def _build_vebisun(model_dir, cfg, **options):
    return vebisun.build(cfg, load_weights_dir(model_dir), **options)


def _is_fimadra(cfg: dict) -> bool:
    return cfg.get("architecture") == fimadra.ARCHITECTURE


def _build_fimadra(model_dir, cfg, **options):
    return fimadra.build(cfg, load_weights_dir(model_dir), **options)


FAMILIES: List[Family] = [Family("llama", _is_llama, _build_llama), Family("vebisun", _is_vebisun, _build_vebisun),
                          Family("fimadra", _is_fimadra, _build_fimadra)]


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def family_of(cfg: dict) -> Family:
    for fam in FAMILIES:
        if fam.matches(cfg):
            return fam
    what = cfg.get("architecture") or cfg.get("model_type") or cfg.get("architectures")
    raise ValueError(f"no model family for config.json of {what!r} (known: {', '.join(f.name for f in FAMILIES)})")


def load_model(model_dir: str, **options):
    """The resident model of a directory: options as for the family's class (dtype, max_seq_len, batch, output, max_prefill, ...)."""
    cfg = read_config(model_dir)
    return family_of(cfg).build(model_dir, cfg, **options)
