"""Host side of the block decoder: models given as a list of layers with sizes of their own, over unquantised weights.

``BlockModelSpec`` describes such a model without naming one (a model family's module fills it in from its config.json, see
vebisun.py and fimadra.py); ``BlockDecoder`` lays the weights and the state of every layer run out in HBM and drives the same library entry
points as ``DecoderModel``.

State per layer run (a layer repeated by the loop has one per pass).  Attention: a K ring and a V ring
``[batch, kv_heads, cache_rows, dim]`` and, with a short convolution, a ring of unconvolved projections
``[batch, history_rows, channels]``; position p of a sequence always lives in row ``p % rows``.  A layer with a sliding window or
chunks keeps only as many rows as the window, one prefill chunk and the allowed rewind need.  Attention through latents: one row of
``kv_rank`` numbers per position, ``[batch, cache_rows, kv_rank]``.  Matrix memory: f32 ``[batch, heads, dim, vdim]``,
``[batch, heads, dim]`` and ``[batch, heads]``; it belongs to the last position stored and cannot go back.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import List, Optional, Tuple

import numpy as np
import torch

from . import ffi
from .decoder import _FFI_DT, _TORCH_DT, DeviceModel


@dataclass
class RotaryScaling:
    """Frequencies whose wavelength exceeds ``original / low`` are divided by ``factor``; those below ``original / high`` stay;
    in between the two are blended linearly in original / wavelength."""
    factor: float
    low: float
    high: float
    original: float


@dataclass
class Rotary:
    base: float
    dims: int
    scaling: Optional[RotaryScaling] = None

    def frequencies(self) -> np.ndarray:
        i = np.arange(self.dims // 2, dtype=np.float64)
        f = np.power(float(self.base), -2.0 * i / self.dims)
        if self.scaling is None:
            return f
        sc = self.scaling
        turns = sc.original * f / (2.0 * math.pi)  # wavelengths in the original context
        if sc.high == sc.low:
            share = (turns >= sc.high).astype(np.float64)
        else:
            share = np.clip((turns - sc.low) / (sc.high - sc.low), 0.0, 1.0)
        return f * (share + (1.0 - share) / sc.factor)

    def table(self, positions: int) -> Tuple[np.ndarray, np.ndarray]:
        """cos / sin [positions, dims / 2] in f32, from angles in f64."""
        ang = np.arange(positions, dtype=np.float64)[:, None] * self.frequencies()[None, :]
        return np.cos(ang).astype(np.float32), np.sin(ang).astype(np.float32)


@dataclass
class BlockLayer:
    """One layer: its mixer ('attention', 'latent_attention' or 'mlstm'), that mixer's sizes, and its feed-forward (a mixture of
    ``experts``, or dense with ``dense_ff`` > 0, or none)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0           # 0: none
    window: int = 0                # 0: the whole past
    conv_taps: int = 0             # 0: none
    rotary: Optional[Rotary] = None
    experts: int = 0               # 0: no feed-forward
    expert_ff: int = 0
    top: int = 0
    groups: int = 1
    groups_keep: int = 1
    mixer: str = "attention"
    chunk: int = 0                 # positions per chunk of the mask, 0: none
    rot_halves: bool = False       # rotation pairs (i, i + dims / 2) instead of (2i, 2i + 1)
    qk_norm: bool = False          # q and k heads over their root mean square after the rotation
    q_rank: int = 0                # latent_attention
    kv_rank: int = 0
    gate_cap: float = 0.0          # mlstm
    dense_ff: int = 0
    ff_act: str = "none"           # activation of the dense feed-forward: 'none' or 'square_relu'

    @property
    def channels(self) -> int:
        """Rows of the mixer's first product."""
        if self.mixer == "latent_attention":
            return self.q_rank + self.kv_rank
        if self.mixer == "mlstm":
            return self.heads * (2 * (self.dim + self.vdim) + 2)
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)

    @property
    def reach(self) -> int:
        """How many positions up to its own a query sees at most, 0: all of them."""
        return min(self.window, self.chunk) if self.window and self.chunk else max(self.window, self.chunk)

    def state_shapes(self, batch: int, cache_rows: int, history_rows: int):
        """Shape and whether it is f32 whatever the model's dtype (None: absent) of the three state buffers."""
        if self.mixer == "latent_attention":
            return [((batch, cache_rows, self.kv_rank), False), None, None]
        if self.mixer == "mlstm":
            return [((batch, self.heads, self.dim, self.vdim), True), ((batch, self.heads, self.dim), True), ((batch, self.heads), True)]
        return [((batch, self.kv_heads, cache_rows, self.dim), False), ((batch, self.kv_heads, cache_rows, self.vdim), False),
                ((batch, history_rows, self.channels), False) if self.conv_taps else None]


_MIXERS = {"attention": ffi.MIX_ATTENTION, "latent_attention": ffi.MIX_LATENT, "mlstm": ffi.MIX_MLSTM}
_ACTS = {"none": ffi.ACT_NONE, "square_relu": ffi.ACT_SQUARE_RELU}


@dataclass
class BlockModelSpec:
    hidden: int
    vocab: int
    layers: List[BlockLayer]
    norm_eps: float
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None  # start, stop, times
    rms_norm: bool = False       # norms by root mean square, without bias, instead of layer norms
    post_norm: bool = True       # a norm behind each sublayer as well
    logit_scale: float = 1.0

    def runs(self) -> List[int]:
        """Layer indices in execution order."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


def _round_up(x: int, m: int) -> int:
    return -(-x // m) * m


class BlockDecoder(DeviceModel):
    """A block decoder resident on the current CUDA device.

    weights: ``embed`` [V, H], ``head`` [V, H], ``final_norm`` (w, b), ``layers``: per layer a dict with ``norm1``, ``norm1b``,
    ``norm2``, ``norm2b`` as (w, b) pairs (b None with rms_norm; the -b ones only with post_norm, the 2 ones only with a
    feed-forward), ``qkv`` (the rows of the mixer's first product stacked: q, k, v; latents: dq, dkv; mlstm: q, k, v, output, input and
    forget gate), ``o``; attention: ``conv`` [channels, taps] or None; latents: ``q_norm``, ``kv_norm``, ``uq``, ``uk``, ``uv``; mlstm:
    ``head_norm``, ``gate_bias`` (input, forget); experts: ``router``, ``gate_up`` [experts, 2 ff, H] (gate rows first), ``down``
    [experts, H, ff]; dense: ``up``, ``down``.  The logits' scale is folded into the final norm.
    output: 'logits' (f32) or 'ids' (greedy argmax on the device, last maximum).  max_rewind: how many positions a step may go
    back behind what has been stored (a conversation that drops its last tokens)."""

    def __init__(self, spec: BlockModelSpec, weights: dict, dtype: str = "bf16", max_seq_len: int = 256, batch: int = 1,
                 output: str = "logits", use_graph: bool = True, max_prefill: int = 0, max_rewind: int = 32, device=None):
        if not torch.cuda.is_available():
            raise RuntimeError("BlockDecoder needs a CUDA device: the decode path has no CPU implementation")
        self.lib = ffi.lib()
        self.device = dev = torch.device(device if device is not None else f"cuda:{torch.cuda.current_device()}")
        self.spec, self.dtype, self.max_seq_len, self.batch, self.output = spec, dtype, max_seq_len, batch, output
        self.vocab, self.max_prefill, self.streaming = spec.vocab, max_prefill, None
        self.can_rewind = all(L.mixer != "mlstm" for L in spec.layers)
        td = _TORCH_DT[dtype]
        self._keep, init = [], []
        chunk = max(max_prefill, 1)

        def put(t, dt):
            if t is None:
                init.append(None)
                return
            t = t.to(device=dev, dtype=dt).contiguous()
            self._keep.append(t)
            init.append(t.data_ptr())

        tables = {}
        put(weights["embed"], td)
        layers = (ffi.Block * len(spec.layers))()
        for i, (L, w) in enumerate(zip(spec.layers, weights["layers"])):
            ff = L.experts > 0 or L.dense_ff > 0
            latent, mlstm = L.mixer == "latent_attention", L.mixer == "mlstm"

            def put_norm(n, wanted):
                wb = w[n] if wanted else (None, None)
                put(wb[0], torch.float32)
                put(None if spec.rms_norm else wb[1], torch.float32)

            put_norm("norm1", True)
            put_norm("norm1b", spec.post_norm)
            put(w["qkv"], td)
            put(w["conv"].float().t() if L.conv_taps else None, torch.float32)
            put(w["o"], td)
            if L.rotary is not None:
                key = repr(L.rotary)
                if key not in tables:
                    tables[key] = [torch.from_numpy(t).to(dev) for t in L.rotary.table(max_seq_len)]
                    self._keep += tables[key]
                init += [t.data_ptr() for t in tables[key]]
            else:
                init += [None, None]
            put_norm("norm2", ff)
            put_norm("norm2b", ff and spec.post_norm)
            put(w["router"] if L.experts else None, td)
            put(None if not ff else w["up" if L.dense_ff else "gate_up"], td)
            put(w["down"] if ff else None, td)
            put(w["q_norm"] if latent else w["head_norm"] if mlstm else None, torch.float32)
            put(w["kv_norm"] if latent else w["gate_bias"] if mlstm else None, torch.float32)
            put(w["uq"] if latent else None, td)
            put(w["uk"] if latent else None, td)
            put(w["uk"].reshape(L.heads, L.dim, L.kv_rank).transpose(1, 2) if latent else None, td)
            put(w["uv"] if latent else None, td)
            need = max_seq_len if not L.reach else min(max_seq_len, L.reach - 1 + chunk + max_rewind)
            layers[i] = ffi.Block(heads=L.heads, kv_heads=L.kv_heads, dim=L.dim, vdim=L.vdim, conv_taps=L.conv_taps,
                                  rot_dims=L.rotary.dims if L.rotary else 0, window=L.window, cache_rows=_round_up(need, 128),
                                  history_rows=L.conv_taps + max_rewind if L.conv_taps else 0, experts=L.experts, expert_ff=L.expert_ff,
                                  top=L.top, groups=L.groups, groups_keep=L.groups_keep, attn_scale=L.scale, softcap=L.softcap,
                                  mixer=_MIXERS[L.mixer], rot_halves=int(L.rot_halves), qk_norm=int(L.qk_norm), chunk=L.chunk, q_rank=L.q_rank,
                                  kv_rank=L.kv_rank, dense_ff=L.dense_ff, ff_act=_ACTS[L.ff_act], gate_cap=L.gate_cap)
        for t in weights["final_norm"]:  # the head is linear in the normed row
            put(None if t is None else t.float() * spec.logit_scale, torch.float32)
        put(weights["head"], td)

        self.run_states, states = [], []
        for i in spec.runs():
            L, b = spec.layers[i], layers[i]
            bufs = [None if s is None else torch.zeros(s[0], dtype=torch.float32 if s[1] else td, device=dev)
                    for s in L.state_shapes(batch, b.cache_rows, b.history_rows)]
            self.run_states.append(bufs)
            states += [None if t is None else t.data_ptr() for t in bufs]
        loop = spec.loop or (0, 0, 1)
        self._layers_arr = layers
        c = ffi.BlockModelConfig(n_layers=len(spec.layers), hidden=spec.hidden, vocab=spec.vocab, max_seq_len=max_seq_len, batch=batch,
                                 dtype=_FFI_DT[dtype], output_mode=1 if output == "ids" else 0, use_graph=int(use_graph),
                                 max_prefill=max_prefill, max_rewind=max_rewind, loop_start=loop[0], loop_stop=loop[1], loop_times=loop[2],
                                 rms_norm=int(spec.rms_norm), post_norm=int(spec.post_norm),
                                 embed_scale=spec.embed_scale, residual_mult=spec.residual_mult, norm_eps=spec.norm_eps,
                                 layers=ctypes.cast(layers, ctypes.POINTER(ffi.Block)))
        self._open(self.lib.mynn_b200_model_configure_blocks, c, init, states, torch.float32)

    def reset_cache(self):
        for bufs in self.run_states:
            for t in bufs:
                if t is not None:
                    t.zero_()

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._keep)
