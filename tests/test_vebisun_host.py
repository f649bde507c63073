"""Vebisun on the host: the oracle's own consistency, configuration and weight mapping, the family registry, the session's feed
and the trace runner's protocol (CPU only)."""
import io
import json
import math

import numpy as np
import pytest
import torch

from my_nn_engine_b200 import ffi, registry, vebisun
from my_nn_engine_b200.block_decoder import Rotary, RotaryScaling
from my_nn_engine_b200.checkpoint import CheckpointError
from my_nn_engine_b200.session import LlmSession, PromptTooLong
from my_nn_engine_b200.trace import replay
from oracle import ref_vebisun as R
from tests import block_models as bm


# ---- the oracle, one mechanism at a time, against hand-computed or structural facts ----
def test_oracle_conv_and_norm():
    u = np.array([[1.0], [2.0], [3.0]])
    assert R.short_conv(u, np.array([[10.0, 1.0]]))[:, 0].tolist() == [1.0, 12.0, 23.0]
    assert R.short_conv(u[:1], np.array([[7.0, 5.0, 2.0]]))[0, 0] == 2.0
    y = R.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 2.0]), np.array([0.5, 0.0]), 0.0)
    assert np.allclose(y, [[-1.5, 2.0]])


def test_oracle_rotation_keeps_relative_angles_and_the_rest():
    rng = np.random.default_rng(0)
    f = R.rotary_frequencies(100.0, 6)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    d = [(R.rotate_interleaved(q, [p + 5], f) * R.rotate_interleaved(k, [p], f)).sum() for p in (0, 3, 1000)]
    assert np.allclose(d, d[0])
    assert np.array_equal(R.rotate_interleaved(q, [9], f)[..., 6:], q[..., 6:])
    one = R.rotate_interleaved(np.array([[[1.0, 0.0]]]), [1], [math.pi / 2])
    assert np.allclose(one, [[[0.0, 1.0]]])


def test_oracle_attention_window_and_cap():
    T, W = 12, 4
    q = np.ones((T, 1, 2))
    k = np.zeros((T, 1, 2))
    k[3] = 50.0  # stands out wherever it is seen
    v = np.arange(T, dtype=float).reshape(T, 1, 1)
    out = R.windowed_attention(q, k, v, 1.0, None, W)[:, 0, 0]
    assert np.allclose(out[3:3 + W], 3.0) and not np.isclose(out[3 + W], 3.0)
    capped = R.windowed_attention(q, k, v, 1.0, 2.0, W)[4, 0, 0]  # scores at most 2: e^2 against 1 each
    assert np.isclose(capped, (1 + 2 + 3 * math.exp(2.0 * math.tanh(50.0)) + 4) / (3 + math.exp(2.0 * math.tanh(50.0))))


def test_oracle_routing():
    z = np.log(np.array([0.1, 0.3, 0.05, 0.15, 0.25, 0.15]))
    assert R.route(z, 2)[0] == [1, 4]
    idx, w = R.route(z, 2, groups=3, keep=1)  # the group of 0.1 and 0.3
    assert idx == [1, 0] and np.allclose(w, [0.3, 0.1])
    assert R.route(z, 3, groups=3, keep=2)[0] == [1, 4, 5]


def test_oracle_loop_order():
    cfg = bm.config(8, 8, [None] * 4, loop={"start": 1, "stop": 3, "times": 3})
    assert R.layer_runs(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert [i for i, _ in R.layer_runs(cfg)] == [0, 1, 2, 1, 2, 1, 2, 3]


def test_oracle_is_causal():
    cfg = bm.mixed()
    W = bm.as_numpy(bm.weights(cfg))
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 30)
    full, part = R.forward(cfg, W, toks), R.forward(cfg, W, toks[:17])
    assert np.abs(full[:17] - part).max() < 1e-9


# ---- product host code ----
@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 2000.0), (32.0, 2.0, 3.0, 100.0)])
def test_rotary_frequencies_match_the_oracle(scaling):
    for base, dims in ((1e4, 64), (5e5, 16), (100.0, 2)):
        ours = Rotary(base, dims, RotaryScaling(*scaling) if scaling else None).frequencies()
        ref = R.rotary_frequencies(base, dims, dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None)
        assert np.allclose(ours, ref, rtol=1e-12)


def test_configuration_is_read_in_full():
    spec = vebisun.spec_from_config(bm.mixed())
    a = spec.layers[0]
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.conv_taps, a.softcap) == (6, 2, 24, 40, 19, 3, 15.0)
    assert (a.experts, a.expert_ff, a.top, a.groups, a.groups_keep) == (6, 24, 2, 3, 1)
    assert a.rotary.scaling.factor == 8.0 and a.channels == 6 * 24 + 2 * 64
    assert spec.layers[2].experts == 0 and spec.loop == (1, 3, 2) and spec.runs() == [0, 1, 2, 1, 2, 3]
    assert (spec.embed_scale, spec.residual_mult, spec.norm_eps) == (2.0, 0.7, 1e-5)
    bad = bm.mixed()
    bad["layers"][1]["type"] = "recurrent"
    with pytest.raises(ValueError, match="recurrent"):
        vebisun.spec_from_config(bad)


def test_weights_are_mapped_and_checked():
    cfg = bm.mixed()
    state, spec = bm.weights(cfg), vebisun.spec_from_config(cfg)
    w = vebisun.weights_from_state(spec, state)
    L = w["layers"][0]
    assert torch.equal(L["qkv"][6 * 24:6 * 24 + 2 * 24], state["l0.mix.k"]) and torch.equal(L["conv"][-2 * 40:], state["l0.mix.v.conv"])
    assert torch.equal(L["gate_up"][4, :24], state["l0.mlp.e4.gate"]) and torch.equal(L["gate_up"][4, 24:], state["l0.mlp.e4.up"])
    assert torch.equal(L["down"][5], state["l0.mlp.e5.down"]) and "router" not in w["layers"][2]
    broken = dict(state)
    broken["l1.mix.q.conv"] = broken["l1.mix.q.conv"][:, :1]
    with pytest.raises(CheckpointError, match="l1.mix.q.conv"):
        vebisun.weights_from_state(spec, broken)
    del broken["l1.mix.q.conv"]
    with pytest.raises(CheckpointError, match="missing"):
        vebisun.weights_from_state(spec, broken)


def test_registry_chooses_by_configuration(tmp_path):
    assert registry.family_of(bm.mixed()).name == "vebisun"
    assert registry.family_of({"model_type": "llama"}).name == "llama"
    assert registry.family_of({"architectures": ["LlamaForCausalLM"]}).name == "llama"
    with pytest.raises(ValueError, match="Other"):
        registry.family_of({"architecture": "Other"})
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Other"}))
    with pytest.raises(ValueError, match="Other"):
        registry.load_model(str(tmp_path))


def _configure(**change):
    layer = dict(heads=4, kv_heads=2, dim=16, vdim=16, conv_taps=3, rot_dims=8, window=20, cache_rows=128, history_rows=11, experts=8, expert_ff=16,
                 top=2, groups=4, groups_keep=2, attn_scale=0.25, softcap=10.0)
    model = dict(n_layers=1, hidden=32, vocab=50, max_seq_len=500, batch=1, dtype=ffi.BF16, output_mode=0, use_graph=1, max_prefill=64, max_rewind=8,
                 loop_start=0, loop_stop=1, loop_times=2, embed_scale=1.0, residual_mult=1.0, norm_eps=1e-5)
    for k, v in change.items():
        (layer if k in layer else model)[k] = v
    arr = (ffi.Block * 1)(ffi.Block(**layer))
    return ffi.lib().mynn_b200_model_configure_blocks(ffi.BlockModelConfig(layers=arr, **model))


def test_block_configuration_is_validated():
    assert _configure() == ffi.OK
    for bad in (dict(heads=3), dict(rot_dims=7), dict(rot_dims=18), dict(cache_rows=64), dict(cache_rows=130), dict(window=90), dict(window=0),
                dict(history_rows=10), dict(groups=3), dict(groups_keep=5), dict(top=5), dict(loop_stop=2), dict(dtype=9), dict(vocab=0)):
        assert _configure(**bad) == ffi.E_ARG, bad
    assert _configure(experts=0) == ffi.OK
    assert ffi.lib().mynn_b200_model_configure_blocks(None) == ffi.E_ARG


class FakeModel:
    """Logits that name the position and the token: enough to follow the session and the runner."""
    batch, output, max_seq_len, vocab, streaming, max_prefill = 1, "logits", 40, 3, None, 4

    def feed(self, tokens, past_len, want):
        return torch.tensor([[past_len + w, tokens[w], 0.0] for w in want], dtype=torch.float32).reshape(len(want), 3)

    def step(self, tokens, past_len):
        return torch.zeros(1, 3)

    def prefill(self, tokens, past_len):
        return torch.zeros(1, 3)


def test_session_feed_advances_and_is_bounded():
    s = LlmSession.for_model(FakeModel(), -1, prefill_len=4)
    assert s.feed([5, 6, 7], [2, 0]).tolist() == [[2, 7, 0], [0, 5, 0]]
    assert s.past_len() == 3 and s.feed([9], [0]).tolist() == [[3, 9, 0]]
    with pytest.raises(PromptTooLong):
        s.feed([0] * 37)
    s.reset()
    assert s.feed([1] * 40).shape == (0, 3)


def test_runner_protocol(tmp_path):
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [4, 5, 6], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [7, 8], "want": [1, 0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": ["b"]}]
    said = []
    replay(LlmSession.for_model(FakeModel(), -1), 3, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "0.f32").exists()
    assert np.fromfile(tmp_path / "1.f32", "<f4").reshape(-1, 3).tolist() == [[4, 8, 0], [3, 7, 0]]
    assert np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [0, 9, 0]
    with pytest.raises(ValueError, match="before"):
        replay(LlmSession.for_model(FakeModel(), -1), 3,
               [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": [1]}], "end": []}),
                json.dumps({"step": 1, "entries": [{"id": "b", "tokens": [1]}], "end": []})], str(tmp_path), said.append)
