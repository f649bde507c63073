"""Fimadra on the host: the oracle against hand-computed or structural facts, configuration and weight mapping, the family registry,
validation of the block configuration, and a session over a model that cannot go back (CPU only)."""
import math

import numpy as np
import pytest
import torch

from my_nn_engine_b200 import ffi, fimadra, registry
from my_nn_engine_b200.block_decoder import Rotary
from my_nn_engine_b200.checkpoint import CheckpointError
from my_nn_engine_b200.session import GenerateOptions, LlmSession
from oracle import ref_fimadra as R
from tests import block_models as bm
from tests import fimadra_models as fm


# ---- the oracle, one mechanism at a time ----
def test_oracle_norm_and_activation():
    assert np.allclose(R.rms(np.array([[3.0, 4.0]]), 0.0), np.array([[3.0, 4.0]]) / math.sqrt(12.5))
    assert np.allclose(R.rms(np.array([[3.0, 4.0]]), 3.5), [[0.75, 1.0]])  # 12.5 + 3.5 = 16
    assert R.square_relu(np.array([-2.0, 3.0])).tolist() == [0.0, 9.0]


def test_oracle_rotation_pairs_halves_and_keeps_relative_angles():
    one = R.rotate_halves(np.array([[[1.0, 5.0, 0.0, 0.0, 7.0]]]), [1], [math.pi / 2, 0.0])
    assert np.allclose(one, [[[0.0, 5.0, 1.0, 0.0, 7.0]]])
    rng = np.random.default_rng(0)
    f = R.half_frequencies(100.0, 6)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    d = [(R.rotate_halves(q, [p + 5], f) * R.rotate_halves(k, [p], f)).sum() for p in (0, 3, 1000)]
    assert np.allclose(d, d[0]) and np.allclose(f, [1.0, 100.0 ** (-1 / 3), 100.0 ** (-2 / 3)])


def test_oracle_chunks():
    assert [R.first_visible(i, 4) for i in (0, 3, 4, 7, 8)] == [0, 0, 4, 4, 8] and R.first_visible(9) == 0
    T = 12
    q, k = np.ones((T, 1, 2)), np.zeros((T, 1, 2))
    k[3] = 50.0
    v = np.arange(T, dtype=float).reshape(T, 1, 1)
    out = R.softmax_attention(q, k, v, 1.0, 5)[:, 0, 0]
    assert np.allclose(out[3:5], 3.0) and np.allclose(out[5:10], [5.0, 5.5, 6.0, 6.5, 7.0]) and np.allclose(out[10:], [10.0, 10.5])


def test_oracle_memory_by_hand_and_against_the_unstabilised_sums():
    one = np.ones((1, 1, 1))
    out = R.matrix_memory(2 * one, 3 * one, 5 * one, np.array([[-1.0]]), np.array([[-0.5]]))  # m = max(-0.5, -1) = -0.5
    w = math.exp(-0.5)
    assert np.isclose(out[0, 0, 0], 30 * w / (max(6 * w, math.exp(0.5)) + 1e-6))
    rng = np.random.default_rng(1)
    T, D, E = 9, 3, 2
    q, k, v = rng.standard_normal((T, 1, D)), rng.standard_normal((T, 1, D)), rng.standard_normal((T, 1, E))
    i, f = rng.standard_normal((T, 1)) * 3, R.log_sigmoid(rng.standard_normal((T, 1)))
    out = R.matrix_memory(q, k, v, i, f)
    S, n = np.zeros((D, E)), np.zeros(D)
    for t in range(T):  # no maximum taken out: |n.q| against 1, the floor scaled by e^-m
        S, n = math.exp(f[t, 0]) * S + math.exp(i[t, 0]) * np.outer(k[t, 0], v[t, 0]), math.exp(f[t, 0]) * n + math.exp(i[t, 0]) * k[t, 0]
        assert np.allclose(out[t, 0], S.T @ q[t, 0] / max(abs(n @ q[t, 0]), 1.0), rtol=1e-3)


def test_oracle_latents_equal_their_absorbed_form():
    cfg = fm.mixed()
    W = bm.as_numpy(fm.weights(cfg))
    m, eps, h = cfg["layers"][0]["mixer"], 1e-5, np.random.default_rng(2).standard_normal((8, 72))
    H, D, E = m["heads"], m["dim"], m["vdim"]
    c = R.rms(h @ W["l0.mix.dkv"].T, eps) * W["l0.mix.dkv.norm"]
    q = ((R.rms(h @ W["l0.mix.dq"].T, eps) * W["l0.mix.dq.norm"]) @ W["l0.mix.uq"].T).reshape(8, H, D)
    q = np.einsum("thd,hdr->thr", q, W["l0.mix.uk"].reshape(H, D, -1))
    lat = R.softmax_attention(q, c[:, None], c[:, None], m["scale"])
    o = np.einsum("thr,her->the", lat, W["l0.mix.uv"].reshape(H, E, -1)).reshape(8, -1) @ W["l0.mix.o"].T
    assert np.allclose(o, R.latent_mixer(W, "l0", h, m, eps))


@pytest.mark.parametrize("name", sorted(fm.ALL))
def test_oracle_is_causal(name):
    cfg = fm.ALL[name]()
    W = bm.as_numpy(fm.weights(cfg))
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 30)
    full, part = R.forward(cfg, W, toks), R.forward(cfg, W, toks[:17])
    assert np.abs(full[:17] - part).max() < 1e-9


# ---- product host code ----
def test_rotary_frequencies_match_the_oracle():
    for base, dims in ((1e4, 64), (5e5, 16), (100.0, 2)):
        assert np.allclose(Rotary(base, dims).frequencies(), R.half_frequencies(base, dims), rtol=1e-12)


def test_configuration_is_read_in_full():
    spec = fimadra.spec_from_config(fm.mixed())
    a, b, c, d, _ = spec.layers
    assert (a.mixer, a.heads, a.dim, a.vdim, a.q_rank, a.kv_rank, a.dense_ff, a.ff_act) == ("latent_attention", 3, 20, 28, 36, 24, 56, "square_relu")
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.chunk, b.rot_halves, b.qk_norm, b.dense_ff) == ("attention", 6, 2, 24, 40, 37, True, True, 0)
    assert (b.rotary.dims, b.rotary.base, b.scale, d.scale) == (16, 500.0, 1.0, 0.7)
    assert (c.mixer, c.heads, c.dim, c.vdim, c.gate_cap, c.dense_ff) == ("mlstm", 3, 20, 28, 9.0, 40)
    assert (a.channels, b.channels, c.channels) == (60, 6 * 24 + 2 * 64, 3 * (2 * 48 + 2))
    assert (spec.rms_norm, spec.post_norm, spec.logit_scale, spec.norm_eps, spec.runs()) == (True, False, 0.6, 1e-5, [0, 1, 2, 3, 4])
    assert a.state_shapes(2, 128, 0)[0] == ((2, 128, 24), False) and c.state_shapes(2, 0, 0) == [((2, 3, 20, 28), True), ((2, 3, 20), True), ((2, 3), True)]
    for change in ({"type": "other"}, {"mlp": {"kind": "moe", "ff": 3}}):
        bad = fm.mixed()
        bad["layers"][1].update(change)
        with pytest.raises(ValueError, match="layer 1"):
            fimadra.spec_from_config(bad)


def test_weights_are_mapped_and_checked():
    cfg = fm.mixed()
    state, spec = fm.weights(cfg), fimadra.spec_from_config(cfg)
    w = fimadra.weights_from_state(spec, state)["layers"]
    assert torch.equal(w[0]["qkv"][36:], state["l0.mix.dkv"]) and torch.equal(w[1]["qkv"][6 * 24:8 * 24], state["l1.mix.k"])
    assert torch.equal(w[2]["qkv"][-3:], state["l2.mix.f"]) and torch.equal(w[2]["qkv"][-6 - 84:-6], state["l2.mix.g"])
    assert torch.equal(w[2]["gate_bias"], torch.cat([state["l2.mix.i.b"], state["l2.mix.f.b"]]))
    assert torch.equal(w[0]["up"], state["l0.mlp.up"]) and "up" not in w[1] and "norm2" not in w[1]
    broken = dict(state)
    broken["l2.mix.f.b"] = broken["l2.mix.f.b"][:1]
    with pytest.raises(CheckpointError, match="l2.mix.f.b"):
        fimadra.weights_from_state(spec, broken)
    del broken["l2.mix.f.b"]
    with pytest.raises(CheckpointError, match="missing"):
        fimadra.weights_from_state(spec, broken)


def test_registry_chooses_by_configuration():
    assert registry.family_of(fm.odd()).name == "fimadra" and registry.family_of(bm.mixed()).name == "vebisun"


def _configure(**change):
    layer = dict(heads=4, kv_heads=2, dim=16, vdim=16, cache_rows=128, attn_scale=0.25, dense_ff=8, ff_act=ffi.ACT_SQUARE_RELU)
    model = dict(n_layers=1, hidden=32, vocab=50, max_seq_len=500, batch=1, dtype=ffi.BF16, max_prefill=64, max_rewind=8, loop_times=1, rms_norm=1,
                 embed_scale=1.0, residual_mult=1.0, norm_eps=1e-5)
    fields = {n for n, _ in ffi.Block._fields_}
    for k, v in change.items():
        (layer if k in fields else model)[k] = v
    arr = (ffi.Block * 1)(ffi.Block(**layer))
    return ffi.lib().mynn_b200_model_configure_blocks(ffi.BlockModelConfig(layers=arr, **model))


def test_block_configuration_is_validated():
    lat = dict(mixer=ffi.MIX_LATENT, kv_heads=4, q_rank=8, kv_rank=8, cache_rows=512)
    mem = dict(mixer=ffi.MIX_MLSTM, kv_heads=4, gate_cap=15.0, cache_rows=0)
    assert _configure(chunk=20, qk_norm=1, rot_halves=1, rot_dims=8) == ffi.OK and _configure(**lat) == ffi.OK and _configure(**mem) == ffi.OK
    for bad in (dict(chunk=90), dict(), dict(chunk=20, dense_ff=-1), dict(chunk=20, ff_act=7), dict(chunk=20, conv_taps=2, history_rows=20, qk_norm=1),
                dict(chunk=20, experts=4, expert_ff=8, top=1, groups=1, groups_keep=1), dict(chunk=20, mixer=9), {**lat, "cache_rows": 384},
                {**lat, "kv_rank": 0}, {**lat, "chunk": 20}, {**lat, "softcap": 3.0}, {**mem, "gate_cap": 0.0}, {**mem, "dim": 600}, {**mem, "window": 3}):
        assert _configure(**bad) == ffi.E_ARG, bad
    assert _configure(chunk=20, dense_ff=0) == ffi.OK


class Recurrent:
    """A stand-in whose next token is the sum of all it has seen; it refuses to go back."""
    batch, output, max_seq_len, vocab, streaming, max_prefill, can_rewind = 1, "ids", 60, 1000, None, 4, False

    def __init__(self):
        self.seen = []

    def _take(self, tokens, past_len):
        if past_len == 0:
            self.seen = []
        assert past_len == len(self.seen), "went back"
        self.seen += list(tokens)
        return [sum(self.seen) % 97]

    def step(self, tokens, past_len):
        return self._take(tokens, past_len)

    def prefill(self, tokens, past_len):
        return self._take(tokens[0], past_len)


class Letters:
    def decode(self, ids):
        return "".join(f"<{i}>" for i in ids)


@pytest.mark.parametrize("prefill", [None, 4])
def test_session_runs_a_shortened_conversation_again(prefill):
    model = Recurrent()
    s = LlmSession.for_model(model, -1, prefill_len=prefill, tokenizer=Letters())
    free = s.generate_ids([5, 6, 7], 6)
    s.reset()
    got = s.generate_ids([5, 6, 7], opts=GenerateOptions(6, [f"<{free[2]}><{free[3]}>"]))
    assert got == free[:3]  # the stop string's last token is dropped, past_len with it
    kept = [5, 6, 7] + free[:3]
    assert s.past_len() == 5
    more = s.generate_ids([1, 2], 2)
    assert model.seen[:7] == kept[:5] + [1, 2] and more[0] == (sum(kept[:5]) + 3) % 97
    s.reset()
    assert s.generate_ids([9], 1) == [9]


def test_rewinding_models_are_not_run_again():
    class Ring(Recurrent):
        can_rewind = True
    assert LlmSession.for_model(Ring(), -1)._stored is None
