"""The Vebisun family on the GPU against the oracle: whole prompts, portions, decoding, reuse of the state, batches, generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

from my_nn_engine_b200 import ffi, registry, vebisun  # noqa: E402
from my_nn_engine_b200.checkpoint import write_safetensors  # noqa: E402
from my_nn_engine_b200.session import GenerateOptions, LlmSession  # noqa: E402
from oracle import ref_vebisun as R  # noqa: E402
from tests import block_models as bm  # noqa: E402

LIMIT = {"f32": 2e-5, "bf16": 4e-2}
LENGTH = 330
_cache = {}


def case(name, dtype="f32"):
    """(cfg, state, tokens, oracle logits [LENGTH, vocab]) of a small model, computed once; for bf16 the variant without an expert
    choice to tip."""
    if (name, dtype) not in _cache:
        cfg = bm.ALL[name]() if dtype == "f32" else bm.all_chosen(bm.ALL[name]())
        state = bm.weights(cfg, seed=len(name))
        toks = np.random.default_rng(5).integers(0, cfg["vocab"], LENGTH).tolist()
        _cache[name, dtype] = cfg, state, toks, R.forward(cfg, bm.as_numpy(state), toks)
    return _cache[name, dtype]


def model_of(name, dtype, routed=False, **kw):
    cfg, state, _, _ = case(name, "f32" if routed else dtype)
    kw.setdefault("max_seq_len", LENGTH + 20)
    return vebisun.build(cfg, state, dtype=dtype, **kw)


def run(model, toks, portions, past=0):
    """Logits of every token, fed in portions."""
    out, pos = [], 0
    for n in portions:
        out.append(model.feed(toks[pos:pos + n], past + pos, range(n)).numpy().copy())
        pos += n
    assert pos == len(toks)
    return np.concatenate(out)


def portions(total, sizes):
    out, i = [], 0
    while sum(out) < total:
        out.append(min(sizes[i % len(sizes)], total - sum(out)))
        i += 1
    return out


def check(got, want, dtype, what=""):
    e = bm.rel_error(got, want)
    worst = int(e.argmax())
    assert e[worst] <= LIMIT[dtype], f"{what}: {(e > LIMIT[dtype]).mean():.3f} of the rows over the limit, worst {e[worst]:.3g} at {worst}, first at {int(np.argmax(e > LIMIT[dtype]))}"


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(bm.ALL))
@pytest.mark.parametrize("sizes", [[LENGTH], [1], [2], [3, 64, 2, 17, 1, 5], [100, 129], [16]], ids=str)
def test_portions(name, dtype, sizes):
    _, _, toks, want = case(name, dtype)
    m = model_of(name, dtype, max_prefill=LENGTH if sizes == [LENGTH] else 130)
    check(run(m, toks, portions(LENGTH, sizes)), want, dtype, f"{name} {sizes}")
    m.close()


@pytest.mark.parametrize("name", sorted(bm.ALL))
@pytest.mark.parametrize("sizes", [[LENGTH], [1], [40, 3]], ids=str)
def test_routed_experts_in_16_bits(name, sizes):
    """With a real expert choice 16-bit rounding tips a close call now and then, and the rows that look at such a token follow it: the
    bulk of the rows has to agree."""
    _, _, toks, want = case(name)
    m = model_of(name, "bf16", routed=True, max_prefill=LENGTH)
    e = bm.rel_error(run(m, toks, portions(LENGTH, sizes)), want)
    assert np.median(e) < 2.5e-2 and (e < 0.1).mean() > 0.8, (np.median(e), (e < 0.1).mean())
    m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_prompt_then_long_decoding_past_several_ring_turns(dtype):
    _, _, toks, want = case("mixed", dtype)
    m = model_of("mixed", dtype, max_prefill=8, max_rewind=0)  # rings as short as they can be
    assert min(s[0].shape[2] for s in m.run_states) == 128
    check(run(m, toks, [8, 5] + [1] * (LENGTH - 13)), want, dtype)
    m.close()


@pytest.mark.parametrize("name", ["even_group", "odd_group"])
def test_without_a_graph_and_with_the_plain_prefill_kernels(name):
    _, _, toks, want = case(name, "bf16")
    m = model_of(name, "bf16", max_prefill=64, use_graph=False)
    ffi.set_option(ffi.OPT_PREFILL_ATTENTION, 0)
    ffi.set_option(ffi.OPT_DECODE_RING, 0)
    try:
        check(run(m, toks, portions(LENGTH, [64, 33, 1, 1, 1])), want, "bf16")
    finally:
        ffi.set_option(ffi.OPT_PREFILL_ATTENTION, 1)
        ffi.set_option(ffi.OPT_DECODE_RING, 1)
    m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(bm.ALL))
def test_state_is_given_back_and_used_again(name, dtype):
    """A long sequence, then shorter ones in the same rings: nothing of the earlier one may show, also in its first tokens."""
    cfg, state, toks, want = case(name, dtype)
    m = model_of(name, dtype, max_prefill=50)
    run(m, toks[::-1], portions(LENGTH, [50]))
    check(run(m, toks[:1], [1]), want[:1], dtype, "one token")
    check(run(m, toks[:23], [2, 1, 20]), want[:23], dtype, "short")
    fresh = model_of(name, dtype, max_prefill=50)
    a, b = run(m, toks[:90], [50, 40]), run(fresh, toks[:90], [50, 40])
    assert np.array_equal(a, b)  # the same kernels on the same inputs: not even rounding may differ
    m.close()
    fresh.close()


def test_rewind_within_the_allowed_positions_and_errors():
    _, _, toks, want = case("mixed")
    m = model_of("mixed", "f32", max_prefill=32, max_rewind=6)
    run(m, toks[:200], portions(200, [32]))
    got = run(m, toks[194:210], [4, 1, 11], past=194)
    check(got, want[194:210], "f32")
    with pytest.raises(ffi.MynnError, match="stored"):
        m.feed([1], 300)
    with pytest.raises(ffi.MynnError, match="rewind"):
        m.feed([1, 2], 5)
    check(run(m, toks[:40], [7, 32, 1]), want[:40], "f32", "a new sequence after an error")
    m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "even_group"])
def test_batch_against_each_alone(name, dtype):
    """Three different sequences side by side (one past length for all, as every model here batches)."""
    cfg, state, toks, _ = case(name, dtype)
    rng = np.random.default_rng(9)
    seqs = [toks[:150], rng.integers(0, cfg["vocab"], 150).tolist(), toks[100:250]]
    W = bm.as_numpy(state)
    m = model_of(name, dtype, batch=3, max_prefill=64)
    got = [[] for _ in seqs]
    pos = 0
    for n in [64, 37, 2] + [1] * 47:
        chunk = [s[pos:pos + n] for s in seqs]
        if n == 1:
            out = m.step([c[0] for c in chunk], pos).clone()
        else:
            out = m.prefill(chunk, pos).clone()
        pos += n
        for b in range(3):
            got[b].append((pos - 1, out[b].numpy()))
    for b, s in enumerate(seqs):
        want = R.forward(cfg, W, s)
        check(np.stack([g for _, g in got[b]]), want[[p for p, _ in got[b]]], dtype, f"sequence {b}")
    m.close()


def test_first_tokens_and_single_token_prompts():
    for name in sorted(bm.ALL):
        _, _, toks, want = case(name)
        m = model_of(name, "f32", max_prefill=16)
        for n in (1, 2, 3, 5):
            check(run(m, toks[:n], [n]), want[:n], "f32", f"{name} {n}")
        m.close()


def save(tmp_path, name, dtype="f32"):
    cfg, state, toks, want = case(name, dtype)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), state)
    return str(tmp_path), cfg, state, toks, want


@pytest.mark.parametrize("output", ["ids", "logits"])
def test_greedy_generation_through_the_session(tmp_path, output):
    d, cfg, state, toks, _ = save(tmp_path, "mixed")
    W, prompt, n = bm.as_numpy(state), toks[:37], 24
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(R.forward(cfg, W, ids)[-1].argmax()))
    m = registry.load_model(d, dtype="f32", max_seq_len=128, max_prefill=16, output=output)
    s = LlmSession.for_model(m, eos_token_id=-1, prefill_len=16)
    assert s.generate_ids(prompt, n) == ids[37:]
    s.reset()
    assert LlmSession.for_model(m, eos_token_id=-1).generate_ids(prompt, 5) == ids[37:42]  # the prompt token by token
    s.reset()
    assert s.generate_ids(prompt, opts=GenerateOptions(n)) == ids[37:]
    m.close()


def test_generate_command(tmp_path):
    d, cfg, state, toks, _ = save(tmp_path, "even_group")
    W, ids = bm.as_numpy(state), list(toks[:20])
    for _ in range(6):
        ids.append(int(R.forward(cfg, W, ids)[-1].argmax()))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "my_nn_engine_b200.generate", "--model", d, "--prompt-ids", ",".join(map(str, toks[:20])), "--dtype", "f32",
                        "--max-new-tokens", "6", "--max-seq-len", "64", "--prefill", "16"], cwd=root, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.strip().split(",")] == ids[20:]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(tmp_path, dtype):
    dt = {"float32": "f32", "bfloat16": "bf16"}[dtype]
    d, cfg, state, toks, want = save(tmp_path, "mixed", dt)
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:100], "want": [99, 0, 41]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[100:102], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[102:103], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": toks[:200], "want": list(range(0, 200, 2))}], "end": ["y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "220"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]

    def read(n):
        return np.fromfile(out / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"])

    check(read(0), want[[99, 0, 41]], dt)
    assert not (out / "1.f32").exists()
    check(read(2), want[[102]], dt)
    check(read(3), want[0:200:2], dt)


def test_other_families_feed_too():
    """The row-wise logits of prefill chunks on the int8 Llama graph agree with its own steps."""
    from my_nn_engine_b200.decoder import DecoderModel
    from my_nn_engine_b200.quantize import random_llama_state
    cfg = dict(hidden_size=256, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, head_dim=64, intermediate_size=512,
               vocab_size=300, rms_norm_eps=1e-5, rope_theta=10000.0)
    m = DecoderModel(cfg, random_llama_state(cfg, seed=3), dtype="f32", max_seq_len=128, max_prefill=70)
    toks = np.random.default_rng(0).integers(0, 300, 90).tolist()
    a = m.feed(toks, 0, range(90)).numpy()
    b = np.stack([m.step([t], i).clone().float().numpy()[0] for i, t in enumerate(toks)])
    assert bm.rel_error(a, b).max() < 1e-3
    m.close()
