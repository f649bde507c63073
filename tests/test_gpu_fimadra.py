"""The Fimadra family on the GPU against the oracle: whole prompts, portions, decoding, reuse of the state, batches, generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

from my_nn_engine_b200 import ffi, fimadra, registry  # noqa: E402
from my_nn_engine_b200.checkpoint import write_safetensors  # noqa: E402
from my_nn_engine_b200.session import GenerateOptions, LlmSession  # noqa: E402
from oracle import ref_fimadra as R  # noqa: E402
from tests import block_models as bm  # noqa: E402
from tests import fimadra_models as fm  # noqa: E402

F32_LIMIT = 2e-5
LENGTH = 330
_cache = {}


def case(name):
    """(cfg, state, tokens, oracle logits [LENGTH, vocab]) of a small model, computed once."""
    if name not in _cache:
        cfg = fm.ALL[name]()
        state = fm.weights(cfg, seed=len(name))
        toks = np.random.default_rng(5).integers(0, cfg["vocab"], LENGTH).tolist()
        _cache[name] = cfg, state, toks, R.forward(cfg, bm.as_numpy(state), toks)
    return _cache[name]


def model_of(name, dtype, **kw):
    cfg, state, _, _ = case(name)
    kw.setdefault("max_seq_len", LENGTH + 20)
    return fimadra.build(cfg, state, dtype=dtype, **kw)


def run(model, toks, portions):
    """Logits of every token, fed in portions."""
    out, pos = [], 0
    for n in portions:
        out.append(model.feed(toks[pos:pos + n], pos, range(n)).numpy().copy())
        pos += n
    assert pos == len(toks)
    return np.concatenate(out)


def portions(total, sizes):
    out, i = [], 0
    while sum(out) < total:
        out.append(min(sizes[i % len(sizes)], total - sum(out)))
        i += 1
    return out


def limit(name, dtype):
    """What a row's error may be: in 16 bits 2.5 times the worst that rounding the stored activations alone does to this model."""
    if dtype == "f32":
        return F32_LIMIT
    if (name, dtype) not in _cache:
        cfg, state, toks, want = case(name)
        _cache[name, dtype] = 2.5 * bm.rel_error(R.forward(cfg, bm.as_numpy(state), toks, store=R.bf16), want).max()
    return _cache[name, dtype]


def check(got, want, dtype, name, what=""):
    e, top = bm.rel_error(got, want), limit(name, dtype)
    worst = int(e.argmax())
    assert e[worst] <= top, f"{name} {what}: {(e > top).mean():.3f} of the rows over {top:.3g}, worst {e[worst]:.3g} at {worst}, first at {int(np.argmax(e > top))}"


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(fm.ALL))
@pytest.mark.parametrize("sizes", [[LENGTH], [1], [2], [3, 64, 2, 17, 1, 5], [100, 129], [16], [37, 13]], ids=str)
def test_portions(name, dtype, sizes):
    _, _, toks, want = case(name)
    m = model_of(name, dtype, max_prefill=LENGTH if sizes == [LENGTH] else 130)
    check(run(m, toks, portions(LENGTH, sizes)), want, dtype, name, str(sizes))
    m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_prompt_then_long_decoding_past_several_ring_turns(name, dtype):
    _, _, toks, want = case(name)
    m = model_of(name, dtype, max_prefill=8, max_rewind=0)  # rings as short as they can be
    if name == "mixed":
        assert min(s[0].shape[2] for s, L in zip(m.run_states, m.spec.layers) if L.chunk) == 128
    check(run(m, toks, [8, 5] + [1] * (LENGTH - 13)), want, dtype, name)
    m.close()


@pytest.mark.parametrize("name", ["chunkwise", "wide"])
def test_without_a_graph_and_with_the_plain_prefill_kernels(name):
    _, _, toks, want = case(name)
    m = model_of(name, "bf16", max_prefill=64, use_graph=False)
    ffi.set_option(ffi.OPT_PREFILL_ATTENTION, 0)
    ffi.set_option(ffi.OPT_DECODE_RING, 0)
    try:
        check(run(m, toks, portions(LENGTH, [64, 33, 1, 1, 1])), want, "bf16", name)
    finally:
        ffi.set_option(ffi.OPT_PREFILL_ATTENTION, 1)
        ffi.set_option(ffi.OPT_DECODE_RING, 1)
    m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(fm.ALL))
def test_state_is_given_back_and_used_again(name, dtype):
    """A long sequence, then shorter ones in the same caches and memories: nothing of the earlier one may show, also in its first tokens."""
    _, _, toks, want = case(name)
    m = model_of(name, dtype, max_prefill=50)
    run(m, toks[::-1], portions(LENGTH, [50]))
    check(run(m, toks[:1], [1]), want[:1], dtype, name, "one token")
    check(run(m, toks[:23], [2, 1, 20]), want[:23], dtype, name, "short")
    fresh = model_of(name, dtype, max_prefill=50)
    a, b = run(m, toks[:90], [50, 40]), run(fresh, toks[:90], [50, 40])
    assert np.array_equal(a, b)  # the same kernels on the same inputs: not even rounding may differ
    m.close()
    fresh.close()


def test_a_recurrent_state_does_not_go_back():
    _, _, toks, want = case("mixed")
    m = model_of("mixed", "f32", max_prefill=32)
    assert not m.can_rewind
    run(m, toks[:60], portions(60, [32]))
    for pos in (59, 61, 20):
        with pytest.raises(ffi.MynnError, match="recurrent state"):
            m.feed(toks[:2], pos)
        with pytest.raises(ffi.MynnError, match="recurrent state"):
            m.step(toks[:1], pos)
    check(m.feed(toks[60:70], 60, range(10)).numpy(), want[60:70], "f32", "mixed", "the refused steps changed nothing")
    check(run(m, toks[:40], [7, 32, 1]), want[:40], "f32", "mixed", "a new sequence after an error")
    m.close()
    cfg, state, _, _ = case("mixed")  # without its recurrent layer the same model can
    cfg = {**cfg, "layers": [e for e in cfg["layers"] if e["type"] != "mlstm"]}
    keep = [i for i, e in enumerate(case("mixed")[0]["layers"]) if e["type"] != "mlstm"]
    sub = {n: t for n, t in state.items() if not n.startswith("l")}
    sub.update({f"l{j}." + n.split(".", 1)[1]: t for j, i in enumerate(keep) for n, t in state.items() if n.startswith(f"l{i}.")})
    m = fimadra.build(cfg, sub, dtype="f32", max_seq_len=300, max_prefill=32, max_rewind=6)
    assert m.can_rewind
    want = R.forward(cfg, bm.as_numpy(sub), toks[:220])
    run(m, toks[:200], portions(200, [32]))
    check(m.feed(toks[194:210], 194, range(16)).numpy(), want[194:210], "f32", "mixed")
    m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(fm.ALL))
@pytest.mark.parametrize("sizes", [[64, 37, 2] + [1] * 47, [20, 109, 150, 1, 20]], ids=["decoding", "portions"])
def test_batch_against_each_alone(name, dtype, sizes):
    """Three different sequences side by side (one past length for all, as every model here batches)."""
    cfg, state, toks, _ = case(name)
    rng = np.random.default_rng(9)
    length = sum(sizes)
    seqs = [toks[:length], rng.integers(0, cfg["vocab"], length).tolist(), toks[30:30 + length]]
    W = bm.as_numpy(state)
    m = model_of(name, dtype, batch=3, max_prefill=max(sizes))
    got = [[] for _ in seqs]
    pos = 0
    for n in sizes:
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
        check(np.stack([g for _, g in got[b]]), want[[p for p, _ in got[b]]], dtype, name, f"sequence {b}")
    m.close()


def test_first_tokens_and_single_token_prompts():
    for name in sorted(fm.ALL):
        _, _, toks, want = case(name)
        m = model_of(name, "f32", max_prefill=16)
        for n in (1, 2, 3, 5):
            check(run(m, toks[:n], [n]), want[:n], "f32", name, str(n))
        m.close()


def save(tmp_path, name):
    cfg, state, toks, want = case(name)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), state)
    return str(tmp_path), cfg, state, toks, want


def greedy(cfg, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(R.forward(cfg, W, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("output", ["ids", "logits"])
def test_greedy_generation_through_the_session(tmp_path, output):
    d, cfg, state, toks, _ = save(tmp_path, "mixed")
    prompt, n = toks[:37], 24
    ids = greedy(cfg, bm.as_numpy(state), prompt, n)
    m = registry.load_model(d, dtype="f32", max_seq_len=128, max_prefill=16, output=output)
    s = LlmSession.for_model(m, eos_token_id=-1, prefill_len=16)
    assert s.generate_ids(prompt, n) == ids
    s.reset()
    assert LlmSession.for_model(m, eos_token_id=-1).generate_ids(prompt, 5) == ids[:5]  # the prompt token by token
    s.reset()
    assert s.generate_ids(prompt, opts=GenerateOptions(n)) == ids
    m.close()


class Letters:
    def decode(self, ids):
        return "".join(f"<{i}>" for i in ids)


def test_a_conversation_goes_on_behind_a_stop_string(tmp_path):
    d, cfg, state, toks, _ = save(tmp_path, "odd")
    W, prompt = bm.as_numpy(state), toks[:21]
    ids = greedy(cfg, W, prompt, 8)
    m = registry.load_model(d, dtype="f32", max_seq_len=128, max_prefill=16, output="ids")
    s = LlmSession.for_model(m, eos_token_id=-1, prefill_len=16, tokenizer=Letters())
    got = s.generate_ids(prompt, opts=GenerateOptions(8, [f"<{ids[3]}><{ids[4]}>"]))
    held = (prompt + got)[:s.past_len()]  # what the session counts as stored
    assert got == ids[:len(got)] and len(got) < 8
    more = toks[40:44]
    assert s.generate_ids(more, 5) == greedy(cfg, W, held + more, 5)
    m.close()


def test_generate_command(tmp_path):
    d, cfg, state, toks, _ = save(tmp_path, "chunkwise")
    ids = greedy(cfg, bm.as_numpy(state), toks[:20], 6)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "my_nn_engine_b200.generate", "--model", d, "--prompt-ids", ",".join(map(str, toks[:20])), "--dtype", "f32",
                        "--max-new-tokens", "6", "--max-seq-len", "64", "--prefill", "16"], cwd=root, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.strip().split(",")] == ids


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(tmp_path, dtype):
    dt = {"float32": "f32", "bfloat16": "bf16"}[dtype]
    d, cfg, _, toks, want = save(tmp_path, "mixed")
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

    check(read(0), want[[99, 0, 41]], dt, "mixed")
    assert not (out / "1.f32").exists()
    check(read(2), want[[102]], dt, "mixed")
    check(read(3), want[0:200:2], dt, "mixed")
