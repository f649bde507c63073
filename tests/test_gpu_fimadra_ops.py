"""The operators behind Fimadra on the GPU, each alone against the oracle (float64)."""
import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

from my_nn_engine_b200 import ffi, ops  # noqa: E402
from oracle import ref_fimadra as R  # noqa: E402
from oracle import ref_vebisun as RV  # noqa: E402

DT = {"bf16": torch.bfloat16, "f16": torch.float16, "f32": torch.float32}
TOL = {"bf16": 1.2e-2, "f16": 2e-3, "f32": 3e-6}


def cuda(a, dt=torch.float32):
    return torch.as_tensor(np.ascontiguousarray(a)).to(dt).cuda()


def host(t):
    return t.double().cpu().numpy()


def close(got, want, tol, what=""):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape, (got.shape, want.shape)
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= tol, f"{what}: {err:.3g} > {tol}"


def past(n):
    return torch.tensor([n], dtype=torch.int32, device="cuda")


# ---- norm with residual ----
@pytest.mark.parametrize("W", [5, 50, 72, 1000, 2048, 4100])
@pytest.mark.parametrize("dt", ["bf16", "f32"])
def test_residual_rms_norm(W, dt):
    rng = np.random.default_rng(W)
    x, sub, w = cuda(rng.standard_normal((5, W)) + 3.0), cuda(rng.standard_normal((5, W)) * 4, DT[dt]), cuda(rng.standard_normal(W))
    want = host(x) + host(sub)
    y = x.clone()
    out = ops.residual_rms_norm(y, sub, w, 1e-5)
    close(host(y), want, 1e-6)
    close(host(out), R.rms(want, 1e-5) * host(w), TOL[dt])
    close(host(ops.residual_rms_norm(y, None, w, 1e-5, DT[dt])), R.rms(host(y), 1e-5) * host(w), TOL[dt])
    tiny = cuda(rng.standard_normal((3, W)) * 1e-2)  # eps counts
    close(host(ops.residual_rms_norm(tiny, None, w, 0.5)), R.rms(host(tiny), 0.5) * host(w), 3e-6)
    z = x.clone()
    assert ops.residual_rms_norm(z, sub, None, 1e-5) is None and torch.equal(y, z)


# ---- rotation, head norms, append ----
@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("H,G,D,E,dims,rows,start,S", [(6, 2, 24, 40, 16, 128, 0, 50), (3, 1, 14, 9, 6, 128, 120, 20), (4, 4, 64, 64, 64, 256, 250, 1),
                                                        (8, 2, 128, 128, 32, 128, 300, 77), (2, 2, 10, 6, 10, 128, 5, 2), (1, 1, 32, 16, 0, 128, 7, 3)])
def test_rotary_append(dt, H, G, D, E, dims, rows, start, S):
    rng = np.random.default_rng(H * D)
    B, C = 2, H * D + G * (D + E)
    proj = cuda(rng.standard_normal((B, S, C)) * 3, DT[dt])
    f = R.half_frequencies(700.0, dims)
    ang = np.arange(start + S)[:, None] * f[None]
    cos, sin = (cuda(np.cos(ang)), cuda(np.sin(ang))) if dims else (None, None)
    pos = np.arange(start, start + S)
    x = host(proj)
    for halves, qk_norm in ((True, True), (False, True), (True, False)):
        kc, vc = torch.full((B, G, rows, D), 9.0, dtype=DT[dt], device="cuda"), torch.full((B, G, rows, E), 9.0, dtype=DT[dt], device="cuda")
        q = ops.rotary_append(proj, past(start), kc, vc, H, cos, sin, halves, qk_norm, 1e-3)
        turn = R.rotate_halves if halves else RV.rotate_interleaved
        norm = (lambda a: R.rms(a, 1e-3)) if qk_norm else (lambda a: a)
        for b in range(B):
            wq = norm(turn(x[b, :, :H * D].reshape(S, H, D), pos, f))
            wk = norm(turn(x[b, :, H * D:(H + G) * D].reshape(S, G, D), pos, f))
            wv = x[b, :, (H + G) * D:].reshape(S, G, E)
            close(host(q)[b], wq.transpose(1, 0, 2), TOL[dt] / 2, "q")
            close(host(kc)[b][:, pos % rows], wk.transpose(1, 0, 2), TOL[dt] / 2, "k")
            assert np.array_equal(host(vc)[b][:, pos % rows], wv.transpose(1, 0, 2))
            rest = np.setdiff1d(np.arange(rows), pos % rows)
            assert (host(kc)[b][:, rest] == 9.0).all() and (host(vc)[b][:, rest] == 9.0).all()


# ---- chunk mask ----
def ring(x, rows, dt):
    """[T, G, D] -> ring [1, G, rows, D] that holds the last positions, others a finite mark."""
    T, G, D = x.shape
    out = np.full((1, G, rows, D), 5.0)
    for p in range(max(0, T - rows), T):
        out[0, :, p % rows] = x[p]
    return cuda(out, DT[dt])


CHUNK_SHAPES = [("f32", 4, 2, 20, 12), ("bf16", 4, 2, 64, 64), ("bf16", 3, 1, 128, 128), ("bf16", 6, 2, 64, 64), ("f16", 2, 2, 128, 128), ("bf16", 4, 1, 24, 40)]


@pytest.mark.parametrize("dt,H,G,D,E", CHUNK_SHAPES)
@pytest.mark.parametrize("size", [1, 16, 100, 128, 1000])
def test_chunk_mask_shows_at_every_edge(dt, H, G, D, E, size):
    """One key stands out wherever it is seen; it sits on either side of a chunk's edge, and every query row is compared."""
    rng = np.random.default_rng(size)
    T = 330
    u = np.sign(rng.standard_normal(D))
    spots = sorted({p for e in (size, 2 * size, 3 * size) for p in (e - 1, e) if 0 < p < T} | {0, 200})[:6]
    for i, spot in enumerate(spots):
        q = np.broadcast_to(u, (T, H, D)) + 0.1 * rng.standard_normal((T, H, D))
        k, v = 0.3 * rng.standard_normal((T, G, D)), rng.standard_normal((T, G, E))
        k[spot], v[spot] = u, 6.0
        q, k, v = (host(cuda(a, DT[dt])) for a in (q, k, v))
        want = R.softmax_attention(q, k, v, 12.0 / D, size)
        rows = 384 if i % 2 else 128 * (-(-(min(size, T) + 63) // 128))  # a ring as short as the chunk allows, or the whole past
        for Sq in (1, 2, 17, 64):
            for active in sorted({T, min(T, spot + 1), min(T, max(Sq, spot + Sq // 2 + 1)), min(T, max(Sq, 2 * size))}):
                if active < Sq or rows < Sq + min(size, active) - 1:
                    continue
                kc, vc = ring(k[:active], rows, dt), ring(v[:active], rows, dt)
                qt = cuda(q[active - Sq:active].transpose(1, 0, 2)[None], DT[dt])
                for plain in (False, True):
                    got = host(ops.chunk_attention(qt, kc, vc, 12.0 / D, active, chunk=size, plain=plain))[0]
                    close(got, want[active - Sq:active], TOL[dt], f"spot {spot}, {Sq} rows up to {active}, ring {rows}, plain {plain}")
    ops.attention_check()


@pytest.mark.parametrize("dt,H,G,D,E", [("bf16", 4, 2, 64, 64), ("bf16", 5, 5, 128, 128), ("f32", 3, 3, 20, 28)])
def test_head_major_layout_equals_the_other(dt, H, G, D, E):
    rng = np.random.default_rng(3)
    B, S, rows = 3, 40, 256
    q, k, v = (cuda(rng.standard_normal(s), DT[dt]) for s in ((B, H, S, D), (B, G, rows, D), (B, G, rows, E)))
    a = ops.chunk_attention(q, k, v, 0.2, 170)
    b = ops.chunk_attention(*(t.transpose(0, 1).contiguous() for t in (q, k, v)), 0.2, 170, head_major=True)
    assert torch.equal(a, b)
    # window and chunk together: the nearer bound counts
    c = host(ops.chunk_attention(q, k, v, 0.2, 170, window=30, chunk=64))
    for b_ in range(B):
        qq, kk, vv = host(q)[b_].transpose(1, 0, 2), host(k)[b_].transpose(1, 0, 2), host(v)[b_].transpose(1, 0, 2)
        for s in (0, 1, S - 1):
            p = 170 - S + s
            lo = max(p - 29, p - p % 64)
            want = R.softmax_attention(np.concatenate([np.zeros((p - lo, H, D)), qq[s:s + 1]]), kk[lo:p + 1], vv[lo:p + 1], 0.2)[-1]
            close(c[b_, s], want, TOL[dt])


# ---- latents ----
@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("Q,RK,start,S", [(36, 24, 0, 9), (11, 13, 120, 30), (128, 512, 3, 1), (1, 1, 0, 2)])
def test_latent_append(dt, Q, RK, start, S):
    rng = np.random.default_rng(Q)
    proj, wq, wc = cuda(rng.standard_normal((2, S, Q + RK)) * 2, DT[dt]), cuda(rng.standard_normal(Q)), cuda(rng.standard_normal(RK))
    cache = torch.full((2, 256, RK), 3.0, dtype=DT[dt], device="cuda")
    got = ops.latent_append(proj, past(start), cache, wq, wc, 0.01)
    x = host(proj)
    close(host(got), R.rms(x[..., :Q], 0.01) * host(wq), TOL[dt] / 2)
    close(host(cache)[:, start:start + S], R.rms(x[..., Q:], 0.01) * host(wc), TOL[dt] / 2)
    assert (host(cache)[:, start + S:] == 3.0).all() and (host(cache)[:, :start] == 3.0).all()


@pytest.mark.parametrize("dt,RK", [("bf16", 128), ("bf16", 256), ("bf16", 512), ("f16", 256), ("bf16", 64), ("bf16", 40), ("f32", 24), ("f32", 700)])
@pytest.mark.parametrize("H", [1, 16, 18, 40])
def test_latent_attention(dt, RK, H):
    rng = np.random.default_rng(RK + H)
    rows = 640
    c = rng.standard_normal((2, rows, RK))
    u = np.sign(rng.standard_normal(RK))
    c[:, 64], c[:, 127], c[:, 300] = u, -u, 0.7 * u  # keys that stand out, at tile borders and far back
    cache = cuda(c, DT[dt])
    c = host(cache)
    scale = 14.0 / RK
    for Sq, active, B in ((1, 1, 2), (1, 64, 1), (1, 65, 1), (2, 129, 2), (16, 301, 1), (3, 640, 1), (1, 640, 2)):
        q = cuda(rng.standard_normal((B, Sq, H, RK)) * 0.3 + u, DT[dt])
        want = []
        for b in range(B):
            rowsq = []
            for s in range(Sq):
                n = active - Sq + s + 1
                sc = host(q)[b, s] @ c[b, :n].T * scale
                e = np.exp(sc - sc.max(-1, keepdims=True))
                rowsq.append((e / e.sum(-1, keepdims=True)) @ c[b, :n])
            want.append(rowsq)
        for kw in ({}, {"plain": True}, {"workspace": False}):
            close(host(ops.latent_attention(q, cache[:B].contiguous(), scale, active, **kw)), np.array(want), TOL[dt], f"{Sq} rows up to {active}, {kw}")
    assert torch.equal(ops.latent_attention(q, cache, scale, 640), ops.latent_attention(q, cache, scale, 640))


# ---- matrix memory ----
def memory_inputs(rng, B, S, H, D, E, dt, forget=4.0, spread=2.0):
    proj = cuda(rng.standard_normal((B, S, 2 * H * (D + E))), DT[dt])
    gates = cuda(rng.standard_normal((B, S, 2 * H)) * spread)
    bias = cuda(np.concatenate([rng.standard_normal(H), forget + rng.standard_normal(H)]))
    return proj, gates, bias, cuda(1 + 0.2 * rng.standard_normal(H * E))


def memory_oracle(proj, gates, bias, norm, H, D, E, cap, eps):
    """[B, S, H E] and the last state, per sequence from its first token."""
    outs, states = [], []
    for b in range(proj.shape[0]):
        x, g, S = host(proj)[b], host(gates)[b] + host(bias), proj.shape[1]
        q, k = (x[:, i * H * D:(i + 1) * H * D].reshape(S, H, D) for i in (0, 1))
        v, z = (x[:, 2 * H * D + i * H * E:2 * H * D + (i + 1) * H * E] for i in (0, 1))
        tr = []
        o = R.matrix_memory(q * D ** -0.5, k, v.reshape(S, H, E), R.soft_cap(g[:, :H], cap), R.log_sigmoid(R.soft_cap(g[:, H:], cap)), tr)
        outs.append(R.rms(o, eps).reshape(S, H * E) * host(norm) / (1 + np.exp(-z)))
        states.append(tr[-1])
    return np.array(outs), states


MEMORY_SHAPES = [("f32", 3, 20, 28, [0, 1]), ("f32", 1, 70, 33, [1]), ("bf16", 2, 48, 40, [1, 2]), ("bf16", 1, 64, 96, [0, 1, 2]), ("bf16", 2, 128, 72, [1, 2, 3]),
                 ("bf16", 1, 200, 32, [1, 2]), ("bf16", 1, 200, 136, [0, 2]), ("bf16", 1, 256, 136, [0, 2, 3]), ("f16", 1, 32, 32, [1, 2]), ("f16", 1, 128, 264, [2, 3]),
                 ("f32", 1, 300, 16, [1]), ("bf16", 2, 6, 10, [0, 1])]


@pytest.mark.parametrize("dt,H,D,E,forms", MEMORY_SHAPES)
def test_matrix_memory_in_portions(dt, H, D, E, forms):
    rng = np.random.default_rng(D)
    B, S, cap, eps = 2, 200, 6.0, 1e-4
    proj, gates, bias, norm = memory_inputs(rng, B, S, H, D, E, dt)
    want, states = memory_oracle(proj, gates, bias, norm, H, D, E, cap, eps)
    for form in forms:
        for sizes in ([S], [63, 1, 64, 2, 65, 5], [1] * 8 + [2, 3, 129, 58]):
            st, pos, got = ops.MlstmState(B, H, D, E), 0, []
            for t in (st.mem, st.sum, st.top):
                t.fill_(77.0)  # what an earlier sequence left: nothing of it may count
            for n in sizes:
                got.append(ops.mlstm(proj[:, pos:pos + n].contiguous(), gates[:, pos:pos + n].contiguous(), bias, norm, st, past(pos), cap, eps, form))
                pos += n
            close(host(torch.cat(got, 1)), want, TOL[dt], f"form {form}, {sizes}")
            for b in range(B):
                for name, mine, ref in zip(("S", "n", "m"), (st.mem, st.sum, st.top), states[b]):
                    # 32-bit whatever the dtype; chunkwise products keep the values as two 16-bit parts
                    close(host(mine)[b], ref, 4e-6 if dt == "f32" or form == 1 else 2e-5, f"state {name}, form {form}, {sizes}")
            assert not st.tickets.any() and not st.status.any()


@pytest.mark.parametrize("form", [1, 2, 3])
@pytest.mark.parametrize("forget,spread", [(-30.0, 3.0), (30.0, 0.1), (0.0, 40.0)], ids=["forgets all", "keeps all", "gates at their caps"])
def test_matrix_memory_with_extreme_gates(form, forget, spread):
    rng = np.random.default_rng(4)
    H, D, E, cap = 2, 128, 72, 15.0
    proj, gates, bias, norm = memory_inputs(rng, 1, 350, H, D, E, "bf16", forget, spread)
    want, _ = memory_oracle(proj, gates, bias, norm, H, D, E, cap, 1e-6)
    st = ops.MlstmState(1, H, D, E)
    got = [ops.mlstm(proj[:, a:b].contiguous(), gates[:, a:b].contiguous(), bias, norm, st, past(a), cap, 1e-6, form) for a, b in ((0, 300), (300, 350))]
    close(host(torch.cat(got, 1)), want, TOL["bf16"])
    assert not st.status.any()


def test_matrix_memory_remembers_one_token_over_hundreds():
    """A key that comes once, far back, and a query for it at the end: the state in between has to carry it."""
    rng = np.random.default_rng(5)
    H, D, E, T = 1, 128, 64, 700
    for dt, forms in (("f32", [1]), ("bf16", [1, 2, 3])):
        x = 0.05 * rng.standard_normal((1, T, 2 * H * (D + E)))
        u = np.sign(rng.standard_normal(D))
        x[0, 3, D:2 * D] = u
        x[0, 3, 2 * D:2 * D + E] = 4.0
        x[0, -1, :D] = u
        proj, gates = cuda(x, DT[dt]), cuda(np.zeros((1, T, 2)))
        bias, norm = cuda(np.array([0.0, 9.0])), cuda(np.ones(E))
        want, _ = memory_oracle(proj, gates, bias, norm, H, D, E, 10.0, 1e-6)
        assert (want[0, -1] > 0.3).all() and np.abs(want[0, -2]).max() < 10  # (the gate halves what the norm brings to about one)
        for form in forms:
            st = ops.MlstmState(1, H, D, E)
            got = [ops.mlstm(proj[:, a:b].contiguous(), gates[:, a:b].contiguous(), bias, norm, st, past(a), 10.0, 1e-6, form) for a, b in ((0, 640), (640, 699), (699, 700))]
            close(host(got[-1])[0, -1], want[0, -1], TOL[dt])


def test_matrix_memory_in_segments_equals_token_by_token():
    """Long prompts over few heads are cut into segments that run side by side; two prompts in a row, state and outputs."""
    rng = np.random.default_rng(6)
    for H, D, E, S in ((1, 256, 128, 1100), (3, 128, 200, 700), (2, 64, 64, 900)):
        proj, gates, bias, norm = memory_inputs(rng, 1, S, H, D, E, "bf16", 5.0, 1.0)
        ref, refs = ops.MlstmState(1, H, D, E), []
        for a, b in ((0, S - 130), (S - 130, S)):
            refs.append(ops.mlstm(proj[:, a:b].contiguous(), gates[:, a:b].contiguous(), bias, norm, ref, past(a), 12.0, 1e-6, 1))
        for form in (0, 2):
            st = ops.MlstmState(1, H, D, E)
            for (a, b), want in zip(((0, S - 130), (S - 130, S)), refs):
                got = ops.mlstm(proj[:, a:b].contiguous(), gates[:, a:b].contiguous(), bias, norm, st, past(a), 12.0, 1e-6, form)
                close(host(got), host(want), 1e-2, f"{H} {D} {E} form {form} from {a}")
            for mine, theirs in ((st.mem, ref.mem), (st.sum, ref.sum), (st.top, ref.top)):
                close(host(mine), host(theirs), 3e-5)
            assert not st.status.any()


# ---- products ----
@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("M", [1, 7, 40, 64, 200])
@pytest.mark.parametrize("N,K", [(96, 72), (333, 40), (1040, 256), (60, 50)])
def test_product_options(dt, M, N, K):
    rng = np.random.default_rng(M + N)
    act, w = cuda(rng.standard_normal((M, K)), DT[dt]), cuda(rng.standard_normal((N, K)) * K ** -0.5, DT[dt])
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ref = host(act) @ host(w).T
    close(host(ops.dense_matmul_ex(act, w, ffi.ACT_SQUARE_RELU, status=status)), R.square_relu(ref), TOL[dt])
    for cols in (1, 6, 40):
        main, extra = ops.dense_matmul_ex(act, w, f32_columns=cols, status=status)
        close(host(main), ref[:, :-cols], TOL[dt])
        assert extra.dtype == torch.float32
        close(host(extra), ref[:, -cols:], 3e-6)
    for block in [b for b in (5, 12, 32, 16, 111, 208) if N % b == 0]:
        got = ops.dense_matmul_ex(act, w, block=block, status=status)
        close(host(got), ref.reshape(M, N // block, block).transpose(1, 0, 2), TOL[dt])
    assert int(status) == 0


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("M,H,N,K", [(1, 3, 24, 20), (5, 18, 256, 128), (33, 2, 40, 64), (130, 4, 128, 64), (2, 1, 7, 13)])
def test_one_product_per_head(dt, M, H, N, K):
    rng = np.random.default_rng(M + N)
    act, w = cuda(rng.standard_normal((M, H, K)), DT[dt]), cuda(rng.standard_normal((H, N, K)) * K ** -0.5, DT[dt])
    close(host(ops.dense_matmul_heads(act, w)), np.einsum("mhk,hnk->mhn", host(act), host(w)), TOL[dt])


def test_operators_refuse_what_they_cannot_do():
    x = torch.zeros(1, 4, 2 * 2 * 20, device="cuda", dtype=torch.bfloat16)
    st, g, w = ops.MlstmState(1, 2, 10, 10), torch.zeros(1, 4, 4, device="cuda"), torch.ones(20, device="cuda")
    with pytest.raises(ffi.MynnError, match="chunkwise"):
        ops.mlstm(x, g, torch.zeros(4, device="cuda"), w, st, past(0), 5.0, 1e-6, form=2)
    with pytest.raises(ffi.MynnError, match="bad shape"):
        ops.mlstm(x, g, torch.zeros(4, device="cuda"), w, st, past(0), 0.0, 1e-6)
    with pytest.raises(ffi.MynnError, match="positions"):
        ops.latent_attention(torch.zeros(1, 2, 1, 128, device="cuda", dtype=torch.bfloat16), torch.zeros(1, 128, 128, device="cuda", dtype=torch.bfloat16), 1.0, 129)
    with pytest.raises(ffi.MynnError, match="ring"):
        ops.rotary_append(torch.zeros(1, 9, 24, device="cuda"), past(0), torch.zeros(1, 1, 8, 8, device="cuda"), torch.zeros(1, 1, 8, 8, device="cuda"), 1, None, None)
