"""The block decoder's operators on the GPU, each alone against the oracle (float64)."""
import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

from my_nn_engine_b200 import ops  # noqa: E402
from oracle import ref_vebisun as R  # noqa: E402

DT = {"bf16": torch.bfloat16, "f16": torch.float16, "f32": torch.float32}
TOL = {"bf16": 1.5e-2, "f16": 2e-3, "f32": 2e-6}


def cuda(a, dt=torch.float32):
    return torch.as_tensor(np.ascontiguousarray(a)).to(dt).cuda()


def host(t):
    return t.double().cpu().numpy()


def close(got, want, tol, what=""):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= tol, f"{what}: {err:.3g} > {tol}"


# ---- norms ----
@pytest.mark.parametrize("W", [5, 72, 256, 1000, 2048, 4100, 9001])
def test_layer_norm(W):
    rng = np.random.default_rng(W)
    x = rng.standard_normal((7, W)) * 3 + 40.0  # a mean that is large against the deviations
    w, b = rng.standard_normal(W), rng.standard_normal(W)
    xt, wt, bt = cuda(x), cuda(w), cuda(b)
    for dt in ("f32", "bf16"):
        close(host(ops.layer_norm(xt, wt, bt, 1e-5, DT[dt])), R.layer_norm(host(xt), host(wt), host(bt), 1e-5), 3e-5 if dt == "f32" else 5e-3)
    tiny = cuda(rng.standard_normal((3, W)) * 1e-3)  # eps counts
    close(host(ops.layer_norm(tiny, wt, bt, 1e-5)), R.layer_norm(host(tiny), host(wt), host(bt), 1e-5), 3e-5)


@pytest.mark.parametrize("W", [72, 513, 2048])
@pytest.mark.parametrize("dt", ["bf16", "f32"])
def test_residual_layer_norm(W, dt):
    rng = np.random.default_rng(W)
    x, sub, extra = cuda(rng.standard_normal((5, W))), cuda(rng.standard_normal((5, W)) * 7, DT[dt]), cuda(rng.standard_normal((5, W)))
    p, n = [cuda(rng.standard_normal(W)) for _ in range(2)], [cuda(rng.standard_normal(W)) for _ in range(2)]
    for ex in (None, extra):
        want = host(x) + 0.35 * R.layer_norm(host(sub), host(p[0]), host(p[1]), 1e-6) + (host(ex) if ex is not None else 0)
        y = x.clone()
        out = ops.residual_layer_norm(y, sub, p, 0.35, 1e-6, extra=ex, norm=n)
        close(host(y), want, 3e-6)
        close(host(out), R.layer_norm(want, host(n[0]), host(n[1]), 1e-6), TOL[dt])
        z = x.clone()
        assert ops.residual_layer_norm(z, sub, p, 0.35, 1e-6, extra=ex) is None
        assert torch.equal(z, y)


# ---- convolution, rotation, append ----
@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("Hq,G,D,E,taps,rotd", [(4, 2, 16, 24, 4, 8), (3, 1, 10, 6, 3, 10), (2, 2, 64, 64, 1, 0), (4, 4, 8, 8, 6, 2), (2, 1, 24, 8, 0, 24)])
@pytest.mark.parametrize("portions", [[29], [1] * 29, [2, 3, 2, 7, 2, 13], [20, 1, 1, 7]])
def test_short_conv_append(dt, Hq, G, D, E, taps, rotd, portions):
    rng = np.random.default_rng(7)
    B, T, rows, hist_rows = 2, 29, 32, taps + 5
    C = Hq * D + G * (D + E)
    u = cuda(rng.standard_normal((B, T, C)), DT[dt])
    w = cuda(rng.standard_normal((taps, C))) if taps else None
    f = R.rotary_frequencies(300.0, rotd) if rotd else None
    cos = cuda(np.cos(np.arange(T)[:, None] * f)) if rotd else None
    sin = cuda(np.sin(np.arange(T)[:, None] * f)) if rotd else None
    k, v = torch.zeros(B, G, rows, D, dtype=DT[dt]).cuda(), torch.zeros(B, G, rows, E, dtype=DT[dt]).cuda()
    hist = torch.full((B, hist_rows, C), 1e4, dtype=DT[dt]).cuda() if taps else None  # what an earlier sequence left
    past, qs = 0, []
    for n in portions:
        qs.append(ops.short_conv_append(u[:, past:past + n].contiguous(), torch.tensor([past], dtype=torch.int32).cuda(), k, v, Hq, w, hist, cos, sin))
        past += n
    q = torch.cat(qs, 2)
    for b in range(B):
        y = R.short_conv(host(u[b]), host(w).T) if taps else host(u[b])
        qr, kr, vr = y[:, :Hq * D].reshape(T, Hq, D), y[:, Hq * D:Hq * D + G * D].reshape(T, G, D), y[:, Hq * D + G * D:].reshape(T, G, E)
        if rotd:
            qr, kr = R.rotate_interleaved(qr, range(T), f), R.rotate_interleaved(kr, range(T), f)
        close(host(q[b]).transpose(1, 0, 2), qr, TOL[dt], "q")
        close(host(k[b, :, :T]).transpose(1, 0, 2), kr, TOL[dt], "k")
        close(host(v[b, :, :T]).transpose(1, 0, 2), vr, TOL[dt], "v")
        if taps:
            for p in range(T - min(hist_rows, portions[-1]), T):
                assert torch.equal(hist[b, p % hist_rows], u[b, p])


# ---- attention ----
def ring_of(x, rows):
    """[T, G, D] -> ring [G, rows, D] as it stands after position T - 1."""
    r = np.full((x.shape[1], rows, x.shape[2]), 3.0)
    for p in range(max(0, x.shape[0] - rows), x.shape[0]):
        r[:, p % rows] = x[p]
    return r


SHAPES = [(4, 2, 64, 64), (3, 1, 128, 128), (8, 2, 128, 128), (2, 2, 64, 64), (6, 2, 24, 40), (4, 1, 33, 9)]


@pytest.mark.parametrize("dt", ["bf16", "f16", "f32"])
@pytest.mark.parametrize("Hq,G,D,E", SHAPES)
@pytest.mark.parametrize("T,Sq,window,rows", [(50, 50, 0, 128), (300, 1, 33, 128), (300, 40, 33, 128), (700, 1, 500, 640), (777, 129, 200, 384),
                                              (1000, 2, 17, 128), (640, 128, 513, 640), (5, 5, 9, 128), (400, 17, 1, 128), (1300, 1, 1200, 1280)])
def test_window_attention_random(dt, Hq, G, D, E, T, Sq, window, rows):
    rng = np.random.default_rng(T + D)
    B = 2
    q, k, v = rng.standard_normal((B, T, Hq, D)) * 2, rng.standard_normal((B, T, G, D)), rng.standard_normal((B, T, G, E))
    t = DT[dt]
    q, k, v = (torch.as_tensor(a).to(t).double().numpy() for a in (q, k, v))
    qd = cuda(q[:, T - Sq:].transpose(0, 2, 1, 3), t)
    kd, vd = cuda(np.stack([ring_of(k[b], rows) for b in range(B)]), t), cuda(np.stack([ring_of(v[b], rows) for b in range(B)]), t)
    for cap in (0.0, 6.0):
        want = np.stack([oracle_rows(q[b], k[b], v[b], D ** -0.5, cap, window, range(T - Sq, T)) for b in range(B)])
        for plain in (False, True):
            got = ops.window_attention(qd, kd, vd, D ** -0.5, T, window, cap, plain)
            ops.attention_check()
            close(host(got), want, {"bf16": 2e-2, "f16": 4e-3, "f32": 5e-6}[dt], f"cap {cap} plain {plain}")


def oracle_rows(q, k, v, scale, cap, window, rows):
    """R.windowed_attention for some rows only: each as the last row of its own prefix."""
    out = []
    for i in rows:
        lo = max(0, i + 1 - (window or i + 1))
        qs = np.zeros((i + 1 - lo,) + q.shape[1:])
        qs[-1] = q[i]
        out.append(R.windowed_attention(qs[-1:], k[i:i + 1], v[i:i + 1], scale, cap or None, None)[0] if lo == i else _one(qs[-1], k[lo:i + 1], v[lo:i + 1], scale, cap))
    return np.stack(out)


def _one(q, k, v, scale, cap):
    H, G = q.shape[0], k.shape[1]
    out = np.zeros((H, v.shape[2]))
    for h in range(H):
        s = k[:, h // (H // G)] @ q[h] * scale
        if cap:
            s = cap * np.tanh(s / cap)
        e = np.exp(s - s.max())
        out[h] = (e / e.sum()) @ v[:, h // (H // G)]
    return out


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("Hq,G,D", [(4, 2, 64), (3, 1, 128), (2, 1, 48)])
@pytest.mark.parametrize("Sq", [1, 2, 16, 70, 200])
@pytest.mark.parametrize("window", [16, 100, 128, 129])
def test_a_key_that_stands_out_counts_exactly_inside_the_window(dt, Hq, G, D, Sq, window):
    """One key dominates every query that sees it (its value is 1, all others 0): the output of a row says whether it was seen.
    The key is put just inside and just outside the windows of the first and the last query row, at tile and ring borders."""
    rows, T = 384, 1000
    first, last = T - Sq, T - 1
    places = {first - window + 1, first - window, last - window + 1, last - window, first, last, 768, 767, 896, 895, 944, 943}
    t = DT[dt]
    q = torch.ones(1, Hq, Sq, D).to(t).cuda()
    for j in sorted(p for p in places if last - rows < p <= last and p >= 0):
        k, v = torch.zeros(1, G, rows, D), torch.zeros(1, G, rows, D)
        k[:, :, j % rows] = 1.0
        v[:, :, j % rows] = 1.0
        for plain in (False, True):
            got = host(ops.window_attention(q, k.to(t).cuda(), v.to(t).cuda(), 20.0 / D, T, window, 50.0, plain))[0]
            ops.attention_check()
            for r in range(Sq):
                sees = 0 <= first + r - j < window
                assert (got[r] > 0.99).all() if sees else (got[r] == 0.0).all(), (j, r, plain, got[r].min(), got[r].max())


# ---- routing and products ----
@pytest.mark.parametrize("M", [1, 3, 33, 65, 400])
@pytest.mark.parametrize("E,top,groups,keep", [(6, 2, 3, 2), (16, 4, 4, 1), (1, 1, 1, 1), (8, 8, 2, 2), (130, 5, 13, 3), (64, 1, 64, 2), (256, 8, 1, 1)])
def test_routing(M, E, top, groups, keep):
    rng = np.random.default_rng(M * E)
    z = cuda(rng.standard_normal((M, E)) * 2)
    r = ops.MoeRouting(z, top, groups, keep)
    rows, chosen, wts = r.rows().cpu().numpy(), r.chosen.cpu().numpy(), host(r.weights)
    for t in range(M):
        idx, s = R.route(host(z)[t], top, groups, keep)
        assert chosen[t].tolist() == list(idx)
        close(wts[t], s, 3e-6)
    order = np.empty(M * top, int)
    order[rows.reshape(-1)] = chosen.reshape(-1)  # a permutation, ordered by expert
    assert sorted(rows.reshape(-1).tolist()) == list(range(M * top)) and (np.diff(order) >= 0).all()


def test_routing_ties_go_to_the_lower_expert():
    z = torch.zeros(2, 40).cuda()
    assert ops.MoeRouting(z, 3).chosen.cpu().tolist() == [[0, 1, 2]] * 2
    assert ops.MoeRouting(z, 3, 10, 2).chosen.cpu().tolist() == [[0, 1, 2]] * 2


@pytest.mark.parametrize("dt", ["bf16", "f16", "f32"])
@pytest.mark.parametrize("M", [1, 5, 9, 31, 33, 64, 200])
@pytest.mark.parametrize("N,K", [(16, 40), (200, 72), (640, 256), (129, 1000), (4100, 64), (37, 51)])
def test_dense_matmul(dt, M, N, K):
    rng = np.random.default_rng(M + N)
    a = cuda(rng.standard_normal((M, K)), DT[dt])
    status = torch.zeros(1, dtype=torch.int32).cuda()
    for glu in (False, True):
        w = cuda(rng.standard_normal((2 * N if glu else N, K)) * K ** -0.5, DT[dt])
        want = host(a) @ host(w).T
        if glu:
            want = R.silu(want[:, :N]) * want[:, N:]
        for st in (None, status):
            close(host(ops.dense_matmul(a, w, glu, status=st)), want, TOL[dt] * 2, f"glu {glu}")
            close(host(ops.dense_matmul(a, w, glu, out_dtype=torch.float32, status=st)), want, 4e-6 if dt == "f32" else 3e-5, f"f32 out, glu {glu}")
    assert int(status.item()) == 0


@pytest.mark.parametrize("dt", ["bf16", "f32"])
@pytest.mark.parametrize("M,E,top,N,K,skew", [(1, 8, 2, 48, 64, 0), (3, 5, 3, 24, 40, 0), (30, 4, 2, 136, 72, 0), (70, 3, 1, 64, 128, 9), (300, 6, 2, 40, 96, 0),
                                              (300, 16, 1, 200, 64, 9), (150, 2, 2, 130, 200, 0), (37, 2, 2, 48, 50, 0)])
def test_expert_products(dt, M, E, top, N, K, skew):
    """Gate/up with gating over gathered rows, then down over the routed rows; ``skew`` sends most tokens to expert 1."""
    rng = np.random.default_rng(M)
    z = rng.standard_normal((M, E))
    z[: M - 2, 1] += skew
    h = cuda(rng.standard_normal((M, K)), DT[dt])
    gu, dn = cuda(rng.standard_normal((E, 2 * N, K)) * K ** -0.5, DT[dt]), cuda(rng.standard_normal((E, K, N)) * N ** -0.5, DT[dt])
    r = ops.MoeRouting(cuda(z), top)
    rows, chosen = r.rows().cpu().numpy(), r.chosen.cpu().numpy()
    for tc in (True, False):
        hid = r.matmul(h, gu, gather=True, glu=True, tensor_core=tc)
        out = r.matmul(hid, dn, gather=False, out_dtype=torch.float32, tensor_core=tc)
        assert not tc or int(r.status.item()) == 0
        want_h, want_o = np.zeros((M * top, N)), np.zeros((M * top, K))
        for t in range(M):
            for s in range(top):
                e, p = chosen[t, s], rows[t, s]
                g = host(gu[e]) @ host(h[t])
                want_h[p] = R.silu(g[:N]) * g[N:]
                want_o[p] = host(dn[e]) @ host(hid[p])
        close(host(hid), want_h, TOL[dt] * 2, "hidden")
        close(host(out), want_o, 4e-6 if dt == "f32" else 3e-5, "down")
