"""The operators that Fekopel added to the CUDA layer, each alone against the plain float64 functions of tests/fekopel_plain.py: the
residual pass with a layer norm (residual.cu), norms per head in front of the cache, the sink and the element gate behind a window's
soft-max (window_attention.cu), the grouped soft-max router with more rows, gelu experts and the shared expert beside them
(moe.cu, dense.cu, prefill.cu).  Windows get one key made to stand out just inside and just outside every edge, at page borders and
at the kept first positions, in portions and in single-token steps."""
import numpy as np
import pytest

import fekopel_fixture as F
import fekopel_plain as FP
from device_util import BF16, F32, as_dt, at, dev, f32, from_dt, i32, ptr, release, size_of, zeros

pytestmark = pytest.mark.gpu


@pytest.fixture(autouse=True)
def _release_buffers():
    yield
    release()


# ------------------------------------------------------------------------------------------------ the residual pass
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("W,T", [(7, 3), (40, 41), (130, 70), (516, 5), (1024, 2), (2052, 66), (4096, 1), (4100, 3)])
def test_residual_pass_adds_what_waits_and_takes_the_layer_norm(gpu, dt, W, T):
    r = np.random.default_rng(W)
    V, eps = 19, 1e-5
    lib, es = gpu.cuda_lib(), size_of(dt)
    (tv, tu), ids = as_dt(dt, r.standard_normal((V, W))), r.integers(0, V, T)
    x, y, add, nw, nb = r.standard_normal((T, W)) + 3.0, r.standard_normal((T, W)), r.standard_normal(W), r.uniform(0.3, 1.5, W), r.standard_normal(W)
    table, di, dy, da, dnw, dnb = dev(gpu, tu), dev(gpu, i32(ids)), dev(gpu, f32(y)), dev(gpu, f32(add)), dev(gpu, f32(nw)), dev(gpu, f32(nb))
    rows = np.arange(T)[::-2].copy()

    def run(x_in, with_y, emb, with_add, pick):
        dx = dev(gpu, f32(x)) if x_in else None
        n = len(rows) if pick else T
        xo = zeros(gpu, n * W * 4) if pick or not x_in else dx   # in place where it may be
        h = zeros(gpu, n * W * es)
        gpu.check(lib.ggb_op_residual_layer_norm(dt, ptr(dx), dy.ptr if with_y else None, None, None, None, 0, 0, 0, None, None, 0, table.ptr if emb else None, di.ptr,
                                                 da.ptr if with_add else None, dnw.ptr, dnb.ptr, eps, W, n, dev(gpu, i32(rows)).ptr if pick else None, xo.ptr, h.ptr), "residual")
        want = (x if x_in else 0) + (y if with_y else 0) + (tv[ids] if emb else 0) + (add if with_add else 0)
        want = want[rows] if pick else want
        assert F.rel_err(xo.download(np.float32, n * W).reshape(n, W), want) < 1e-6
        assert F.rel_err(from_dt(dt, h, (n, W)), FP.layer_norm(want, nw, nb, eps)) < (5e-3 if dt == BF16 else 2e-6)
    run(False, False, True, False, False)   # the first layer
    run(False, False, True, True, False)    # a looped block that starts there
    run(True, True, False, False, False)    # between two sublayers
    run(True, True, True, True, False)      # a later pass begins
    run(True, False, False, True, False)
    run(True, True, False, False, True)     # a few rows at the end, backwards


def test_layer_norm_does_not_cancel_on_a_large_mean(gpu):
    W, T = 512, 4
    x = np.random.default_rng(0).standard_normal((T, W)) * 0.5 + 1000.0
    x = f32(x).astype(np.float64)
    h = zeros(gpu, T * W * 4)
    gpu.check(gpu.cuda_lib().ggb_op_residual_layer_norm(F32, dev(gpu, f32(x)).ptr, None, None, None, None, 0, 0, 0, None, None, 0, None, None, None, dev(gpu, f32(np.ones(W))).ptr,
                                                        dev(gpu, f32(np.zeros(W))).ptr, 1e-6, W, T, None, None, h.ptr), "residual")
    assert F.rel_err(from_dt(F32, h, (T, W)), FP.layer_norm(x, 1.0, 0.0, 1e-6)) < 3e-4  # the mean itself is rounded to 6e-5


def test_residual_pass_refuses_what_it_cannot_do(gpu):
    lib, b = gpu.cuda_lib(), zeros(gpu, 4096)
    tail = (b.ptr, b.ptr, 1e-5, 8, 2)
    for args in ((None, None, None, None, None, 0, 0, 0, None, None, 0, None, None, None) + tail + (None, b.ptr, None),          # nothing to start from
                 (b.ptr, None, b.ptr, b.ptr, b.ptr, 2, 65, 70, None, None, 0, None, None, None) + tail + (None, b.ptr, None),   # too many slots
                 (b.ptr, b.ptr, b.ptr, b.ptr, b.ptr, 2, 2, 4, None, None, 0, None, None, None) + tail + (None, b.ptr, None),    # two outputs at once
                 (b.ptr, None, None, None, None, 0, 0, 0, None, None, 0, None, None, None) + tail + (b.ptr, b.ptr, None)):      # chosen rows in place
        assert lib.ggb_op_residual_layer_norm(F32, *args) != 0


# ------------------------------------------------------------------------------------------------ attention
def cos_sin(rot, n):
    d = rot["dims"]
    a = np.arange(n)[:, None] * (rot["base"] ** (-2.0 * np.arange(d // 2) / d))[None, :]
    return f32(np.stack([np.cos(a), np.sin(a)], -1))


def run_attn(gpu, dt, q, k, v, H, G, D, cuts, page, window=0, keep=0, scale=1.0, cap=0.0, eps=1e-5, qn=None, kn=None, rot=None, sink=None, gate=None, seed=0, scratch=True):
    """feeds rows in portions through head_qkv_store + masked_attn_gated over shuffled pages; returns [T, H Dv]"""
    T, Dv = q.shape[0], v.shape[1] // G
    lib, es = gpu.cuda_lib(), size_of(dt)
    ld = int(lib.ggb_window_cache_ld(G, D, Dv))
    n_pages = (T + page - 1) // page + 3
    tb = dev(gpu, np.random.default_rng(seed).permutation(n_pages).astype(np.int32))
    cache = zeros(gpu, n_pages * page * ld * es)
    cs = dev(gpu, cos_sin(rot, T + 1)) if rot else None
    dqn, dkn, dsink = (dev(gpu, f32(a)) if a is not None else None for a in (qn, kn, sink))
    rows = f32(np.concatenate([q, k, v] + ([gate] if gate is not None else []), 1))
    nq, nk, nv, ldr = q.shape[1], k.shape[1], v.shape[1], rows.shape[1]
    ws = zeros(gpu, lib.ggb_window_attn_scratch_bytes(H)) if scratch else None
    lo, got = 0, []
    for c in cuts:
        xr, qo, out, pos0 = dev(gpu, rows[lo:lo + c]), zeros(gpu, c * nq * 4), zeros(gpu, c * H * Dv * es), dev(gpu, i32([lo]))
        gpu.check(lib.ggb_op_head_qkv_store(dt, xr.ptr, at(xr, 4 * nq), at(xr, 4 * (nq + nk)), ldr, c, H, G, D, Dv, ptr(dqn), ptr(dkn), eps, rot["dims"] if rot else 0, 1, ptr(cs), scale,
                                            pos0.ptr, tb.ptr, page, cache.ptr, qo.ptr), "head_qkv_store")
        gpu.check(lib.ggb_op_masked_attn_gated(dt, qo.ptr, cache.ptr, tb.ptr, page, pos0.ptr, c, H, G, D, Dv, window, keep, cap, ptr(dsink),
                                               at(xr, 4 * (nq + nk + nv)) if gate is not None else None, ldr, out.ptr, ptr(ws)), "masked_attn_gated")
        got.append(from_dt(dt, out, (c, H * Dv)))
        lo += c
    assert lo == T
    return np.concatenate(got)


def attn_want(q, k, v, H, G, D, window=0, keep=0, scale=1.0, cap=0.0, eps=1e-5, qn=None, kn=None, rot=None, sink=None, gate=None):
    T, Dv = q.shape[0], v.shape[1] // G
    one = np.ones(D)
    qq = FP.rotate_halves(FP.rms_unit(q.reshape(T, H, D), eps) * (one if qn is None else qn), np.arange(T), rot)
    kk = FP.rotate_halves(FP.rms_unit(k.reshape(T, G, D), eps) * (one if kn is None else kn), np.arange(T), rot)
    o = FP.attention_core(qq, kk, v.reshape(T, G, Dv), scale, FP.visible(T, window, keep), cap, sink).reshape(T, H * Dv)
    return o * FP.sigmoid(gate) if gate is not None else o


SHAPES = [(4, 2, 8, 6, 11, 3, 8, 4, 2.0), (3, 3, 16, 16, 64, 0, 16, 16, 0.0), (6, 1, 7, 34, 5, 9, 7, 2, 1.5), (2, 2, 64, 128, 33, 40, 64, 32, 30.0), (5, 5, 24, 10, 0, 0, 16, 0, 0.7),
          (1, 1, 1, 2, 1, 1, 4, 0, 0.0), (8, 2, 32, 256, 300, 33, 16, 8, 0.0), (4, 2, 40, 70, 1, 64, 32, 8, 3.0), (2, 1, 96, 96, 150, 2, 16, 96, 0.0)]


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,Gk,D,Dv,window,keep,page,dims,cap", SHAPES)
def test_norms_per_head_sink_and_gate_in_portions_and_single_tokens(gpu, dt, H, Gk, D, Dv, window, keep, page, dims, cap):
    G = Gk
    r = np.random.default_rng(H * 100 + D)
    T = 150
    q, k, v, gate = (r.standard_normal((T, n)) * s for n, s in ((H * D, 3.0), (G * D, 0.2), (G * Dv, 1.0), (H * Dv, 1.5)))
    qn, kn, sink = r.uniform(0.4, 1.6, D), r.uniform(0.4, 1.6, D), 2.0 * r.standard_normal(H)
    rot = {"dims": dims, "base": 40.0} if dims else None
    forms = (dict(window=window, keep=keep, scale=0.8 / np.sqrt(D) ** 0.5, cap=cap, qn=qn, kn=kn, rot=rot, gate=gate),
             dict(window=window, scale=1.7 / np.sqrt(D) ** 0.5, sink=sink), dict(window=window, keep=keep, cap=cap, rot=rot, sink=np.zeros(H), gate=gate, kn=kn, eps=0.3))
    for form in forms:
        want = attn_want(q, k, v, H, G, D, **form)
        for cuts in ([T], [40] + [1] * 30 + [2, 3, 33, 42], [1] * 20 + [130]):
            got = run_attn(gpu, dt, q, k, v, H, G, D, cuts, page, scratch=len(cuts) != 21, **form)
            assert F.rel_err(got, want) < (2e-2 if dt == BF16 else 1e-5), (sorted(form), cuts[:3])


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("steps", ["portion", "single"])
@pytest.mark.parametrize("with_sink", [False, True])
def test_window_edges_and_kept_positions_with_one_key_standing_out(gpu, dt, steps, with_sink):
    """Query i points at key j alone: seen, that key takes the head over; unseen, nothing of its value.  j walks over the last place
    inside the window and the first one outside, the last kept position and the next one, page borders, position 0 and the token itself."""
    H, G, D, Dv, page = 2, 1, 8, 6, 16
    T = 200
    r = np.random.default_rng(9)
    cases = ((32, 4, 199, 168), (32, 4, 199, 167), (32, 4, 199, 3), (32, 4, 199, 4), (17, 16, 67, 15), (17, 16, 67, 16), (17, 16, 33, 16), (17, 0, 67, 51), (17, 0, 67, 50), (17, 0, 17, 0),
             (17, 0, 16, 0), (17, 1, 40, 0), (17, 40, 199, 39), (17, 40, 199, 40), (17, 33, 150, 32), (17, 33, 150, 33), (0, 0, 199, 0), (1, 2, 77, 77), (1, 2, 77, 76), (1, 2, 77, 1), (200, 5, 199, 0))
    for window, keep, i, j in cases:
        # heads are unit after their norm, so all other keys are made to point away from the query
        u = r.standard_normal(D)
        u /= np.linalg.norm(u)
        away = r.standard_normal((T, 1, D))
        away -= (away @ u)[..., None] * u
        q, k, v = r.standard_normal((T, H * D)), away.reshape(T, G * D).copy(), r.standard_normal((T, G * Dv))
        q[i, :D] = 3.0 * u   # head 0 of token i
        k[j] = 5.0 * u
        form = dict(window=window, keep=keep, scale=1.5, sink=np.zeros(H) if with_sink else None)
        want = attn_want(q, k, v, H, G, D, **form)
        k2 = k.copy()
        k2[j] = away[j, 0]
        moved = np.abs(attn_want(q, k2, v, H, G, D, **form)[i, :Dv] - want[i, :Dv]).max()
        visible = j <= i and (window == 0 or i - j < window or j < keep)
        only = not with_sink and window == 1 and j == i and keep == 0
        assert (moved > 3e-2) == (visible and not only), (window, keep, i, j, moved)  # the oracle itself tells inside from outside
        cuts = [T] if steps == "portion" else [i - 3] + [1] * (T - i + 3)
        got = run_attn(gpu, dt, q, k, v, H, G, D, cuts, page, seed=i, **form)
        assert np.abs(got[i] - want[i]).max() < (3e-2 if dt == BF16 else 2e-5), (window, keep, i, j)
        assert F.rel_err(got, want) < (2e-2 if dt == BF16 else 1e-5), (window, keep, i, j)


@pytest.mark.parametrize("T", [9, 70])
def test_the_sink_takes_its_share_whatever_the_scores_are(gpu, T):
    """Equal scores s of n visible keys leave n e^s / (n e^s + e^sink) of the mean value: for the first token, full windows, and scores and
    sinks of +-60 whose exponentials alone would leave fp32."""
    H, G, D, Dv, window = 2, 2, 4, 2, 6
    v = np.random.default_rng(T).standard_normal((T, G * Dv))
    one = np.ones((T, H * D))
    for s in (0.0, -60.0, 60.0, 2.0):
        for sink in (0.0, 55.0, -120.0):
            got = run_attn(gpu, F32, one, np.sign(s if s else 1.0) * one, v, H, G, D, [T], 4, window=window, scale=abs(s) / D, eps=0.0, sink=np.full(H, sink))
            n = np.minimum(np.arange(T) + 1, window)
            mean = np.stack([v[max(0, i - window + 1):i + 1].mean(0) for i in range(T)])
            share = n / (n + np.exp(np.clip(sink - s, -300, 300)))
            assert np.abs(got - mean * share[:, None]).max() < 2e-5, (s, sink)


def test_heads_are_normed_one_by_one_and_an_all_zero_head_stays_zero(gpu):
    """Scaling one head of q or k changes nothing (eps aside); with eps a head of zeros scores zero against everything."""
    H, G, D, Dv, T = 4, 2, 6, 4, 40
    r = np.random.default_rng(3)
    q, k, v = (r.standard_normal((T, n)) for n in (H * D, G * D, G * Dv))
    base = run_attn(gpu, F32, q, k, v, H, G, D, [T], 8, eps=1e-12)
    q2, k2 = q.copy(), k.copy()
    q2[:, D:2 * D] *= 50.0
    k2[:, :D] *= 0.01
    assert F.rel_err(run_attn(gpu, F32, q2, k2, v, H, G, D, [T], 8, eps=1e-12), base) < 1e-5
    q2[:, :D] = 0.0
    got = run_attn(gpu, F32, q2, k2, v, H, G, D, [T], 8, eps=1e-5)
    assert F.rel_err(got[:, :Dv], np.cumsum(v[:, :Dv], 0) / (np.arange(T) + 1)[:, None]) < 1e-5


# ------------------------------------------------------------------------------------------------ products with gelu
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("T,N,K", [(1, 24, 40), (3, 17, 33), (8, 64, 128), (9, 24, 40), (70, 96, 64), (64, 32, 64), (300, 544, 320), (200, 64, 1024)])
def test_a_product_with_its_activation_in_every_form(gpu, dt, T, N, K):
    """mat-vec, tile kernel, tensor cores (a whole tile and past its edge), and tensor cores with the product split along K"""
    r = np.random.default_rng(T + N)
    (w, wu), (a, au) = as_dt(dt, 2 * r.standard_normal((N, K)) / np.sqrt(K)), as_dt(dt, r.standard_normal((T, K)))
    y = zeros(gpu, T * N * size_of(dt))
    dw, da = dev(gpu, wu), dev(gpu, au)
    z = a @ w.T
    for act, want in ((1, np.maximum(z, 0) ** 2), (4, FP.gelu_erf(z))):
        gpu.check(gpu.cuda_lib().ggb_op_linear_act(dt, dw.ptr, N, K, da.ptr, K, T, act, y.ptr), "linear_act")
        assert F.rel_err(from_dt(dt, y, (T, N)), want) < (6e-3 if dt == BF16 else 3e-6), act
    assert gpu.cuda_lib().ggb_op_linear_act(dt, dw.ptr, N, K, da.ptr, K, T, 2, y.ptr) != 0


def test_gelu_is_the_exact_one_on_both_sides_and_far_out(gpu):
    z = np.concatenate([np.linspace(-9, 9, 400), [0.0, -0.0, 1e-6, -1e-6, 80.0, -80.0]])
    y = zeros(gpu, z.size * 4)
    gpu.check(gpu.cuda_lib().ggb_op_act_rows(F32, dev(gpu, f32(z)).ptr, z.size, 1, z.size, 4, y.ptr), "act_rows")
    assert np.abs(from_dt(F32, y, z.shape) - FP.gelu_erf(z)).max() < 2e-6
    tanh_form = 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))
    assert np.abs(from_dt(F32, y, z.shape) - tanh_form).max() > 1e-4  # the other gelu is told apart


# ------------------------------------------------------------------------------------------------ router, experts, shared expert
def run_moe(gpu, dt, h, W, p, f, x):
    """router -> groups -> up with gelu -> down, the shared expert beside them -> the weighted sum inside the residual pass, as the
    model calls them; returns what came out and what the oracle gives for the matrices' rounded values"""
    lib, es = gpu.cuda_lib(), size_of(dt)
    T, Wd = h.shape
    r, g, sh = f["router"], f["router"].get("groups") or {"count": 1, "keep": 1}, f.get("shared")
    E, top, FF, extra = r["experts"], r["top"], f["expert"]["ff"], 1 if sh else 0
    hv, hu = as_dt(dt, h)
    Wq, up, dn = dict(W), [], []
    for e in range(E):
        for n, dst in (("up", up), ("down", dn)):
            Wq[p + "e%d.%s" % (e, n)], code = as_dt(dt, W[p + "e%d.%s" % (e, n)])
            dst.append(code.reshape(W[p + "e%d.%s" % (e, n)].shape))
            Wq[p + "e%d.%s" % (e, n)] = Wq[p + "e%d.%s" % (e, n)].reshape(dst[-1].shape)
    rt = W[p + "router"]
    n = T * top
    hd, upd, dnd = dev(gpu, hu), dev(gpu, np.concatenate(up)), dev(gpu, np.concatenate(dn))
    z, idx, wt = zeros(gpu, T * (E + extra) * 4), zeros(gpu, n * 4), zeros(gpu, n * 4)
    ws = zeros(gpu, int(lib.ggb_moe_group_ints(n, E)) * 4)
    act, y2, ys, x2, hn = zeros(gpu, n * FF * es), zeros(gpu, n * Wd * 4), None, dev(gpu, f32(x)), zeros(gpu, T * Wd * es)
    if sh:
        FS = sh["ff"]
        (Wq[p + "shared.up"], su), (Wq[p + "shared.down"], sd) = as_dt(dt, W[p + "shared.up"]), as_dt(dt, W[p + "shared.down"])
        rt = np.concatenate([rt, W[p + "shared.sg"]])
        sud, sdd, acts, ys = dev(gpu, su), dev(gpu, sd), zeros(gpu, T * FS * es), zeros(gpu, T * Wd * 4)
    gpu.check(lib.ggb_op_moe_route_softmax_groups(dt, hd.ptr, Wd, T, dev(gpu, f32(rt)).ptr, None, E, extra, top, g["count"], g["keep"], r.get("scale", 1.0), z.ptr, idx.ptr, wt.ptr,
                                                  ws.ptr), "route")
    if not lib.ggb_moe_step_form(n):
        gpu.check(lib.ggb_op_moe_group(idx.ptr, T, top, E, ws.ptr), "group")
    if sh:
        gpu.check(lib.ggb_op_moe_linear_shared(dt, upd.ptr, FF, Wd, hd.ptr, Wd, 1, T, top, E, ws.ptr, 4, act.ptr, FF, sud.ptr, FS, Wd, hd.ptr, Wd, acts.ptr), "up")
        gpu.check(lib.ggb_op_moe_linear_shared(dt, dnd.ptr, Wd, FF, act.ptr, FF, 0, T, top, E, ws.ptr, 0, y2.ptr, Wd, sdd.ptr, Wd, FS, acts.ptr, FS, ys.ptr), "down")
    else:
        gpu.check(lib.ggb_op_moe_linear(dt, upd.ptr, FF, Wd, hd.ptr, Wd, 1, T, top, E, ws.ptr, 4, act.ptr, FF), "up")
        gpu.check(lib.ggb_op_moe_linear(dt, dnd.ptr, Wd, FF, act.ptr, FF, 0, T, top, E, ws.ptr, 0, y2.ptr, Wd), "down")
    gpu.check(lib.ggb_op_residual_layer_norm(dt, x2.ptr, None, y2.ptr, ws.ptr, wt.ptr, T, top, E, ptr(ys), at(z, 4 * E) if sh else None, E + extra, None, None, None,
                                             dev(gpu, f32(np.ones(Wd))).ptr, dev(gpu, f32(np.zeros(Wd))).ptr, 1e-5, Wd, T, None, x2.ptr, hn.ptr), "residual")
    xo = x2.download(np.float32, T * Wd).reshape(T, Wd).astype(np.float64)
    return xo, from_dt(dt, hn, (T, Wd)), idx.download(np.int32, n).reshape(T, top), wt.download(np.float32, n).reshape(T, top), hv, Wq


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("E,top,FF,groups,keep,scale,shared,Wd,T", [
    (6, 2, 9, 3, 2, 1.7, 14, 38, 4), (6, 2, 9, 3, 2, 1.7, 14, 38, 70), (1, 1, 5, 1, 1, 0.5, 1, 22, 3), (8, 4, 16, 4, 2, 2.5, 24, 32, 1), (8, 4, 16, 8, 4, 1.0, 0, 33, 40),
    (64, 6, 32, 8, 3, 2.0, 40, 64, 33), (12, 3, 64, 2, 1, 3.0, 128, 128, 300), (40, 4, 8, 0, 0, 1.0, 96, 24, 2), (5, 5, 8, 5, 5, 1.0, 8, 40, 200)])
def test_router_experts_and_the_shared_expert(gpu, dt, E, top, FF, groups, keep, scale, shared, Wd, T):
    r = np.random.default_rng(E * 10 + T)
    f = F.moe(experts=E, top=top, ff=FF, groups=groups, keep=keep, scale=scale, shared=shared)
    W = FP.random_weights(F.config([F.attn(mlp=f)], width=Wd), seed=T)
    h, x = r.standard_normal((T, Wd)), r.standard_normal((T, Wd))
    xo, hn, idx, wt, hv, Wq = run_moe(gpu, dt, h, W, "l0.mlp.", f, x)
    for n in ("router", "shared.sg"):
        if "l0.mlp." + n in Wq:
            Wq["l0.mlp." + n] = f32(Wq["l0.mlp." + n]).astype(np.float64)
    widx, wwt = FP.route(hv, Wq["l0.mlp.router"], top, max(groups, 1), keep or 1, scale)
    same = (idx == widx).all(-1)
    assert same.mean() > 0.95  # a close call of two scores may fall the other way in fp32
    assert np.abs(wt[same] - wwt[same]).max() < 1e-5 * scale and np.abs(wt.sum(-1) - scale).max() < 1e-5 * scale
    want = FP.moe_ff(hv, Wq, "l0.mlp.", f)
    assert F.rel_err((xo - x)[same], want[same]) < (1.5e-2 if dt == BF16 else 1e-5)
    assert F.rel_err(hn, FP.layer_norm(xo, 1.0, 0.0, 1e-5)) < (5e-3 if dt == BF16 else 5e-6)


@pytest.mark.parametrize("T", [1, 40])
def test_a_hidden_group_keeps_its_best_expert_out_and_a_group_counts_by_its_largest(gpu, T):
    """Scores 0.40, 0.02 | 0.30, 0.28: with one group kept the choice is {0, 1}, although 2 and 3 score more than 1 and more together."""
    Wd = 4
    W = FP.random_weights(F.config([F.attn(mlp=F.moe(experts=4, top=2, groups=2, keep=1, shared=3))], width=Wd), seed=1)
    W["l0.mlp.router"] = np.log(np.array([0.40, 0.02, 0.30, 0.28]))[:, None] * np.eye(Wd)[0]
    h = np.zeros((T, Wd))
    h[:, 0] = 1.0
    x = np.zeros((T, Wd))
    for groups, keep, want in ((2, 1, [0, 1]), (2, 2, [0, 2]), (0, 0, [0, 2]), (4, 1, None), (4, 3, [0, 2])):
        f = F.moe(experts=4, top=1 if want is None else 2, groups=groups, keep=keep, scale=2.0, shared=3)
        xo, _, idx, wt, hv, Wq = run_moe(gpu, F32, h, W, "l0.mlp.", f, x)
        want = want or [0]
        s = np.array([0.40, 0.02, 0.30, 0.28])[want]
        assert (idx == want).all() and np.abs(wt - 2.0 * s / s.sum()).max() < 1e-5
        assert F.rel_err(xo, FP.moe_ff(hv, Wq, "l0.mlp.", f)) < 1e-5


@pytest.mark.parametrize("T", [2, 50])
def test_the_shared_gate_opens_and_closes_per_token(gpu, T):
    """A gate row that reads the first coordinate: tokens with +30 add the shared expert whole, tokens with -30 nothing of it."""
    Wd = 12
    f = F.moe(experts=3, top=1, groups=0, shared=7)
    W = FP.random_weights(F.config([F.attn(mlp=f)], width=Wd), seed=5)
    W["l0.mlp.shared.sg"] = 30.0 * np.eye(Wd)[:1]
    h = np.random.default_rng(0).standard_normal((T, Wd))
    h[:, 0] = np.where(np.arange(T) % 2 == 0, 1.0, -1.0)
    x = np.zeros((T, Wd))
    xo, _, _, _, hv, Wq = run_moe(gpu, F32, h, W, "l0.mlp.", f, x)
    Wn = {k: (0 * v if ".shared.down" in k else v) for k, v in Wq.items()}
    with_s, without = FP.moe_ff(hv, Wq, "l0.mlp.", f), FP.moe_ff(hv, Wn, "l0.mlp.", f)
    assert F.rel_err(xo, with_s) < 1e-5 and np.abs(xo - without)[1::2].max() < 1e-5 and np.abs(xo - without)[::2].max() > 0.1


def test_logits_that_are_no_numbers_choose_experts_that_exist(gpu):
    lib, Wd, E, top = gpu.cuda_lib(), 8, 6, 3
    for T in (2, 40):
        h = dev(gpu, f32(np.full((T, Wd), np.nan)))
        z, idx, wt = zeros(gpu, T * E * 4), zeros(gpu, T * top * 4), zeros(gpu, T * top * 4)
        rt = dev(gpu, f32(np.ones((E, Wd))))
        gpu.check(lib.ggb_op_moe_route_softmax_groups(F32, h.ptr, Wd, T, rt.ptr, None, E, 0, top, 3, 2, 1.0, z.ptr, idx.ptr, wt.ptr, None), "route")
        got = idx.download(np.int32, T * top)
        assert (got >= 0).all() and (got < E).all()
