"""The operators that Tezesun added to the CUDA layer, each alone against the plain float64 functions of tests/tezesun_plain.py:
the pass between two layers with its token shift, two products in one launch, xIELU (dense.cu), differential attention over a window
that keeps the first positions (window_attention.cu), the halves layout and both forms of the latent attention
(latent_attention.cu), and the gated diagonal recurrence in its step and portion forms (rglru.cu).  Operators with a state are fed
in portions that continue from what they left; windows get one key made to stand out just inside and just outside every edge, at
page borders and at the kept first positions, in portions and in single-token steps."""
import numpy as np
import pytest

import tezesun_fixture as F
import tezesun_plain as TP

pytestmark = pytest.mark.gpu
BF16, F32 = 30, 0
_ALIVE = []


@pytest.fixture(autouse=True)
def _release_buffers():
    yield
    _ALIVE.clear()


def dev(G, a):
    _ALIVE.append(G.DeviceBuffer.from_numpy(np.ascontiguousarray(a)))
    return _ALIVE[-1]


def zeros(G, nbytes):
    b = G.DeviceBuffer(max(int(nbytes), 16))
    b.zero()
    _ALIVE.append(b)
    return b


def f32(a):
    return np.ascontiguousarray(a, dtype=np.float32)


def i32(a):
    return np.ascontiguousarray(a, dtype=np.int32)


def as_dt(dt, a):
    """(values as float64 after rounding into dt, the array to upload)"""
    if dt == BF16:
        return F.bf16_round(a)
    a32 = f32(a)
    return a32.astype(np.float64), a32


def from_dt(dt, buf, shape):
    n = int(np.prod(shape))
    if dt == BF16:
        return (buf.download(np.uint16, n).astype(np.uint32) << 16).view(np.float32).reshape(shape).astype(np.float64)
    return buf.download(np.float32, n).reshape(shape).astype(np.float64)


def ptr(b):
    return b.ptr if b is not None else None


def at(buf, byte_offset):
    return buf.ptr.value + byte_offset


def cos_sin(rot, n):
    f, mag = TP.rot_frequencies(rot)
    a = np.arange(n)[:, None] * f[None, :]
    return f32(mag * np.stack([np.cos(a), np.sin(a)], -1))


# ------------------------------------------------------------------------------------------------ between two layers
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("W", [7, 40, 516, 2048])
def test_layer_pass_enters_both_outputs_norms_and_shifts_across_portions(gpu, dt, W):
    r = np.random.default_rng(W)
    T, V, eps = 41, 19, 1e-5
    lib = gpu.cuda_lib()
    es = 2 if dt == BF16 else 4
    (tv, tu), ids = as_dt(dt, r.standard_normal((V, W))), r.integers(0, V, T)
    a, b = r.standard_normal((T, W)), r.standard_normal((T, W))
    l1, l2, n1, n2, mu1, mu2 = (r.uniform(0.2, 1.2, W) for _ in range(6))
    prev1, prev2 = zeros(gpu, W * 4), zeros(gpu, W * 4)
    table, dl1, dl2, dn1, dn2, dm1, dm2 = [dev(gpu, tu)] + [dev(gpu, f32(v)) for v in (l1, l2, n1, n2, mu1, mu2)]
    x0 = tv[ids]
    h0 = TP.rms_norm(x0, n1, eps)
    x1 = x0 + a * l1 + b * l2
    h1 = TP.rms_norm(x1, n2, eps)
    want = [x0, h0, TP.token_shift(h0, mu1), x1, h1, TP.token_shift(h1, mu2), TP.rms_norm(x0 + a * l1, n2, eps)]
    got = [[] for _ in want]
    lo = 0
    for c in (1, 2, 1, 30, 1, 6):
        di, da, db = dev(gpu, i32(ids[lo:lo + c])), dev(gpu, f32(a[lo:lo + c])), dev(gpu, f32(b[lo:lo + c]))
        xa, xb = zeros(gpu, c * W * 4), zeros(gpu, c * W * 4)
        h, hs, h2, hs2, hr = (zeros(gpu, c * W * es) for _ in range(5))
        # the first layer starts the residual from the embedding rows
        gpu.check(lib.ggb_op_shift_norm(dt, None, table.ptr, di.ptr, None, None, None, None, dn1.ptr, eps, dm1.ptr, prev1.ptr, W, c, None, xa.ptr, h.ptr, hs.ptr), "shift_norm")
        gpu.check(lib.ggb_op_shift_norm(dt, xa.ptr, None, None, da.ptr, dl1.ptr, db.ptr, dl2.ptr, dn2.ptr, eps, dm2.ptr, prev2.ptr, W, c, None, xb.ptr, h2.ptr, hs2.ptr), "shift_norm")
        # a few rows at the end, here all of them backwards; a layer without a feed-forward has one output
        rows = np.arange(c)[::-1]
        gpu.check(lib.ggb_op_shift_norm(dt, xa.ptr, None, None, da.ptr, dl1.ptr, None, None, dn2.ptr, eps, None, None, W, c, dev(gpu, i32(rows)).ptr, None, hr.ptr, None), "shift_norm")
        for k, v in enumerate((xa.download(np.float32, c * W).reshape(c, W), from_dt(dt, h, (c, W)), from_dt(dt, hs, (c, W)), xb.download(np.float32, c * W).reshape(c, W),
                               from_dt(dt, h2, (c, W)), from_dt(dt, hs2, (c, W)), from_dt(dt, hr, (c, W))[::-1])):
            got[k].append(v)
        lo += c
    assert lo == T
    for k, w in enumerate(want):
        assert F.rel_err(np.concatenate(got[k]), w) < (5e-3 if dt == BF16 and k not in (0, 3) else 1e-6), k
    # the carried row keeps 32 bits whatever the type of what it is blended into
    assert F.rel_err(prev2.download(np.float32, W), h1[-1]) < 1e-6


def test_layer_pass_of_many_tokens_takes_several_rows_per_cta(gpu):
    r = np.random.default_rng(1)
    T, W = 2500, 12
    x, mu, nw = r.standard_normal((T, W)), r.uniform(0, 1, W), np.ones(W)
    h, hs, prev = zeros(gpu, T * W * 4), zeros(gpu, T * W * 4), dev(gpu, f32(np.full(W, 0.5)))
    gpu.check(gpu.cuda_lib().ggb_op_shift_norm(F32, dev(gpu, f32(x)).ptr, None, None, None, None, None, None, dev(gpu, f32(nw)).ptr, 1e-6, dev(gpu, f32(mu)).ptr, prev.ptr, W, T, None,
                                               None, h.ptr, hs.ptr), "shift_norm")
    hw = TP.rms_unit(x, 1e-6)
    before = np.concatenate([np.full((1, W), 0.5), hw[:-1]])
    assert F.rel_err(from_dt(F32, h, (T, W)), hw) < 1e-6 and F.rel_err(from_dt(F32, hs, (T, W)), hw + (before - hw) * mu) < 1e-6
    assert F.rel_err(prev.download(np.float32, W), hw[-1]) < 1e-6


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("T,N1,K1,N2,K2", [(1, 24, 40, 9, 16), (3, 17, 33, 64, 128), (8, 64, 128, 5, 7), (9, 24, 40, 30, 24), (70, 64, 128, 96, 64)])
def test_two_products_with_and_without_the_activation(gpu, dt, T, N1, K1, N2, K2):
    r = np.random.default_rng(T + N1)
    (w1, u1), (a1, v1), (w2, u2), (a2, v2) = (as_dt(dt, r.standard_normal(s) / np.sqrt(s[1]) ** (i % 2 == 0)) for i, s in enumerate(((N1, K1), (T, K1), (N2, K2), (T, K2))))
    p, q = 0.4, -0.7
    ap, an = float(TP.softplus(p)), float(0.5 + TP.softplus(q))
    lib = gpu.cuda_lib()
    dw = [dev(gpu, u) for u in (u1, v1, u2, v2)]
    for act in (False, True):
        c1, c2, y1 = zeros(gpu, T * N1 * 4), zeros(gpu, T * N2 * 4), zeros(gpu, T * N1 * 4)
        gpu.check(lib.ggb_op_linear_pair(dt, dw[0].ptr, N1, K1, dw[1].ptr, K1, dw[2].ptr, N2, K2, dw[3].ptr, K2, T, c1.ptr, N1, y1.ptr if act else None, ap, an, c2.ptr, N2), "linear_pair")
        z = a1 @ w1.T
        got = from_dt(dt, y1, (T, N1)) if act else c1.download(np.float32, T * N1).reshape(T, N1)
        assert F.rel_err(got, TP.xielu(z, p, q) if act else z) < (6e-3 if dt == BF16 else 3e-6)
        assert F.rel_err(c2.download(np.float32, T * N2).reshape(T, N2), a2 @ w2.T) < (6e-3 if dt == BF16 else 3e-6)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n", [5, 1024])
def test_xielu_on_both_sides_of_zero_and_far_out(gpu, dt, n):
    z = np.concatenate([[0.0, -0.0, 1e-6, -1e-6, -80.0], np.linspace(-9, 9, n - 5)])[:n]
    y = zeros(gpu, n * 4)
    for p, q in ((0.0, 0.0), (2.0, -3.0), (-1.5, 1.0)):
        gpu.check(gpu.cuda_lib().ggb_op_xielu_rows(dt, dev(gpu, f32(z)).ptr, n, float(TP.softplus(p)), float(0.5 + TP.softplus(q)), y.ptr), "xielu")
        want = TP.xielu(z, p, q)
        assert np.abs(from_dt(dt, y, (n,)) - want).max() <= (5e-3 if dt == BF16 else 2e-6) * max(1.0, np.abs(want).max())


# ------------------------------------------------------------------------------------------------ differential attention
def run_diff(gpu, dt, q, k, v, gate, H, G, D, window, keep, scale, cap, lam, diff, eps, rot, cuts, page, seed=0, scratch=True):
    """feeds rows in portions through diff_qkv_store + diff_attn over shuffled pages; returns [T, H Dv]"""
    T = q.shape[0]
    Dv = v.shape[1] // G
    lib = gpu.cuda_lib()
    ld = int(lib.ggb_window_cache_ld(G, 2 * D, Dv))
    n_pages = (T + page - 1) // page + 3
    es = 2 if dt == BF16 else 4
    tb = dev(gpu, np.random.default_rng(seed).permutation(n_pages).astype(np.int32))
    cache = zeros(gpu, n_pages * page * ld * es)
    ck = dev(gpu, cos_sin(rot, T + 1)) if rot else None
    rows = f32(np.concatenate([q, k, v] + ([gate] if gate is not None else []), 1))
    nq, nk, nv, ldr = q.shape[1], k.shape[1], v.shape[1], rows.shape[1]
    ws = zeros(gpu, lib.ggb_window_attn_scratch_bytes(2 * H)) if scratch else None
    lo, got = 0, []
    for c in cuts:
        xr, qo, out = dev(gpu, rows[lo:lo + c]), zeros(gpu, c * nq * 4), zeros(gpu, c * H * Dv * es)
        pos0 = dev(gpu, i32([lo]))
        gpu.check(lib.ggb_op_diff_qkv_store(dt, xr.ptr, at(xr, 4 * nq), at(xr, 4 * (nq + nk)), ldr, c, H, G, D, Dv, rot["dims"] if rot else 0, 0, ptr(ck), scale, pos0.ptr, tb.ptr, page,
                                            cache.ptr, qo.ptr), "diff_qkv_store")
        gpu.check(lib.ggb_op_diff_attn(dt, qo.ptr, cache.ptr, tb.ptr, page, pos0.ptr, c, H, G, D, Dv, window, keep, cap, lam, 1.0 - diff, eps,
                                       at(xr, 4 * (nq + nk + nv)) if gate is not None else None, ldr, out.ptr, ptr(ws)), "diff_attn")
        got.append(from_dt(dt, out, (c, H * Dv)))
        lo += c
    assert lo == T
    return np.concatenate(got)


def diff_want(q, k, v, gate, H, G, D, window, keep, scale, cap, lam, diff, eps, rot):
    T = q.shape[0]
    Dv = v.shape[1] // G
    pos = np.arange(T)
    qq = TP.rotate(q.reshape(T, 2 * H, D), pos, rot, False).reshape(T, H, 2, D)
    kk = TP.rotate(k.reshape(T, 2 * G, D), pos, rot, False).reshape(T, G, 2, D)
    o = TP.diff_core(qq, kk, v.reshape(T, G, Dv), scale, cap, TP.visible(T, window, keep), lam, diff, eps).reshape(T, H * Dv)
    return o * TP.sigmoid(gate) if gate is not None else o


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,Gk,D,Dv,window,keep,page,dims,cap", [(4, 2, 8, 6, 11, 3, 8, 4, 2.0), (3, 3, 16, 16, 64, 0, 16, 16, 0.0), (6, 1, 6, 34, 5, 9, 7, 2, 1.5), (2, 2, 64, 128, 33, 40, 64, 32, 30.0),
                                                                 (2, 1, 24, 10, 0, 0, 16, 0, 0.7), (1, 1, 10, 4, 1, 1, 4, 10, 0.0), (2, 1, 32, 256, 300, 33, 16, 8, 0.0), (4, 2, 8, 70, 1, 64, 32, 8, 3.0)])
def test_differential_attention_portions_and_single_tokens(gpu, dt, H, Gk, D, Dv, window, keep, page, dims, cap):
    G = Gk
    r = np.random.default_rng(H * 100 + D)
    T = 150
    q, k, v, gate = (r.standard_normal((T, n)) for n in (2 * H * D, 2 * G * D, G * Dv, H * Dv))
    rot = {"dims": dims, "base": 40.0, "scaling": {"factor": 5.0, "original": 40, "fast": 4.0, "slow": 0.5}} if dims else None
    lam, diff, eps = 0.45, 0.3, 1e-5
    for g in (gate, None):
        want = diff_want(q, k, v, g, H, G, D, window, keep, 0.4, cap, lam, diff, eps, rot)
        for cuts in ([T], [40] + [1] * 30 + [2, 3, 33, 42], [1] * 20 + [130]):
            got = run_diff(gpu, dt, q, k, v, g, H, G, D, window, keep, 0.4, cap, lam, diff, eps, rot, cuts, page, scratch=len(cuts) != 21)
            assert F.rel_err(got, want) < (3e-2 if dt == BF16 else 2e-5), cuts


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("steps", ["portion", "single"])
@pytest.mark.parametrize("which", [0, 1])
def test_window_edges_and_kept_positions_with_one_key_standing_out(gpu, dt, steps, which):
    """One map of query i points at key j: seen, that map returns j's value (the output is the normed mixture of it with the other
    map's average); unseen, nothing of it.  j walks over the last place inside the window and the first one outside, the last kept
    position and the next one, page borders, position 0 and the token itself."""
    H, G, D, Dv, page = 2, 1, 8, 6, 16
    T = 200
    r = np.random.default_rng(9)
    cases = ((32, 4, 199, 168), (32, 4, 199, 167), (32, 4, 199, 3), (32, 4, 199, 4), (17, 16, 67, 15), (17, 16, 67, 16), (17, 16, 33, 16), (17, 0, 67, 51), (17, 0, 67, 50), (17, 0, 17, 0),
             (17, 0, 16, 0), (17, 1, 40, 0), (17, 40, 199, 39), (17, 40, 199, 40), (17, 33, 150, 32), (17, 33, 150, 33), (0, 0, 199, 0), (1, 2, 77, 77), (1, 2, 77, 76), (1, 2, 77, 1), (200, 5, 199, 0))
    for window, keep, i, j in cases:
        q, k, v = 0.05 * r.standard_normal((T, 2 * H * D)), 0.05 * r.standard_normal((T, 2 * G * D)), r.standard_normal((T, G * Dv))
        u = r.standard_normal(D); u /= np.linalg.norm(u)
        q[i, which * D:(which + 1) * D] = 30.0 * u   # head 0 of token i, one map
        k[j, which * D:(which + 1) * D] = 30.0 * u
        args = (window, keep, 1.0, 0.0, 0.8, 0.2, 1e-6, None)
        want = diff_want(q, k, v, None, H, G, D, *args)
        k2 = k.copy(); k2[j, which * D:(which + 1) * D] = 0
        moved = np.abs(diff_want(q, k2, v, None, H, G, D, *args)[i, :Dv] - want[i, :Dv]).max()
        visible = j <= i and (window == 0 or i - j < window or j < keep)
        alone = window == 1 and j == i and keep == 0
        assert (moved > 1e-2) == (visible and not alone), (window, keep, i, j)  # the oracle itself tells inside from outside
        cuts = [T] if steps == "portion" else [i - 3] + [1] * (T - i + 3)
        got = run_diff(gpu, dt, q, k, v, None, H, G, D, *args, cuts, page, seed=i)
        assert np.abs(got[i] - want[i]).max() < (4e-2 if dt == BF16 else 3e-5), (window, keep, i, j)
        assert F.rel_err(got, want) < (3e-2 if dt == BF16 else 2e-5), (window, keep, i, j)


def test_the_maps_are_laid_out_head_by_head_and_the_difference_has_a_sign(gpu):
    """lambda = 0 leaves the first map alone, whatever the second one holds; swapping the maps is another answer."""
    r = np.random.default_rng(2)
    H, G, D, Dv, T = 2, 2, 6, 4, 20
    q, k, v = (r.standard_normal((T, n)) for n in (2 * H * D, 2 * G * D, G * Dv))
    a = (0, 0, 0.5, 0.0)
    one = run_diff(gpu, F32, q, k, v, None, H, G, D, *a, 0.0, 0.0, 1e-6, None, [T], 8)
    q2, k2 = q.reshape(T, H, 2, D).copy(), k.reshape(T, G, 2, D).copy()
    q2[:, :, 1], k2[:, :, 1] = 7.0, -3.0
    assert F.rel_err(run_diff(gpu, F32, q2.reshape(T, -1), k2.reshape(T, -1), v, None, H, G, D, *a, 0.0, 0.0, 1e-6, None, [T], 8), one) < 1e-6
    both = run_diff(gpu, F32, q, k, v, None, H, G, D, *a, 0.9, 0.0, 1e-6, None, [T], 8)
    swapped = run_diff(gpu, F32, q.reshape(T, H, 2, D)[:, :, ::-1].reshape(T, -1), k.reshape(T, G, 2, D)[:, :, ::-1].reshape(T, -1), v, None, H, G, D, *a, 0.9, 0.0, 1e-6, None, [T], 8)
    assert F.rel_err(both, swapped) > 0.1


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("T", [7, 90])
def test_plain_attention_with_kept_first_positions(gpu, dt, T):
    """one map, the same mask: the operator another design would use"""
    r = np.random.default_rng(T)
    H, G, D, Dv, page, window, keep = 4, 2, 8, 6, 8, 9, 5
    lib = gpu.cuda_lib()
    q, k, v = (r.standard_normal((T, n)) for n in (H * D, G * D, G * Dv))
    ld, es = int(lib.ggb_window_cache_ld(G, D, Dv)), 2 if dt == BF16 else 4
    n_pages = T // page + 2
    cache, qo, out = zeros(gpu, n_pages * page * ld * es), zeros(gpu, T * H * D * 4), zeros(gpu, T * H * Dv * es)
    x, tb, pos0 = dev(gpu, f32(np.concatenate([q, k, v], 1))), dev(gpu, np.random.default_rng(1).permutation(n_pages).astype(np.int32)), dev(gpu, i32([0]))
    gpu.check(lib.ggb_op_masked_qkv_store(dt, x.ptr, at(x, 4 * H * D), at(x, 4 * (H + G) * D), (H + G) * D + G * Dv, T, H, G, D, Dv, None, None, 0.0, 0, 0, None, None, 0.6, pos0.ptr,
                                          tb.ptr, page, cache.ptr, qo.ptr), "store")
    gpu.check(lib.ggb_op_masked_attn_keep(dt, qo.ptr, cache.ptr, tb.ptr, page, pos0.ptr, T, H, G, D, Dv, window, keep, 2.5, out.ptr, None), "attn")
    vis = TP.visible(T, window, keep)
    want = np.concatenate([TP.attention_map(q.reshape(T, H, D)[:, h], k.reshape(T, G, D)[:, h // 2], v.reshape(T, G, Dv)[:, h // 2], 0.6, 2.5, vis) for h in range(H)], 1)
    assert F.rel_err(from_dt(dt, out, (T, H * Dv)), want) < (2e-2 if dt == BF16 else 5e-6)


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,D,Dr,Dv,R,Rq,page,dims", [(3, 7, 4, 6, 9, 11, 8, 4), (2, 16, 8, 16, 64, 24, 16, 8), (5, 4, 6, 2, 33, 5, 4, 6), (2, 8, 10, 12, 130, 3, 32, 6), (1, 2, 2, 2, 1, 1, 2, 2)])
def test_latents_halves_rotation_and_both_forms_of_the_scores(gpu, dt, H, D, Dr, Dv, R, Rq, page, dims):
    """prep (both normed latents, the shared rotated key part) -> absorbed form in portions and single tokens, and the materialised
    form of the same rows; one far query / key pair made to stand out"""
    r = np.random.default_rng(R)
    lib = gpu.cuda_lib()
    T, eps, scale, es = 120, 1e-5, 0.4, 2 if dt == BF16 else 4
    (ukv, uku), (uvv, uvu) = as_dt(dt, r.standard_normal((H * D, R)) / np.sqrt(R)), as_dt(dt, r.standard_normal((H * Dv, R)) / np.sqrt(R))
    dq, dkv, q = r.standard_normal((T, Rq)), r.standard_normal((T, R + Dr)), r.standard_normal((T, H * (D + Dr)))
    dkv[17] *= 3.0                                  # one latent and rotated part that ...
    q[100] *= 4.0                                   # ... one late query looks for among a hundred others
    qn, kn = 1 + 0.2 * r.standard_normal(Rq), 1 + 0.2 * r.standard_normal(R)
    rot = {"dims": dims, "base": 30.0}
    pos = np.arange(T)
    c = TP.rms_norm(dkv[:, :R], kn, eps)
    kr = TP.rotate(dkv[:, None, R:], pos, rot, True)[:, 0]
    qq = q.reshape(T, H, D + Dr)
    qr = TP.rotate(qq[..., D:], pos, rot, True)
    ku, vv = (c @ ukv.T).reshape(T, H, D), (c @ uvv.T).reshape(T, H, Dv)
    want = np.zeros((T, H, Dv))
    for h in range(H):
        s = np.where(TP.visible(T, 0), (qq[:, h, :D] @ ku[:, h].T + qr[:, h] @ kr.T) * scale, -np.inf)
        want[:, h] = TP.softmax(s) @ vv[:, h]
    want = want.reshape(T, H * Dv)
    ldk, n_pages = int(lib.ggb_latent_cache_ld(R, Dr)), T // page + 4
    tb, cs = dev(gpu, np.random.default_rng(3).permutation(n_pages).astype(np.int32)), dev(gpu, cos_sin(rot, T + 1))
    cat = np.concatenate([uku, uvu], 0)
    w_ukv, d_qn, d_kn = dev(gpu, cat), dev(gpu, f32(qn)), dev(gpu, f32(kn))
    uv_at = at(w_ukv, H * D * R * es)
    tol = 2e-2 if dt == BF16 else 2e-5
    for cuts in ([T], [40] + [1] * 30 + [2, 3, 45]):
        cache = zeros(gpu, n_pages * page * ldk * es)
        lo, got, mat, cqs = 0, [], [], []
        for n in cuts:
            x, qd, pos0 = dev(gpu, f32(np.concatenate([dq, dkv], 1)[lo:lo + n])), dev(gpu, f32(q[lo:lo + n])), dev(gpu, i32([lo]))
            cq, qa, ns = zeros(gpu, n * Rq * es), zeros(gpu, n * H * (max(R, D) + Dr) * 4), 1 if n > 8 else 3
            part, out = zeros(gpu, lib.ggb_latent_attn_scratch_bytes(n, H, R, ns)), zeros(gpu, n * H * Dv * es)
            gpu.check(lib.ggb_op_latent_prep(dt, x.ptr, Rq, d_qn.ptr, cq.ptr, at(x, 4 * Rq), Rq + R + Dr, n, R, Dr, dims, 1, d_kn.ptr, eps, cs.ptr, pos0.ptr, tb.ptr, page, cache.ptr), "prep")
            gpu.check(lib.ggb_op_latent_q_absorb_halves(dt, qd.ptr, H * (D + Dr), n, H, D, Dr, dims, cs.ptr, pos0.ptr, w_ukv.ptr, R, scale, qa.ptr), "absorb")
            gpu.check(lib.ggb_op_latent_attn(dt, qa.ptr, cache.ptr, tb.ptr, page, pos0.ptr, n, H, R, Dr, ns, part.ptr), "attn")
            gpu.check(lib.ggb_op_latent_attn_out_gated(dt, part.ptr, ns, None, uv_at, n, H, R, Dv, None, 0, out.ptr), "out")
            got.append(from_dt(dt, out, (n, H * Dv)))
            cqs.append(from_dt(dt, cq, (n, Rq)))
            if n >= 32:  # the window kernel's portion form takes any key size
                vis, ldkv = lo + n, int(lib.ggb_window_cache_ld(H, D + Dr, Dv))
                crows, kvf, kv = zeros(gpu, vis * R * es), zeros(gpu, vis * H * (D + Dv) * 4), zeros(gpu, (vis + 8) * ldkv * es)
                iota = dev(gpu, np.arange(vis // page + 2, dtype=np.int32))
                gpu.check(lib.ggb_op_latent_expand_rot(dt, cache.ptr, tb.ptr, page, 0, vis, R, H, D, Dr, Dv, w_ukv.ptr, crows.ptr, kvf.ptr, kv.ptr, ldkv), "expand")
                gpu.check(lib.ggb_op_latent_q_rotate(qd.ptr, H * (D + Dr), n, H, D, Dr, dims, 1, cs.ptr, pos0.ptr, scale, qa.ptr), "rotate")
                gpu.check(lib.ggb_op_window_attn(dt, qa.ptr, kv.ptr, iota.ptr, page, pos0.ptr, n, H, H, D + Dr, Dv, 0, None, out.ptr, None), "window_attn")
                mat.append((lo, from_dt(dt, out, (n, H * Dv))))
            lo += n
        assert F.rel_err(np.concatenate(cqs), TP.rms_norm(dq, qn, eps)) < (5e-3 if dt == BF16 else 1e-6)
        assert F.rel_err(np.concatenate(got), want) < tol, len(cuts)
        for lo, m in mat:
            assert F.rel_err(m, want[lo:lo + len(m)]) < tol, lo


# ------------------------------------------------------------------------------------------------ gated diagonal recurrence
def rglru_inputs(r, T, nb, d, taps):
    C = nb * d
    v = dict(x=r.standard_normal((T, C)), y=r.standard_normal((T, C)), xb=0.5 * r.standard_normal(C), yb=0.5 * r.standard_normal(C), conv=0.6 * r.standard_normal((C, taps)),
             cb=0.5 * r.standard_normal(C), ra=r.standard_normal((nb, d, d)) / np.sqrt(d), ri=r.standard_normal((nb, d, d)) / np.sqrt(d),
             rab=r.standard_normal((nb, d)) - 1.0, rib=r.standard_normal((nb, d)), lam=r.standard_normal(C) - 2.0)
    v["ra"], v["ri"] = F.bf16_round(v["ra"])[0].reshape(nb, d, d), F.bf16_round(v["ri"])[0].reshape(nb, d, d)
    return v


def rglru_want(v):
    u = TP.causal_conv(v["x"] + v["xb"], v["conv"], v["cb"])
    rr, ii = TP.sigmoid(TP.block_product(u, v["ra"], v["rab"])), TP.sigmoid(TP.block_product(u, v["ri"], v["rib"]))
    S, last = TP.rglru_core(u, rr, ii, v["lam"])
    return S * TP.gelu_tanh(v["y"] + v["yb"]), last


def run_rglru(gpu, dt, v, nb, d, taps, cuts, no_split=False, garbage=False):
    lib = gpu.cuda_lib()
    T, C, es = v["x"].shape[0], nb * d, 2 if dt == BF16 else 4
    pad = np.zeros((T, 3))
    rows = f32(np.concatenate([v["x"], pad, v["y"], pad], 1))   # a row stride of its own
    ld = rows.shape[1]
    stack = np.stack([v["ra"], v["ri"]], 1).reshape(nb, 2 * d, d)
    w2 = dev(gpu, as_dt(dt, stack)[1])
    w3 = dev(gpu, as_dt(dt, np.concatenate([stack] * 3, 2))[1])
    b2 = dev(gpu, f32(np.stack([v["rab"], v["rib"]], 1)))
    cw, cb, xb, yb, rate = (dev(gpu, f32(a)) for a in (v["conv"], v["cb"], v["xb"], v["yb"], -8.0 * TP.softplus(v["lam"])))
    L = int(lib.ggb_rglru_history_rows(taps))
    hist, S = zeros(gpu, L * C * 4), zeros(gpu, C * 4)
    if garbage:  # slots of a ring that no earlier token has written are not read
        hist.upload(f32(np.full(max(L * C, 4), 1e30)))
    lo, got = 0, []
    for n in cuts:
        x, out, pos0 = dev(gpu, rows[lo:lo + n]), zeros(gpu, n * C * es), dev(gpu, i32([lo]))
        y = at(x, 4 * (C + 3))
        if lib.ggb_rglru_step_form(n, d):
            gpu.check(lib.ggb_op_rglru_step(dt, x.ptr, y, ld, n, nb, d, cw.ptr, cb.ptr, taps, xb.ptr, yb.ptr, w2.ptr, b2.ptr, rate.ptr, pos0.ptr, hist.ptr, S.ptr, out.ptr), "step")
        else:
            u, z = zeros(gpu, n * C * 4), zeros(gpu, n * C * 8)
            split = zeros(gpu, n * C * 6) if lib.ggb_rglru_split_fits(dt, n, d) and not no_split else None
            off = zeros(gpu, (nb + 1) * 4)
            gpu.check(lib.ggb_op_rglru_conv(x.ptr, ld, n, nb, d, cw.ptr, cb.ptr, taps, xb.ptr, pos0.ptr, hist.ptr, u.ptr, ptr(split), off.ptr), "conv")
            gpu.check(lib.ggb_op_rglru_gates(dt, u.ptr, ptr(split), off.ptr, n, nb, d, w2.ptr, w3.ptr, z.ptr), "gates")
            gpu.check(lib.ggb_op_rglru_scan(dt, z.ptr, u.ptr, y, ld, n, nb, d, yb.ptr, b2.ptr, rate.ptr, S.ptr, out.ptr), "scan")
        got.append(from_dt(dt, out, (n, C)))
        lo += n
    assert lo == T
    return np.concatenate(got), S.download(np.float32, C)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("nb,d,taps", [(1, 1, 1), (3, 8, 4), (5, 7, 2), (1, 30, 8), (2, 64, 4), (4, 128, 3), (1, 300, 5), (7, 1, 3)])
def test_recurrence_in_steps_and_portions(gpu, dt, nb, d, taps):
    r = np.random.default_rng(nb * 1000 + d)
    T = 180
    v = rglru_inputs(r, T, nb, d, taps)
    want, last = rglru_want(v)
    for cuts in ([T], [1] * 20 + [160], [2, 3, 8, 9, 1, 1, 33, 4, 7, 64, 8, 5, 8, 8, 10, 9], [100, 1, 1, 1, 77]):
        got, S = run_rglru(gpu, dt, v, nb, d, taps, cuts, garbage=True)
        # the state is fp32 in both types: matrices are bf16 numbers already and u keeps all its bits
        assert F.rel_err(S, last) < 5e-6, (cuts[:3], F.rel_err(S, last))
        assert F.rel_err(got, want) < (4e-3 if dt == BF16 else 5e-6), cuts[:3]


def test_gates_on_the_tensor_cores_keep_32_bits(gpu):
    """u as three bf16 numbers: the state after a long portion is as close to the oracle as with the fp32 tile kernel, and
    far closer than u rounded once would be"""
    r = np.random.default_rng(5)
    nb, d, taps, T = 2, 128, 4, 700
    v = rglru_inputs(r, T, nb, d, taps)
    v["x"] *= 3.0
    want, last = rglru_want(v)
    lib = gpu.cuda_lib()
    assert lib.ggb_rglru_split_fits(BF16, T, d) and not lib.ggb_rglru_split_fits(F32, T, d)
    e_split, e_tile = (F.rel_err(run_rglru(gpu, BF16, v, nb, d, taps, [T], no_split=s)[1], last) for s in (False, True))
    u = TP.causal_conv(v["x"] + v["xb"], v["conv"], v["cb"])
    ub = F.bf16_round(u)[0].reshape(u.shape)
    rounded = TP.rglru_core(u, TP.sigmoid(TP.block_product(ub, v["ra"], v["rab"])), TP.sigmoid(TP.block_product(ub, v["ri"], v["rib"])), v["lam"])[1]
    assert e_split < 5e-6 and e_tile < 5e-6 and F.rel_err(rounded, last) > 50 * e_split


def test_hardly_decaying_and_forgetting_channels(gpu):
    """1 - a^2 is taken without cancellation (a channel that keeps everything), and a channel with a = 0 holds its own input only"""
    r = np.random.default_rng(6)
    nb, d, taps, T = 1, 16, 2, 150
    v = rglru_inputs(r, T, nb, d, taps)
    v["lam"][:8], v["lam"][8:] = -16.0, 6.0
    v["rab"][0, 8:] = 9.0
    want, last = rglru_want(v)
    for cuts in ([T], [1] * T, [64, 8, 8, 70]):
        got, S = run_rglru(gpu, F32, v, nb, d, taps, cuts)
        assert F.rel_err(S[:8], last[:8]) < 2e-6 and F.rel_err(S[8:], last[8:]) < 2e-6 and F.rel_err(got, want) < 5e-6
