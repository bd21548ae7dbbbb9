"""Host-side pieces of the Tezesun path that need no GPU: registry, configuration reader and refusals, what the cache keeps, and
the plain oracle's own consistency (token shift, xIELU, the frequency blend, kept first positions, the recurrence continued from a
state, the difference of two maps)."""
import ctypes as C
import json

import numpy as np
import pytest

import tezesun_fixture as F
import tezesun_plain as TP


def probe(G, cfg):
    out = (C.c_int64 * 9)()
    rc = G.host_lib().tz_config_probe(json.dumps(cfg).encode(), out)
    return rc, list(out), G.host_lib().gm_last_error().decode()


def test_registry_knows_the_architecture(G):
    assert "Tezesun" in G.architectures() and "Kibilix" in G.architectures()


def test_config_reader_takes_every_size_and_the_order_of_layers_from_the_file(G):
    rc, out, _ = probe(G, F.small_config())
    assert rc == 0 and out == [6, 2, 2, 2, 3, 61, 36, 0, 0]
    rc, out, _ = probe(G, F.windowed_config(vocab=9, width=8))  # what every layer sees: the widest window and the most kept tokens
    assert rc == 0 and out == [3, 2, 0, 1, 3, 9, 8, 13, 6]
    rc, out, _ = probe(G, F.config([F.layer("attention", F.attention(window=0)), F.layer("attention", F.attention())]))
    assert rc == 0 and out[7:] == [0, 0]                        # one layer sees everything
    rc, out, _ = probe(G, F.config([F.layer("rglru", F.rglru())]))
    assert rc == 0 and out == [1, 0, 0, 1, 0, 61, 36, 0, 0]     # no rows per position at all


@pytest.mark.parametrize("breaker, word", [
    (lambda c: c["layers"][0].update(type="other_mixer"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].update(blocks=5), "blocks must divide"),
    (lambda c: c["layers"][0]["mixer"].update(conv=9), "conv"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads must divide"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=7), "even"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=258), "256"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=12), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "rot.scaling"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=-1), "mask"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1), "softcap"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"].update(q_rank=0), "q_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "rot.dims"),
    (lambda c: c["layers"][2]["mlp"].update(kind="other"), "unknown mlp"),
    (lambda c: c["layers"][2]["mlp"].update(ff=0), "ff must"),
    (lambda c: c.update(layers=[]), "list"),
    (lambda c: c.update(width=0), "positive"),
])
def test_config_reader_refuses_what_the_design_does_not_have(G, breaker, word):
    cfg = F.small_config()
    breaker(cfg)
    rc, _, msg = probe(G, cfg)
    assert rc != 0 and word in msg, msg


def test_token_shift_blends_towards_the_row_before():
    h = np.arange(6.0).reshape(3, 2) + 1
    assert np.array_equal(TP.token_shift(h, np.array([0.0, 1.0])), [[1, 0], [3, 2], [5, 4]])


def test_xielu_is_continuous_with_slope_one_half_at_zero():
    e = 1e-7
    for p, q in ((0.3, -0.2), (-2.0, 1.5)):
        z = np.array([-e, 0.0, e])
        y = TP.xielu(z, p, q)
        assert abs(y[1]) == 0 and abs(y[2] / e - 0.5) < 1e-5 and abs(y[0] / -e - 0.5) < 1e-5
        assert abs(TP.xielu(np.array([2.0]), p, q)[0] - (np.log1p(np.exp(p)) * 4 + 1)) < 1e-12
        assert abs(TP.xielu(np.array([-1.0]), p, q)[0] - ((0.5 + np.log1p(np.exp(q))) * np.exp(-1) - 0.5)) < 1e-12


def test_frequency_blend_keeps_short_waves_divides_long_ones_and_ramps_between():
    rot = {"dims": 32, "base": 10000.0, "scaling": {"factor": 4.0, "original": 512, "fast": 16.0, "slow": 1.0}}
    f, mag = TP.rot_frequencies(rot)
    plain = TP.rot_frequencies({"dims": 32, "base": 10000.0})[0]
    ratio = f / plain
    assert ratio[0] == 1.0 and abs(ratio[-1] - 0.25) < 1e-12 and (np.diff(ratio) <= 1e-12).all() and ((ratio > 0.26) & (ratio < 0.99)).any()
    assert abs(mag - (0.1 * np.log(4.0) + 1.0)) < 1e-12


def test_both_rotary_layouts_turn_lengths_by_the_magnitude_and_leave_the_rest():
    x = np.random.default_rng(0).standard_normal((5, 2, 10))
    rot = {"dims": 8, "base": 10.0, "scaling": {"factor": 3.0, "original": 30, "fast": 4.0, "slow": 1.0}}
    mag = TP.rot_frequencies(rot)[1]
    for halves in (False, True):
        y = TP.rotate(x, np.arange(5) + 3, rot, halves)
        assert np.array_equal(y[..., 8:], x[..., 8:])
        assert np.allclose(np.linalg.norm(y[..., :8], axis=-1), mag * np.linalg.norm(x[..., :8], axis=-1))
    assert not np.allclose(TP.rotate(x, np.arange(5) + 3, rot, False), TP.rotate(x, np.arange(5) + 3, rot, True))


def test_visible_counts_the_window_and_the_kept_positions():
    v = TP.visible(12, 3, 2)
    assert v[11].nonzero()[0].tolist() == [0, 1, 9, 10, 11] and v[2].nonzero()[0].tolist() == [0, 1, 2] and v[0].nonzero()[0].tolist() == [0]
    assert TP.visible(12, 0, 0)[11].all() and TP.visible(12, 3, 0)[11].sum() == 3


def test_recurrence_continues_from_a_state_and_starts_like_every_other_token():
    r = np.random.default_rng(1)
    u, rr, ii, lam = r.standard_normal((9, 4)), r.uniform(0, 1, (9, 4)), r.uniform(0, 1, (9, 4)), r.standard_normal(4)
    whole, last = TP.rglru_core(u, rr, ii, lam)
    a, mid = TP.rglru_core(u[:4], rr[:4], ii[:4], lam)
    b, end = TP.rglru_core(u[4:], rr[4:], ii[4:], lam, mid)
    assert np.allclose(np.concatenate([a, b]), whole) and np.allclose(end, last)
    a0 = np.exp(-8.0 * rr[0] * np.log1p(np.exp(lam)))
    assert np.allclose(whole[0], np.sqrt(1 - a0 ** 2) * ii[0] * u[0])  # the first token's input is scaled too


def test_last_tap_is_the_current_token_and_the_bias_is_added_once():
    x = np.arange(1.0, 5.0)[:, None]
    assert np.array_equal(TP.causal_conv(x, np.array([[10.0, 1.0]]), np.array([100.0]))[:, 0], [101, 112, 123, 134])


def test_equal_maps_cancel_to_a_scaled_single_map():
    """two equal maps and lambda < 1: the difference points where one map points, and the norm removes the factor"""
    r = np.random.default_rng(2)
    T, D, Dv = 6, 4, 5
    q, k, v = r.standard_normal((T, 1, 1, D)), r.standard_normal((T, 1, 1, D)), r.standard_normal((T, 1, Dv))
    two = TP.diff_core(np.repeat(q, 2, 2), np.repeat(k, 2, 2), v, 0.5, 0.0, TP.visible(T, 0), 0.25, 0.4, 0.0)
    one = TP.attention_map(q[:, 0, 0], k[:, 0, 0], v[:, 0], 0.5, 0.0, TP.visible(T, 0))
    assert np.allclose(two[:, 0], 0.6 * TP.rms_unit(one, 0.0))


def test_whole_forward_is_causal():
    cfg = F.small_config()
    W = TP.random_weights(cfg, 3)
    a = np.random.default_rng(0).integers(0, cfg["vocab"], 30)
    b = a.copy()
    b[20] = (b[20] + 1) % cfg["vocab"]
    za, zb = TP.forward(a, W, cfg), TP.forward(b, W, cfg)
    assert np.array_equal(za[:20], zb[:20]) and np.abs(za[20:] - zb[20:]).max(axis=1).min() > 1e-6
