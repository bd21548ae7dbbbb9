"""Host-side pieces of the Fekopel path that need no GPU: registry, configuration reader and refusals, what the cache keeps, and the
plain oracle's own consistency (gelu, layer norm, the sink, kept first positions, groups, the looped block)."""
import ctypes as C
import json

import numpy as np
import pytest

import fekopel_fixture as F
import fekopel_plain as FP


def probe(G, cfg):
    out = (C.c_int64 * 10)()
    rc = G.host_lib().fk_config_probe(json.dumps(cfg).encode(), out)
    return rc, list(out), G.host_lib().gm_last_error().decode()


def test_registry_knows_the_architecture(G):
    assert "Fekopel" in G.architectures() and "Tezesun" in G.architectures()


def test_config_reader_takes_every_size_and_the_order_of_layers_from_the_file(G):
    rc, out, _ = probe(G, F.small_config())
    assert rc == 0 and out == [4, 2, 2, 3, 2, 59, 38, 8, 0, 0]       # one layer sees everything
    rc, out, _ = probe(G, F.windowed_config(vocab=9, width=8))      # what the farthest-looking layer sees
    assert rc == 0 and out == [3, 1, 2, 2, 1, 9, 8, 5, 13, 6]
    rc, out, _ = probe(G, F.config([F.attn()] * 3, loop=(2, 3, 1)))  # a block that runs once is still a pass
    assert rc == 0 and out[7:] == [3, 13, 0]
    rc, out, _ = probe(G, F.config([F.attn(), F.attn2()]))
    assert rc == 0 and out[7:] == [2, 13, 3]
    cfg = F.small_config()
    cfg["loop"] = cfg["layers"][1]["mlp"]["shared"] = cfg["layers"][0]["mlp"]["router"]["groups"] = None  # null: absent
    assert probe(G, cfg)[1][7] == 4


@pytest.mark.parametrize("breaker, word", [
    (lambda c: c["layers"][0].update(type="other_mixer"), "unknown mixer"),
    (lambda c: c["layers"][0].update(mixer=None), "mixer"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads must divide"),
    (lambda c: c["layers"][1]["mixer"].update(dim=0), "positive"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=7), "even"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=258), "256"),
    (lambda c: c["layers"][1]["mixer"].update(dim=514), "512"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0), "rot.base"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=-1), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "mask.keep_first"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1), "softcap"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "unknown mlp"),
    (lambda c: c["layers"][0]["mlp"].update(router=None), "router"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top at most"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(experts=200, top=65, groups=None), "64 a token"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "shared.ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c.update(layers=[]), "list"),
    (lambda c: c.update(width=0), "positive"),
])
def test_config_reader_refuses_what_the_design_does_not_have(G, breaker, word):
    cfg = F.small_config()
    breaker(cfg)
    rc, _, msg = probe(G, cfg)
    assert rc != 0 and word in msg, msg


def test_gelu_is_the_exact_one():
    z = np.array([-3.0, -1.0, 0.0, 0.5, 2.0])
    want = [-0.00404969409489031, -0.15865525393145707, 0.0, 0.34573123063700656, 1.9544997361036416]  # z times the normal distribution function
    assert np.abs(FP.gelu_erf(z) - want).max() < 1e-12


def test_layer_norm_takes_the_mean_off_and_adds_the_bias():
    x = np.random.default_rng(0).standard_normal((3, 50)) + 7.0
    y = FP.layer_norm(x, np.full(50, 2.0), np.full(50, -1.0), 0.0)
    assert np.allclose(y.mean(-1), -1.0) and np.allclose(((y + 1.0) ** 2).mean(-1), 4.0)


def test_a_sink_of_score_zero_is_a_key_of_score_zero_with_a_zero_value():
    s = np.random.default_rng(1).standard_normal((4, 6)) * 3
    p = FP.sink_softmax(s, 0.0)
    assert np.allclose(p, FP.softmax(np.concatenate([s, np.zeros((4, 1))], 1))[:, :6])
    assert np.allclose(FP.sink_softmax(np.zeros((1, 3)), 0.0), 0.25) and np.allclose(FP.sink_softmax(s), FP.softmax(s))
    assert np.allclose(FP.sink_softmax(np.full((1, 2), -800.0), 0.0), 0.0) and np.allclose(FP.sink_softmax(np.full((1, 2), 800.0), 0.0), 0.5)


def test_visible_counts_the_window_and_the_kept_positions():
    v = FP.visible(12, 3, 2)
    assert v[11].nonzero()[0].tolist() == [0, 1, 9, 10, 11] and v[2].nonzero()[0].tolist() == [0, 1, 2] and v[0].nonzero()[0].tolist() == [0]
    assert FP.visible(12, 0)[11].all() and FP.visible(12, 3)[11].sum() == 3 and FP.visible(4, 1)[3].nonzero()[0].tolist() == [3]


def test_groups_hide_the_second_best_expert_and_the_factor_multiplies_the_weights():
    router = np.log(np.array([[0.4], [0.05], [0.3], [0.25]]))  # one input number: the scores are 0.4, 0.05, 0.3, 0.25
    h = np.ones((1, 1))
    idx, w = FP.route(h, router, 2)
    assert idx.tolist() == [[0, 2]] and np.allclose(w, [[0.4 / 0.7, 0.3 / 0.7]])
    idx, w = FP.route(h, router, 2, groups=2, keep=1, scale=3.0)
    assert idx.tolist() == [[0, 1]] and np.allclose(w, [[3 * 0.4 / 0.45, 3 * 0.05 / 0.45]])
    # a group's score is its largest one, not its sum: {0.3, 0.25} has the larger sum
    idx, _ = FP.route(h, router, 1, groups=2, keep=1)
    assert idx.tolist() == [[0]]


def test_a_pass_adds_its_vector_and_every_pass_but_the_first_the_embedding():
    assert FP.layer_runs(F.config([0] * 5, loop=(1, 3, 2))) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None), (4, None)]
    cfg = F.config([F.attn()], width=6, loop=(0, 1, 3))
    W = FP.random_weights(cfg, 1)
    W["l0.mix.o"][:] = 0.0  # the layer adds nothing
    runs = []
    FP.forward([5, 3], W, cfg, runs)
    e, s = W["embed"][[5, 3]], W["loop.step"]
    assert np.allclose(runs[0], e + s[0]) and np.allclose(runs[1], 2 * e + s[0] + s[1]) and np.allclose(runs[2], 3 * e + s.sum(0))


def test_whole_forward_is_causal():
    cfg = F.small_config()
    W = FP.random_weights(cfg, 3)
    a = np.random.default_rng(0).integers(0, cfg["vocab"], 30)
    b = a.copy()
    b[20] = (b[20] + 1) % cfg["vocab"]
    za, zb = FP.forward(a, W, cfg), FP.forward(b, W, cfg)
    assert np.abs(za[:20] - zb[:20]).max() < 1e-12 and np.abs(za[20:] - zb[20:]).max(axis=1).min() > 1e-6
