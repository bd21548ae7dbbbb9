"""Tezesun through the serving engine against the plain numpy oracle (tests/tezesun_plain.py): whole prompts and every layer,
portions down to two tokens, token-by-token decoding, several live sequences of unequal length, slots and pages that are freed
and used again (also by the same sequence, behind its windows), the first tokens of a sequence, long decoding, other sizes and
optional parts, and greedy generation through the engine's own entry point."""
import numpy as np
import pytest

import tezesun_fixture as F
import tezesun_plain as TP

pytestmark = pytest.mark.gpu


def close(got, want, dtype, loose=1.0):
    """every row of logits within rounding of the oracle, in float32 and in bfloat16 (no choice in this design can flip)"""
    got, want = np.atleast_2d(np.asarray(got, dtype=np.float64)), np.atleast_2d(np.asarray(want, dtype=np.float64))
    assert got.shape == want.shape, (got.shape, want.shape)
    e = np.sqrt(((got - want) ** 2).mean(-1)) / (np.sqrt((want ** 2).mean()) + 1e-30)
    lim = (2e-5 if dtype == "float32" else 5e-2) * loose
    if e.max() >= lim or (dtype != "float32" and np.median(e) >= 0.5 * lim):
        print("rows over:", np.nonzero(e >= lim)[0][:20], "worst", e.max(), "median", np.median(e))
        return False
    return bool(np.isfinite(got).all())


def make(tmp_path_factory, cfg, seed, n):
    d, W = F.make_model(str(tmp_path_factory.mktemp("tz") / "m"), cfg, seed=seed)
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], n)
    return cfg, d, W, toks, TP.forward(toks, W, cfg)


@pytest.fixture(scope="module")
def small(gpu, tmp_path_factory):
    return make(tmp_path_factory, F.small_config(), 11, 150)


@pytest.fixture(scope="module")
def windowed(gpu, tmp_path_factory):
    return make(tmp_path_factory, F.windowed_config(), 12, 150)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_and_every_layer(gpu, small, dtype):
    cfg, d, W, toks, want = small
    eng = gpu.Engine(d, dtype=dtype, max_tokens=256, page_size=16)
    assert eng.architecture == "Tezesun"
    eng.capture(True)
    got = eng.step([("a", toks, np.arange(len(toks)))], ["a"])
    assert close(got, want, dtype)
    xs = []
    TP.forward(toks, W, cfg, xs)
    for i, x in enumerate(xs):
        assert close(eng.captured(i, len(toks), cfg["width"]), x, dtype), i
    assert eng.stats()["live_seqs"] == 0 and eng.stats()["free_pages"] == eng.stats()["pages"]
    eng.capture(False)
    again = eng.step([("b", toks, np.arange(len(toks)))], ["b"])
    assert np.abs(again - got).max() < 1e-3
    eng.close()


CUTS = (([1] * 40, 16, 0), ([2] * 20 + [3, 5, 2, 31, 17, 2, 1, 1, 48], 16, 0), ([150], 8, 7), ([63, 1, 1, 1, 64, 2, 18], 64, 32),
        ([2, 1, 2, 4, 3, 33, 1, 1, 2, 60], 4, 0), ([10, 1, 13, 12, 8, 9, 5, 7, 22], 2, 0), ([3] * 13 + [4] * 9, 5, 3), ([8, 8, 9, 9, 7, 8, 32, 33, 31], 16, 0))


@pytest.mark.parametrize("model", ["small", "windowed"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_decoding_equal_the_whole_prompt(gpu, request, model, dtype):
    cfg, d, W, toks, want = request.getfixturevalue(model)
    for cuts, page, portion in CUTS:
        eng = gpu.Engine(d, dtype=dtype, max_tokens=200, page_size=page, max_portion=portion)
        lo, rows = 0, []
        for c in cuts:
            rows.append(eng.step([("s", toks[lo:lo + c], np.arange(c))]))
            lo += c
        got = np.concatenate(rows)
        assert close(got, want[:lo], dtype), cuts[:3]
        eng.end("s")
        whole = eng.step([("w", toks[:lo], np.arange(lo))], ["w"])
        assert close(got, whole, dtype), cuts[:3]
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_several_sequences_reused_slots_and_first_tokens(gpu, small, dtype):
    cfg, d, W, toks, want = small
    r = np.random.default_rng(8)
    seqs = {k: r.integers(0, cfg["vocab"], n) for k, n in (("a", 70), ("b", 9), ("c", 33), ("d", 50), ("e", 1), ("f", 3))}
    alone = {k: TP.forward(v, W, cfg) for k, v in seqs.items()}
    eng = gpu.Engine(d, dtype=dtype, max_tokens=140, page_size=8, max_seqs=3)
    got = {k: [] for k in seqs}
    at = {k: 0 for k in seqs}

    def feed(*items, end=()):
        out = eng.step([(k, seqs[k][at[k]:at[k] + n], np.arange(n)) for k, n in items], end)
        lo = 0
        for k, n in items:
            got[k].append(out[lo:lo + n])
            lo += n
            at[k] += n
    feed(("a", 30), ("b", 2))
    feed(("c", 20), ("a", 1), ("b", 5))
    feed(("b", 2), ("a", 2), ("c", 13), end=["b", "c"])   # two slots and their pages come back
    free_mid = eng.stats()["free_pages"]
    feed(("d", 1), ("e", 1), end=["e"])                    # d and e start in slots that b and c used: state must be clean
    feed(("a", 37), ("d", 2), ("f", 3), end=["a", "f"])
    feed(("d", 47), end=["d"])
    for k in seqs:
        assert at[k] == len(seqs[k]) and close(np.concatenate(got[k]), alone[k], dtype), k
    st = eng.stats()
    assert st["live_seqs"] == 0 and st["free_pages"] == st["pages"] and free_mid < st["pages"]
    with pytest.raises(gpu.GgbError):  # a fourth live sequence has no slot
        eng.step([(k, [1], []) for k in "wxyz"])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_behind_the_windows_are_used_again_and_the_first_tokens_stay(gpu, windowed, dtype):
    cfg, d, W, toks, want = windowed   # windows of 13 and 7 positions, 3 and 6 kept first tokens: with pages of 4 the first two stay
    other = toks[::-1].copy()
    want_other = TP.forward(other, W, cfg)
    eng = gpu.Engine(d, dtype=dtype, max_tokens=150, page_size=4, max_seqs=2)
    lo, rows, rows_o = 0, [], []
    cuts = [9, 1, 1, 7, 16, 2, 2, 1, 16, 13, 1, 1, 1, 16, 3, 16, 16, 12, 2, 14]
    for c in cuts:
        out = eng.step([("s", toks[lo:lo + c], np.arange(c)), ("o", other[lo:lo + c], np.arange(c))])
        rows.append(out[:c]); rows_o.append(out[c:])
        lo += c
        assert eng.seq_live_pages("s") <= 13 // 4 + 2 + 2 and eng.seq_live_pages("o") <= 13 // 4 + 2 + 2
    assert lo == 150 and close(np.concatenate(rows), want, dtype) and close(np.concatenate(rows_o), want_other, dtype)
    pages = eng.seq_pages("s")
    assert len(pages) == (150 + 3) // 4 and (pages >= 0).sum() == eng.seq_live_pages("s") and (pages[:2] >= 0).all() and pages[2] < 0
    with pytest.raises(gpu.GgbError, match="positions"):  # trimming frees pages, not positions
        eng.step([("s", toks[:20], [])])
    eng.end("s", "o")
    assert eng.stats()["free_pages"] == eng.stats()["pages"]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_layer_that_sees_everything_keeps_every_page(gpu, small, dtype):
    cfg, d, W, toks, want = small
    eng = gpu.Engine(d, dtype=dtype, max_tokens=16, page_size=4, max_seqs=2)
    eng.step([("s", toks[:20], [19])])
    assert eng.seq_live_pages("s") == 5
    with pytest.raises(gpu.GgbError, match="out of pages"):
        eng.step([("t", toks[:8], [])])
    eng.close()


def test_long_decoding(gpu, small):
    cfg, d, W, toks, _ = small
    long = np.random.default_rng(2).integers(0, cfg["vocab"], 330)
    want = TP.forward(long, W, cfg)
    for dtype in ("float32", "bfloat16"):
        eng = gpu.Engine(d, dtype=dtype, max_tokens=400, page_size=32)
        rows = [eng.step([("s", long[:10], np.arange(10))])] + [eng.step([("s", long[i:i + 1], [0])]) for i in range(10, 330)]
        assert close(np.concatenate(rows), want, dtype)
        eng.use_graphs(False)  # launches one by one: the same numbers as the replayed step
        eng.end("s")
        again = [eng.step([("s", long[:10], np.arange(10))])] + [eng.step([("s", long[i:i + 1], [0])]) for i in range(10, 60)]
        assert np.abs(np.concatenate(again) - np.concatenate(rows)[:60]).max() < 1e-3
        eng.close()


OTHER = {
    # what the small configuration has unequal, equal or 1; what it has, absent
    "equal_and_absent": lambda: F.config([F.layer("attention", F.attention(heads=2, kv_heads=2, dim=8, vdim=8, window=0, softcap=0, base=0, diff=0.0), 16),
                                          F.layer("rglru", F.rglru(width=16, blocks=1, conv=1), 16),
                                          F.layer("latent_attention", F.latent(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=8, q_rank=8), 16)],
                                         vocab=16, width=16, logit_scale=1.0),
    "ones": lambda: F.config([F.layer("attention", F.attention(heads=1, kv_heads=1, dim=2, vdim=2, window=1, keep=1, dims=2, scaling=False), 1),
                              F.layer("latent_attention", F.latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, q_rank=1), 3),
                              F.layer("rglru", F.rglru(width=5, blocks=5, conv=8), 1)], vocab=30, width=7),
    "only_rglru": lambda: F.config([F.layer("rglru", F.rglru(width=40, blocks=2, conv=2), 12), F.layer("rglru", F.rglru(width=9, blocks=3, conv=4))], vocab=19, width=20),
    "only_attention": lambda: F.config([F.layer("attention", F.attention(heads=6, kv_heads=1, dim=4, vdim=14, window=200, keep=5, dims=2)),
                                        F.layer("attention", F.attention(heads=6, kv_heads=3, dim=12, vdim=4, window=1, keep=0), 9)], vocab=64, width=12, logit_scale=3.0),
    "only_latent": lambda: F.config([F.layer("latent_attention", F.latent(heads=5, dim=3, rot_dim=10, vdim=7, kv_rank=33, q_rank=70)),
                                     F.layer("latent_attention", F.latent(), 31)], vocab=23, width=26),
    # 16-byte pieces everywhere, tensor-core products and gates, the materialised latents, kept tokens over more than one tile
    "wide": lambda: F.config([F.layer("rglru", F.rglru(width=256, blocks=4, conv=4), 320),
                              F.layer("attention", F.attention(heads=4, kv_heads=2, dim=32, vdim=64, window=45, keep=37, dims=16), 160),
                              F.layer("latent_attention", F.latent(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=128, q_rank=64), 96),
                              F.layer("attention", F.attention(heads=2, kv_heads=1, dim=64, vdim=160, window=64, keep=0, dims=None, scaling=False), 64)],
                             vocab=200, width=128),
}


@pytest.mark.parametrize("name", sorted(OTHER))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes_and_optional_parts(gpu, tmp_path, name, dtype):
    cfg = OTHER[name]()
    d, W = F.make_model(str(tmp_path / name), cfg, seed=3)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], 140)
    want = TP.forward(toks, W, cfg)
    # a normed difference of two maps over one or two values is a near sign: rounding shows more there
    loose = 8.0 if name == "ones" else 2.0
    eng = gpu.Engine(d, dtype=dtype, max_tokens=300, page_size=16)
    whole = eng.step([("w", toks, np.arange(140))], ["w"])
    assert close(whole, want, dtype, loose)
    lo, rows = 0, []
    for c in [2, 2, 65, 1, 1, 3, 64, 2]:
        rows.append(eng.step([("s", toks[lo:lo + c], np.arange(c))]))
        lo += c
    assert close(np.concatenate(rows), want, dtype, loose)
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_both_forms_of_the_latent_attention_agree(gpu, tmp_path, dtype, monkeypatch):
    cfg = F.config([F.layer("latent_attention", F.latent(heads=3, dim=16, rot_dim=8, vdim=18, kv_rank=72, q_rank=24), 40)] * 2, vocab=50, width=48)
    d, W = F.make_model(str(tmp_path / "m"), cfg, seed=4)
    toks = np.random.default_rng(3).integers(0, 50, 200)
    want = TP.forward(toks, W, cfg)
    for absorbed in (False, True):
        if absorbed:
            monkeypatch.setenv("GGB_LATENT_ABSORBED", "1")
        eng = gpu.Engine(d, dtype=dtype, max_tokens=256, page_size=16)
        rows = [eng.step([("s", toks[:70], np.arange(70))]), eng.step([("s", toks[70:71], [0])]), eng.step([("s", toks[71:], np.arange(129))])]
        assert close(np.concatenate(rows), want, dtype), absorbed
        eng.close()


def test_a_far_token_reaches_the_end_through_the_recurrence_only(gpu, tmp_path):
    """The attention sees 16 positions; what a token 120 positions back changes in the last logits went through S."""
    cfg = F.config([F.layer("attention", F.attention(window=16, keep=0), 12), F.layer("rglru", F.rglru(width=16, blocks=2), 12)])

    def remember(W):  # hardly any decay: 1 - a is below what 16 bits resolve
        W["l1.mix.lam"][:] = -9.0
    d, W = F.make_model(str(tmp_path / "far"), cfg, seed=9, edit=remember)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 124)
    other = toks.copy()
    other[3] = (other[3] + 1) % cfg["vocab"]
    za, zb = TP.forward(toks, W, cfg)[-1], TP.forward(other, W, cfg)[-1]
    assert np.abs(za - zb).max() > 1e-3
    eng = gpu.Engine(d, dtype="float32", max_tokens=300, page_size=16)
    for seq, want in ((toks, za), (other, zb)):
        eng.step([("s", seq[:100], [])])
        rows = [eng.step([("s", seq[i:i + 1], [0])]) for i in range(100, 124)]
        assert F.rel_err(rows[-1][0], want) < 3e-5
        eng.end("s")
    eng.close()


def test_a_kept_first_token_reaches_the_end_and_the_next_one_does_not(gpu, tmp_path):
    """One attention layer, window 10, three kept tokens: changing token 2 moves the last logits, changing token 3 leaves them."""
    cfg = F.config([F.layer("attention", F.attention(window=10, keep=3), 12)])
    d, W = F.make_model(str(tmp_path / "first"), cfg, seed=2, edit=lambda W: W["l0.shift"].fill(0.0))
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 90)
    eng = gpu.Engine(d, dtype="float32", max_tokens=300, page_size=4)

    def last(seq):
        eng.step([("s", seq[:70], [])])
        out = [eng.step([("s", seq[i:i + 1], [0])]) for i in range(70, 90)][-1][0]
        whole = eng.step([("w", seq, [89])], ["w"])[0]
        eng.end("s")
        assert F.rel_err(out, whole) < 3e-5 and F.rel_err(out, TP.forward(seq, W, cfg)[-1]) < 3e-5
        return out
    base = last(toks)
    for place, moves in ((2, True), (3, False), (79, False), (80, True)):  # the last query, 89, sees 80 .. 89
        seq = toks.copy()
        seq[place] = (seq[place] + 1) % cfg["vocab"]
        diff = np.abs(last(seq) - base).max()
        assert (diff > 1e-4) if moves else (diff < 1e-6), (place, diff)
    eng.close()


def test_random_weight_engine_portions_agree_at_sizes_that_reach_the_tensor_cores(gpu):
    cfg = F.config([F.layer("rglru", F.rglru(width=512, blocks=4, conv=4), 512),
                    F.layer("attention", F.attention(heads=8, kv_heads=2, dim=32, vdim=64, window=100, keep=4, dims=16), 512),
                    F.layer("latent_attention", F.latent(heads=6, dim=64, rot_dim=32, vdim=64, kv_rank=256, q_rank=192), 320)], vocab=500, width=384)
    toks = np.random.default_rng(0).integers(0, 500, 400)
    for dtype in ("bfloat16", "float32"):
        eng = gpu.Engine(config=cfg, seed=7, dtype=dtype, max_tokens=1024)
        whole = eng.step([("w", toks, np.arange(400))], ["w"])
        lo, rows = 0, []
        for c in [130, 2, 1, 1, 64, 200, 2]:
            rows.append(eng.step([("s", toks[lo:lo + c], np.arange(c))]))
            lo += c
        assert np.isfinite(whole).all() and close(np.concatenate(rows), whole, dtype, loose=2.0)
        eng.close()


def test_greedy_generation_through_the_engine(gpu, small):
    cfg, d, W, toks, _ = small
    eng = gpu.Engine(d, dtype="float32", max_tokens=128)
    prompt = toks[:12]
    out = eng.generate("g", prompt, 25)
    assert len(out) == 25 and eng.seq_len("g") == 12 + 24
    z = TP.forward(np.concatenate([prompt, out]), W, cfg)
    for i, t in enumerate(out):  # every chosen token is the oracle's maximum at its place (up to rounding between near-equal logits)
        row = z[len(prompt) - 1 + i]
        assert row[t] >= row.max() - 1e-4, i
    eng.end("g")
    assert eng.stats()["live_seqs"] == 0
    eng.close()


def test_the_command_line_programs_replay_a_trace_and_generate(gpu, small, tmp_path):
    """bin/trace_run as its user starts it: steps on standard input, logits in files, a line per step; two requests one after the
    other with the second one's id used again; bin/lm_generate gives the ids Engine.generate gives."""
    import json
    import os
    import subprocess
    import sys
    cfg, d, W, toks, want = small
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = str(tmp_path / "out")
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:40].tolist(), "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[40:42].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[42:43].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "a", "tokens": toks[:5].tolist(), "want": [4]}], "end": ["a"]}]
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out, "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [line for line in p.stdout.split("\n") if line.startswith("done")] == ["done %d" % i for i in range(4)]
    assert not os.path.exists(os.path.join(out, "1.f32"))
    got = {i: np.fromfile(os.path.join(out, "%d.f32" % i), dtype="<f4").reshape(-1, cfg["vocab"]) for i in (0, 2, 3)}
    assert close(got[0], want[[0, 39]], "float32") and close(got[2], want[[42]], "float32") and close(got[3], want[[4]], "float32")
    g = subprocess.run([sys.executable, os.path.join(root, "bin", "lm_generate"), "--model", d, "--dtype", "float32", "--prompt", ",".join(map(str, toks[:12])), "--new", "9"],
                       capture_output=True, text=True, timeout=600)
    assert g.returncode == 0, g.stderr[-2000:]
    eng = gpu.Engine(d, dtype="float32", max_tokens=128)
    assert [int(t) for t in g.stdout.strip().split("\n")[-1].split(",")] == eng.generate("g", toks[:12], 9).tolist()
    eng.close()
