"""Fekopel through the serving engine against the plain numpy oracle (tests/fekopel_plain.py): whole prompts and every layer run,
portions down to two tokens, token-by-token decoding, several live sequences of unequal length, slots and pages that are freed and
used again (also by the same sequence, behind its windows), the first tokens of a sequence, long decoding, other sizes and
optional parts, and greedy generation through the engine's own entry point."""
import numpy as np
import pytest

import fekopel_fixture as F
import fekopel_plain as FP
from safolorn_fixture import close_enough as mostly_close  # leaves room for a router's close call in bfloat16

pytestmark = pytest.mark.gpu


def make(tmp_path_factory, cfg, seed, n):
    d, W = F.make_model(str(tmp_path_factory.mktemp("fk") / "m"), cfg, seed=seed)
    toks = F.settled_tokens(cfg, W, n, 5)
    return cfg, d, W, toks, FP.forward(toks, W, cfg)


@pytest.fixture(scope="module")
def small(gpu, tmp_path_factory):
    return make(tmp_path_factory, F.small_config(), 11, 150)


@pytest.fixture(scope="module")
def windowed(gpu, tmp_path_factory):
    return make(tmp_path_factory, F.windowed_config(), 12, 150)


def in_cuts(eng, name, toks, cuts):
    lo, rows = 0, []
    for c in cuts:
        rows.append(eng.step([(name, toks[lo:lo + c], np.arange(c))]))
        lo += c
    return np.concatenate(rows)


@pytest.mark.parametrize("model", ["small", "windowed"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_and_every_layer_run(gpu, request, model, dtype):
    cfg, d, W, toks, want = request.getfixturevalue(model)
    eng = gpu.Engine(d, dtype=dtype, max_tokens=256, page_size=16)
    assert eng.architecture == "Fekopel"
    eng.capture(True)
    got = eng.step([("a", toks, np.arange(len(toks)))], ["a"])
    assert F.close_enough(got, want, dtype)
    xs = []
    FP.forward(toks, W, cfg, xs)
    assert len(xs) == {"small": 8, "windowed": 5}[model]
    for i, x in enumerate(xs):
        assert F.close_enough(eng.captured(i, len(toks), cfg["width"]), x, dtype), i
    assert eng.stats()["live_seqs"] == 0 and eng.stats()["free_pages"] == eng.stats()["pages"]
    eng.capture(False)  # the same numbers when nothing is captured
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
        n = sum(cuts)
        got = in_cuts(eng, "s", toks, cuts)
        assert F.close_enough(got, want[:n], dtype), cuts[:3]
        eng.end("s")
        whole = eng.step([("w", toks[:n], np.arange(n))], ["w"])
        assert F.close_enough(got, whole, dtype), cuts[:3]
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_several_sequences_reused_slots_and_first_tokens(gpu, small, dtype):
    cfg, d, W, toks, want = small
    seqs = {k: F.settled_tokens(cfg, W, n, n) for k, n in (("a", 70), ("b", 9), ("c", 33), ("d", 50), ("e", 1), ("f", 3))}
    alone = {k: FP.forward(v, W, cfg) for k, v in seqs.items()}
    eng = gpu.Engine(d, dtype=dtype, max_tokens=140, page_size=8, max_seqs=3)
    got, at = {k: [] for k in seqs}, {k: 0 for k in seqs}

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
    feed(("d", 1), ("e", 1), end=["e"])                    # d and e start in slots and pages that b and c used
    feed(("a", 37), ("d", 2), ("f", 3), end=["a", "f"])
    feed(("d", 47), end=["d"])
    for k in seqs:
        assert at[k] == len(seqs[k]) and F.close_enough(np.concatenate(got[k]), alone[k], dtype), k
    st = eng.stats()
    assert st["live_seqs"] == 0 and st["free_pages"] == st["pages"] and free_mid < st["pages"]
    with pytest.raises(gpu.GgbError):  # a fourth live sequence has no slot
        eng.step([(k, [1], []) for k in "wxyz"])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_behind_the_windows_are_used_again_and_the_first_tokens_stay(gpu, windowed, dtype):
    cfg, d, W, toks, want = windowed   # the widest window has 13 positions, 6 first tokens are kept: with pages of 4 the first two stay
    other = F.settled_tokens(cfg, W, 150, 6)
    want_other = FP.forward(other, W, cfg)
    eng = gpu.Engine(d, dtype=dtype, max_tokens=150, page_size=4, max_seqs=2)
    lo, rows, rows_o = 0, [], []
    for c in [9, 1, 1, 7, 16, 2, 2, 1, 16, 13, 1, 1, 1, 16, 3, 16, 16, 12, 2, 14]:
        out = eng.step([("s", toks[lo:lo + c], np.arange(c)), ("o", other[lo:lo + c], np.arange(c))])
        rows.append(out[:c])
        rows_o.append(out[c:])
        lo += c
        assert eng.seq_live_pages("s") <= 13 // 4 + 2 + 2 and eng.seq_live_pages("o") <= 13 // 4 + 2 + 2
    assert lo == 150 and F.close_enough(np.concatenate(rows), want, dtype) and F.close_enough(np.concatenate(rows_o), want_other, dtype)
    pages = eng.seq_pages("s")
    assert len(pages) == (150 + 3) // 4 and (pages >= 0).sum() == eng.seq_live_pages("s") and (pages[:2] >= 0).all() and pages[2] < 0
    eng.end("s", "o")
    assert eng.stats()["free_pages"] == eng.stats()["pages"]
    eng.close()


def test_a_layer_that_sees_everything_keeps_every_page(gpu, small):
    cfg, d, W, toks, want = small
    eng = gpu.Engine(d, dtype="float32", max_tokens=16, page_size=4, max_seqs=2)
    eng.step([("s", toks[:20], [19])])
    assert eng.seq_live_pages("s") == 5
    with pytest.raises(gpu.GgbError, match="out of pages"):
        eng.step([("t", toks[:8], [])])
    eng.close()


def test_long_decoding(gpu, small):
    cfg, d, W, toks, _ = small
    long = F.settled_tokens(cfg, W, 330, 2)
    want = FP.forward(long, W, cfg)
    for dtype in ("float32", "bfloat16"):
        eng = gpu.Engine(d, dtype=dtype, max_tokens=400, page_size=32)
        rows = in_cuts(eng, "s", long, [10] + [1] * 320)
        assert F.close_enough(rows, want, dtype)
        eng.use_graphs(False)  # launches one by one: the same numbers as the replayed step
        eng.end("s")
        assert np.abs(in_cuts(eng, "s", long, [10] + [1] * 50) - rows[:60]).max() < 1e-3
        eng.close()


OTHER = {
    # what the small configurations have unequal or larger: equal or 1; what they have, absent
    "equal_and_absent": lambda: F.config([F.attn2(F.gated(heads=2, kv_heads=2, dim=8, vdim=8, window=0, softcap=0, base=0), F.moe(experts=2, top=2, ff=16, groups=0, shared=16)),
                                          F.attn(F.sink(heads=2, kv_heads=2, dim=8, vdim=8, window=0))], vocab=16, width=16),
    "ones": lambda: F.config([F.attn(F.sink(heads=1, kv_heads=1, dim=1, vdim=2, window=1), F.moe(experts=1, top=1, ff=1, groups=1, keep=1, shared=1)),
                              F.attn2(F.gated(heads=1, kv_heads=1, dim=2, vdim=2, window=1, keep=1, dims=2), F.moe(experts=3, top=1, ff=2, groups=3, keep=1, shared=0))],
                             vocab=30, width=7, loop=(0, 1, 1)),
    "whole_stack_loops": lambda: F.config([F.attn(mlp=F.moe()), F.attn2()], vocab=41, width=24, loop=(0, 2, 4)),
    "last_layer_loops": lambda: F.config([F.attn2(), F.attn(mlp=F.moe(shared=0)), F.attn(F.sink(window=30), F.moe(groups=0, scale=0.3))], vocab=41, width=20, loop=(2, 3, 3)),
    "only_attention_2": lambda: F.config([F.attn2(F.gated(heads=6, kv_heads=1, dim=4, vdim=14, window=100, keep=50, dims=4)), F.attn2(F.gated(window=1, keep=0), F.moe())], width=12),
    # 16-byte pieces everywhere, tensor-core products and experts, kept tokens over more than one tile, wide values
    "wide": lambda: F.config([F.attn2(F.gated(heads=4, kv_heads=2, dim=32, vdim=64, window=45, keep=37, dims=16), F.moe(experts=16, top=4, ff=64, groups=4, keep=2, shared=192)),
                              F.attn(F.sink(heads=8, kv_heads=2, dim=64, vdim=32, window=64), F.moe(experts=8, top=4, ff=128, groups=2, keep=1, shared=64)),
                              F.attn2(F.gated(heads=2, kv_heads=1, dim=64, vdim=160, window=80, keep=1, dims=64))], vocab=200, width=128, loop=(1, 2, 2)),
}


@pytest.mark.parametrize("name", sorted(OTHER))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes_and_optional_parts(gpu, tmp_path, name, dtype):
    cfg = OTHER[name]()
    d, W = F.make_model(str(tmp_path / name), cfg, seed=3)
    toks = F.settled_tokens(cfg, W, 140, 4)
    want = FP.forward(toks, W, cfg)
    # a unit head of one number is a sign: rounding shows more there
    loose = 8.0 if name == "ones" else 2.0
    eng = gpu.Engine(d, dtype=dtype, max_tokens=300, page_size=16)
    assert F.close_enough(eng.step([("w", toks, np.arange(140))], ["w"]), want, dtype, loose)
    assert F.close_enough(in_cuts(eng, "s", toks, [2, 2, 65, 1, 1, 3, 64, 2]), want, dtype, loose)
    eng.close()


def last_logits(eng, seq, split):
    """the last token's logits after a portion and single tokens, checked against the whole prompt at once"""
    eng.step([("s", seq[:split], [])])
    out = [eng.step([("s", seq[i:i + 1], [0])]) for i in range(split, len(seq))][-1][0]
    whole = eng.step([("w", seq, [len(seq) - 1])], ["w"])[0]
    eng.end("s")
    assert F.rel_err(out, whole) < 3e-5
    return out


@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_a_token_at_the_windows_edge_and_the_first_tokens_reach_the_end(gpu, tmp_path, kind):
    """One layer with a window of 10 (attention_2 keeps three tokens): changing a token that the last query sees moves its logits,
    changing any other leaves them as they were."""
    mixer = F.sink(window=10) if kind == "attention" else F.gated(window=10, keep=3)
    cfg = F.config([{"type": kind, "mixer": mixer, "mlp": None}])
    d, W = F.make_model(str(tmp_path / "edge"), cfg, seed=2)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 90)
    eng = gpu.Engine(d, dtype="float32", max_tokens=300, page_size=4)
    base = last_logits(eng, toks, 70)
    assert F.rel_err(base, FP.forward(toks, W, cfg)[-1]) < 3e-5
    kept = kind == "attention_2"
    for place, moves in ((0, kept), (2, kept), (3, False), (40, False), (79, False), (80, True), (89, True)):  # the last query, 89, sees 80 .. 89
        seq = toks.copy()
        seq[place] = (seq[place] + 1) % cfg["vocab"]
        got = last_logits(eng, seq, 70)
        assert F.rel_err(got, FP.forward(seq, W, cfg)[-1]) < 3e-5
        diff = np.abs(got - base).max()
        assert (diff > 1e-4) if moves else (diff < 1e-6), (place, diff)
    eng.close()


def test_every_pass_of_a_looped_layer_reads_its_own_cache(gpu, tmp_path):
    """Two passes over one layer with a window of 6: a token 10 back reaches the end only through what the first pass left in the second
    one's rows; with rows mixed up between the passes the decoded tokens would not agree with the oracle."""
    cfg = F.config([F.attn(F.sink(window=6, scale=0.05), F.moe(experts=2, top=1, groups=0))], loop=(0, 1, 2))
    d, W = F.make_model(str(tmp_path / "loop"), cfg, seed=6, edit=lambda W: W["loop.step"].__imul__(3.0))
    toks = np.random.default_rng(3).integers(0, cfg["vocab"], 60)
    eng = gpu.Engine(d, dtype="float32", max_tokens=200, page_size=4)
    base = last_logits(eng, toks, 30)
    for place, moves in ((49, True), (48, False), (54, True)):  # 59 sees 54 .. 59, each of which saw five more in the first pass
        seq = toks.copy()
        seq[place] = (seq[place] + 1) % cfg["vocab"]
        got = last_logits(eng, seq, 30)
        assert F.rel_err(got, FP.forward(seq, W, cfg)[-1]) < 3e-5
        assert (np.abs(got - base).max() > 1e-5) == moves, place
    eng.close()


def test_random_weight_engine_portions_agree_at_sizes_that_reach_the_tensor_cores(gpu):
    cfg = F.config([F.attn2(F.gated(heads=8, kv_heads=2, dim=64, vdim=64, window=100, keep=4, scale=0.125, softcap=20.0, dims=32), F.moe(experts=16, top=4, ff=128, groups=4, keep=2, shared=320)),
                    F.attn(F.sink(heads=6, kv_heads=3, dim=64, vdim=96, window=70, scale=0.125), F.moe(experts=8, top=2, ff=256, groups=0, shared=64))], vocab=500, width=384, loop=(1, 2, 2))
    toks = np.random.default_rng(0).integers(0, 500, 400)
    for dtype in ("bfloat16", "float32"):
        eng = gpu.Engine(config=cfg, seed=7, dtype=dtype, max_tokens=1024)
        whole = eng.step([("w", toks, np.arange(400))], ["w"])
        assert np.isfinite(whole).all() and mostly_close(in_cuts(eng, "s", toks, [130, 2, 1, 1, 64, 200, 2]), whole, dtype, loose=2.0)
        eng.close()


def test_greedy_generation_through_the_engine(gpu, small):
    cfg, d, W, toks, _ = small
    eng = gpu.Engine(d, dtype="float32", max_tokens=128)
    prompt = toks[:12]
    out = eng.generate("g", prompt, 25)
    assert len(out) == 25 and eng.seq_len("g") == 12 + 24
    z = FP.forward(np.concatenate([prompt, out]), W, cfg)
    for i, t in enumerate(out):  # every chosen token is the oracle's maximum at its place (up to rounding between near-equal logits)
        row = z[len(prompt) - 1 + i]
        assert row[t] >= row.max() - 1e-4, i
    eng.end("g")
    assert eng.stats()["live_seqs"] == 0
    eng.close()


def test_the_command_line_programs_replay_a_trace_and_generate(gpu, small, tmp_path):
    """bin/trace_run as its user starts it, two requests one after the other with an id used again; bin/lm_generate gives the ids
    Engine.generate gives."""
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
    got = {i: np.fromfile(os.path.join(out, "%d.f32" % i), dtype="<f4").reshape(-1, cfg["vocab"]) for i in (0, 2, 3)}
    assert not os.path.exists(os.path.join(out, "1.f32"))
    assert F.close_enough(got[0], want[[0, 39]], "float32") and F.close_enough(got[2], want[[42]], "float32") and F.close_enough(got[3], want[[4]], "float32")
    g = subprocess.run([sys.executable, os.path.join(root, "bin", "lm_generate"), "--model", d, "--dtype", "float32", "--prompt", ",".join(map(str, toks[:12])), "--new", "9"],
                       capture_output=True, text=True, timeout=600)
    assert g.returncode == 0, g.stderr[-2000:]
    eng = gpu.Engine(d, dtype="float32", max_tokens=128)
    assert [int(t) for t in g.stdout.strip().split("\n")[-1].split(",")] == eng.generate("g", toks[:12], 9).tolist()
    eng.close()
