"""Dapozen through the engine against the plain implementation (tests/plain_dapozen.py), on small configurations of the tests'
own (tests/dapozen_models.py) with weights drawn here: each mechanism alone, whole prompts, decoding token by token, prompts
cut into portions down to two tokens, batches of unequal requests, slots and pages used again, keys just inside and just outside
a run of positions and at page borders with a standout key, prompts around the chunks that the recurrence is computed in, the
first tokens of a sequence, pages given back behind a run, long decoding, and greedy generation through Engine.generate and the
command line.

float32 must agree with the plain implementation to summation order; bfloat16 is compared with a bound relative to the logits'
spread that a few rows may exceed (the experts of a token are its id's, so rounding cannot change them).
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import dapozen_models as models
import harness
import plain_dapozen as plain
import tiny_configs
from friday_inference_engine_b200 import Engine

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [pytest.param("float32", id="f32"), pytest.param("bfloat16", id="bf16")]
STANDOUT_TOKEN = 7

_made = {}


def model(root, name, standout=False):
    key = (str(root), name, standout)
    if key not in _made:
        cfg = models.CONFIGS[name]
        t = models.tensors_of(cfg, np.random.default_rng(models.SEEDS[name]))
        if standout:
            models.standout(cfg, t, STANDOUT_TOKEN)
        d = models.write_folder(os.path.join(str(root), "dapozen_%s_%d" % (name, standout)), cfg, t)
        _made[key] = (d,) + plain.load(d)
    return _made[key]


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("dapozen")


def engine(root, name, dtype, standout=False, **kw):
    d, cfg, t = model(root, name, standout)
    kw.setdefault("max_ctx", 1024)
    kw.setdefault("max_batch", 6)
    return Engine(model_path=d, dtype=dtype, **kw), cfg, t


_plain = {}


def plain_logits(root, name, prompt, standout=False):
    key = (str(root), name, tuple(prompt), standout)
    if key not in _plain:
        _, cfg, t = model(root, name, standout)
        _plain[key] = plain.forward(cfg, t, prompt)
    return _plain[key]


def compare(got, ref, places, dtype, what):
    got = np.asarray(got, dtype=np.float64)
    assert got.shape == (len(places), ref.shape[1]), what
    assert np.isfinite(got).all(), what
    if dtype == "float32":
        spread = np.sqrt((ref ** 2).mean())
        err = np.abs(got - ref[places]).max()
        assert err <= 1e-4 * max(spread, 1.0), "%s: |engine - plain| = %.3g (spread %.3g)" % (what, err, spread)
        return
    # Rounding alone moves a row in a hundred by more than the bound (heads divided by their root mean square make sharp scores, and a
    # sublayer's small result is normed to full size): a few rows may be over it, none by more than twice.  A key, a run's edge or a
    # state that is wrong moves its rows by several times that.
    over = []
    for i in range(len(places)):
        ok, text = harness.bf16_ok(got[i], ref[places[i]], what, harness.BF16_WIDE)
        if not ok:
            over.append("place %d: %s" % (places[i], text))
            twice, text = harness.bf16_ok(got[i], ref[places[i]], what, tuple(2.0 * x for x in harness.BF16_WIDE))
            assert twice, "%s, place %d: %s" % (what, places[i], text)
    assert len(over) <= max(1, len(places) // 40), "%s: %d of %d rows over the bound: %s" % (what, len(over), len(places), over[:4])


def agree(got, root, name, prompt, places, dtype, what, standout=False):
    compare(got, plain_logits(root, name, prompt, standout), places, dtype, what)


def prompts(lengths, vocab, seed, without=None):
    ps = tiny_configs.random_prompts(lengths, vocab, seed)
    if without is not None:
        ps = [[(tok + 1) % vocab if tok == without else tok for tok in p] for p in ps]
    return ps


def nothing_held(eng):
    st = eng.stats()
    return st["slots_held"] == 0 and all(g["pages_held"] == 0 for g in st["groups"])


# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["attention_only", "mamba2_only", "dense_only", "experts_only", "loop_only"])
def test_each_mechanism_alone(root, name, dtype):
    eng, cfg, _ = engine(root, name, dtype)
    for n, p in zip([1, 2, 40, 90], prompts([1, 2, 40, 90], cfg["vocab"], 3)):
        s = eng.alloc_slot()
        got = eng.step([s], [p], [list(range(n))], to="host")
        eng.free_slot(s)
        agree(got, root, name, p, list(range(n)), dtype, "%s alone, %d tokens" % (name, n))
    eng.check()
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n", [("P", 150), ("Q", 70), ("R", 300), ("S", 200), ("T", 130), ("U", 400), ("V", 100), ("long", 500)])
def test_whole_prompt(root, name, n, dtype):
    eng, cfg, _ = engine(root, name, dtype)
    (p,) = prompts([n], cfg["vocab"], 5)
    s = eng.alloc_slot()
    got = eng.step([s], [p], [list(range(n))], to="host")
    eng.free_slot(s)
    agree(got, root, name, p, list(range(n)), dtype, "%s whole %d" % (name, n))
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [31, 32, 33, 63, 64, 65, 127, 128, 129, 255, 256, 257])
def test_prompts_around_chunks(root, n, dtype):
    """Lengths around the chunks that the recurrence is computed in (128 tokens), around the step that starts to use them, and
    around the runs of positions of the attention; then the sequence goes on from what was left."""
    eng, cfg, _ = engine(root, "R", dtype)
    (p,) = prompts([n + 5], cfg["vocab"], 15)
    s = eng.alloc_slot()
    got = [eng.step([s], [p[:n]], [list(range(n))], to="host")]
    for tok in p[n:]:
        got.append(eng.step([s], [[tok]], [[0]], to="host"))
    eng.free_slot(s)
    agree(np.concatenate(got), root, "R", p, list(range(n + 5)), dtype, "R, %d tokens and five more" % n)


MARKS = {"far": (200, [0, 1, 49, 50, 51, 63, 64, 99, 100, 127, 128, 149, 150, 151], [99, 100, 101, 149, 150, 151, 199]),
         "far_pages": (262, [0, 63, 64, 127, 128, 129, 191, 192, 254, 255, 256], [127, 128, 129, 255, 256, 261])}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mode", ["whole", "decode", "portions"])
@pytest.mark.parametrize("name", ["far", "far_pages"])
def test_edges_of_a_run_with_a_standout_key(root, name, mode, dtype):
    """One token whose key outweighs all others, at the first and last places of the runs and of the pages; asked at the last row
    of a run and the first rows of the next, in prompts, in decoding and in portions that begin anywhere."""
    n, marks, asking = MARKS[name]
    size = models.CONFIGS[name]["layers"][0]["mixer"]["mask"]["size"]
    eng, cfg, t = engine(root, name, dtype, standout=True, max_batch=2)
    (base,) = prompts([n], cfg["vocab"], 17, without=STANDOUT_TOKEN)
    without = plain_logits(root, name, base, True)
    for marked in marks:
        p = list(base)
        p[marked] = STANDOUT_TOKEN
        ref = plain_logits(root, name, p, True)
        s = eng.alloc_slot()
        first = asking[0] - 2
        if mode == "whole":
            got = eng.step([s], [p], [asking], to="host")
        elif mode == "decode":
            eng.step([s], [p[:first]], [[]], to="host")
            rows = {first + i: eng.step([s], [[tok]], [[0]], to="host") for i, tok in enumerate(p[first:])}
            got = np.concatenate([rows[a] for a in asking])
        else:
            at, rows, cuts = 0, {}, [2, 48, 3, 11, 2, 35, 17, 2, 2, 30, 19, 2, 33]
            while at < n:
                c = min(cuts.pop(0) if cuts else 23, n - at)
                out = eng.step([s], [p[at:at + c]], [list(range(c))], to="host")
                for i in range(c):
                    rows[at + i] = out[i:i + 1]
                at += c
            got = np.concatenate([rows[a] for a in asking])
        eng.free_slot(s)
        compare(got, ref, asking, dtype, "%s: marked token at %d, %s" % (name, marked, mode))
        # the marked token decides what the last row of its run says, and hardly touches the runs after the next
        spread = np.sqrt((without ** 2).mean())
        last = min(marked // size * size + size, n) - 1
        change = lambda row: np.sqrt(((ref[row] - without[row]) ** 2).mean())
        assert change(last) > 0.2 * spread, "the marked token at %d hardly matters at %d" % (marked, last)


def test_faults_would_show(root):
    """What the comparisons would see: the plain implementation with one mechanism changed a little differs from itself by far
    more than the float32 bound."""
    _, cfg, t = model(root, "P")
    (p,) = prompts([150], cfg["vocab"], 5)
    ref = plain_logits(root, "P", p)
    bound = 30 * 1e-4 * max(np.sqrt((ref ** 2).mean()), 1.0)

    def changed(**kw):
        c = json.loads(json.dumps(cfg))
        for path, v in kw.items():
            node, keys = c, path.split("__")
            for k in keys[:-1]:
                node = node[int(k)] if k.isdigit() else node[k]
            node[int(keys[-1]) if keys[-1].isdigit() else keys[-1]] = v
        return np.abs(plain.forward(c, t, p) - ref).max()

    def scaled(**kw):
        w = dict(t)
        for name, f in kw.items():
            w[name.replace("__", ".")] = f(w[name.replace("__", ".")])
        return np.abs(plain.forward(cfg, w, p) - ref).max()

    assert changed(layers__0__mixer__mask__size=11) > bound
    assert changed(layers__0__mixer__mask__size=9) > bound
    assert changed(layers__2__mixer__mask__size=38) > bound
    assert changed(layers__0__mixer__rot__dims=10) > bound
    assert changed(layers__0__mixer__rot__base=9000.0) > bound
    assert changed(layers__1__mlp__expert__limit=0.85) > bound
    assert changed(layers__1__mlp__shared__limit=1.4) > bound
    assert changed(layers__1__mixer__norm_groups=2) > bound
    assert changed(embedding__scale=2.55) > bound
    assert changed(norm__eps=3e-3) > bound
    assert changed(logit_softcap=12.5) > bound
    assert changed(loop__times=3) > bound
    assert scaled(l0__mix__q__conv=lambda x: x[:, [0, 0, 2, 3]]) > bound
    assert scaled(l1__mix__conv=lambda x: x * np.array([0.0, 1.0, 1.0])) > bound
    assert scaled(l1__mix__D=lambda x: 0.9 * x) > bound
    assert scaled(l1__mix__dt_bias=lambda x: x + 0.05) > bound
    assert scaled(l3__mix__A_log=lambda x: x + 0.1) > bound
    assert scaled(l2__mix__g=lambda x: 0.0 * x) > bound
    assert scaled(l1__mlp__table=lambda x: (x + 1) % 6) > bound
    assert np.abs(plain.forward(cfg, t, [p[0]] + p[2:])[-1] - ref[-1]).max() > bound
    late = plain.forward(cfg, t, p[100:])                       # state lost
    assert np.abs(late[-1] - ref[-1]).max() > bound


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "R", "S", "T", "U", "V"])
def test_prompt_then_token_by_token(root, name, dtype):
    eng, cfg, _ = engine(root, name, dtype)
    n, tail = (330, 150) if name == "R" else (110, 60)
    (p,) = prompts([n], cfg["vocab"], 6)
    s = eng.alloc_slot()
    got = [eng.step([s], [p[:n - tail]], [[n - tail - 1]], to="host")]
    for i in range(n - tail, n):
        got.append(eng.step([s], [[p[i]]], [[0]], to="host"))
    eng.free_slot(s)
    agree(np.concatenate(got), root, name, p, list(range(n - tail - 1, n)), dtype, "%s decode" % name)
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "S", "T"])
def test_all_tokens_one_by_one(root, name, dtype):
    """From the very first token: states and convolutions start at zero."""
    eng, cfg, _ = engine(root, name, dtype)
    (p,) = prompts([90], cfg["vocab"], 7)
    s = eng.alloc_slot()
    got = [eng.step([s], [[tok]], [[0]], to="host") for tok in p]
    eng.free_slot(s)
    agree(np.concatenate(got), root, name, p, list(range(90)), dtype, "%s one by one" % name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,cuts", [("P", [2, 3, 7, 64, 65, 9, 1, 1, 2]), ("R", [64, 2, 128, 100, 6]), ("Q", [1, 2, 30, 37, 3]),
                                       ("S", [5, 64, 3, 70, 2, 2]), ("T", [3, 2, 40, 1, 5, 66, 2]), ("U", [2, 130, 33, 2, 50]), ("V", [2, 2, 40, 30])])
def test_portions(root, name, cuts, dtype):
    eng, cfg, _ = engine(root, name, dtype)
    n = sum(cuts)
    (p,) = prompts([n], cfg["vocab"], 8)
    s = eng.alloc_slot()
    got, at = [], 0
    for c in cuts:
        got.append(eng.step([s], [p[at:at + c]], [list(range(c))], to="host"))
        at += c
    eng.free_slot(s)
    agree(np.concatenate(got), root, name, p, list(range(n)), dtype, "%s portions %s" % (name, cuts))


@pytest.mark.parametrize("dtype", DTYPES)
def test_passes_of_the_step_function(root, dtype):
    """A prompt longer than the step function's pass: states, histories and cache go from pass to pass."""
    eng, cfg, _ = engine(root, "R", dtype, prefill_chunk=64)
    (p,) = prompts([300], cfg["vocab"], 9)
    s = eng.alloc_slot()
    got = eng.step([s], [p], [list(range(300))], to="host")
    eng.free_slot(s)
    agree(got, root, "R", p, list(range(300)), dtype, "R in passes of 64")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "R", "T"])
def test_batch_of_unequal_requests(root, name, dtype):
    """Requests of different lengths in one batch (one of a single token, one shorter than a convolution), then decoded together;
    the shorter ones end earlier.  Every request must come out as it does alone."""
    eng, cfg, _ = engine(root, name, dtype)
    lengths = {"P": [1, 70, 131, 40, 2], "R": [1, 200, 90, 3], "T": [2, 1, 77]}[name]
    tail = 20
    ps = prompts([n + tail for n in lengths], cfg["vocab"], 10)
    slots = [eng.alloc_slot() for _ in ps]
    got = {i: [] for i in range(len(ps))}
    first = eng.step(slots, [p[:n] for p, n in zip(ps, lengths)], [[n - 1] for n in lengths], to="host")
    for i in range(len(ps)):
        got[i].append(first[i:i + 1])
    live = list(range(len(ps)))
    for k in range(tail):
        if k == 7:
            eng.free_slot(slots[live.pop(0)])               # the first request ends early
        out = eng.step([slots[i] for i in live], [[ps[i][lengths[i] + k]] for i in live], [[0]] * len(live), to="host")
        for j, i in enumerate(live):
            got[i].append(out[j:j + 1])
    for i in live:
        eng.free_slot(slots[i])
    for i, p in enumerate(ps):
        n = lengths[i]
        places = list(range(n - 1, n - 1 + len(got[i])))
        agree(np.concatenate(got[i]), root, name, p, places, dtype, "%s request %d of a batch" % (name, i))
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_beside_single_tokens(root, dtype):
    """One step that brings one token of one request and many of others: the states of all move on by what each brought."""
    eng, cfg, _ = engine(root, "R", dtype)
    a, b, c = prompts([150, 150, 150], cfg["vocab"], 20)
    s = [eng.alloc_slot() for _ in range(3)]
    got = [[], [], []]
    at = [0, 0, 0]
    for take in ([40, 2, 1], [1, 70, 3], [2, 1, 130], [1, 1, 1], [106, 76, 15]):
        out = eng.step(s, [p[k:k + n] for p, k, n in zip((a, b, c), at, take)], [list(range(n)) for n in take], to="host")
        row = 0
        for i, n in enumerate(take):
            got[i].append(out[row:row + n])
            row += n
            at[i] += n
    for i, p in enumerate((a, b, c)):
        eng.free_slot(s[i])
        agree(np.concatenate(got[i]), root, "R", p, list(range(150)), dtype, "R, request %d of a mixed batch" % i)


@pytest.mark.parametrize("form", ["grouped", "dense", "pairs"])
def test_forms_of_the_experts(root, form, monkeypatch):
    """The three ways a prompt's rows can run through the experts that the table gives them."""
    monkeypatch.setenv("FRIDAY_EXPERTS", form)
    eng, cfg, _ = engine(root, "R", "bfloat16")
    ps = prompts([150, 33], cfg["vocab"], 18)
    slots = [eng.alloc_slot() for _ in ps]
    got = eng.step(slots, ps, [list(range(len(p))) for p in ps], to="host")
    at = 0
    for s, p in zip(slots, ps):
        eng.free_slot(s)
        agree(got[at:at + len(p)], root, "R", p, list(range(len(p))), "bfloat16", "R, experts %s" % form)
        at += len(p)


@pytest.mark.parametrize("switch", ["FRIDAY_POOLED_TCGEN05", "FRIDAY_POOLED_TC", "FRIDAY_POOLED_MMA", "FRIDAY_SSD_CHUNKS"])
@pytest.mark.parametrize("name", ["R", "U"])
def test_other_kernels_say_the_same(root, name, switch, monkeypatch):
    """The kernels that serve other sizes, on sizes that a faster one would take."""
    monkeypatch.setenv(switch, "0")
    if switch == "FRIDAY_POOLED_TC":
        monkeypatch.setenv("FRIDAY_POOLED_TCGEN05", "0")
    eng, cfg, _ = engine(root, name, "bfloat16")
    (p,) = prompts([230], cfg["vocab"], 22)
    s = eng.alloc_slot()
    got = [eng.step([s], [p[:200]], [list(range(200))], to="host")]
    got += [eng.step([s], [[tok]], [[0]], to="host") for tok in p[200:]]
    eng.free_slot(s)
    agree(np.concatenate(got), root, name, p, list(range(230)), "bfloat16", "%s with %s=0" % (name, switch))


@pytest.mark.parametrize("splits", ["1", "2", "5", "8", "11"])
def test_one_token_steps_in_splits(root, splits, monkeypatch):
    """A sequence's keys shared among CTAs, as a cluster and through memory, some of them with no key at all: gates join once,
    whoever merges, and a run's first key is the first for all."""
    monkeypatch.setenv("FRIDAY_ATTN_SPLITS", splits)
    eng, cfg, _ = engine(root, "long", "bfloat16")
    ps = prompts([390, 40], cfg["vocab"], 19)
    slots = [eng.alloc_slot() for _ in ps]
    eng.step(slots, [p[:-8] for p in ps], [[], []], to="host")
    got = [eng.step(slots, [[p[len(p) - 8 + k]] for p in ps], [[0], [0]], to="host") for k in range(8)]
    for i, p in enumerate(ps):
        eng.free_slot(slots[i])
        agree(np.stack([g[i] for g in got]), root, "long", p, list(range(len(p) - 8, len(p))), "bfloat16", "in %s splits, request %d" % (splits, i))
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_used_again(root, dtype):
    """A slot that held a long request is given to a short one: states and histories start anew, stale pages are not read."""
    eng, cfg, _ = engine(root, "P", dtype, max_batch=2, max_ctx=256, max_tokens=512)
    a, b, c, d = prompts([200, 30, 90, 1], cfg["vocab"], 11)
    for p in (a, b, c, d, b):
        s = eng.alloc_slot()
        got = eng.step([s], [p], [list(range(len(p)))], to="host")
        eng.free_slot(s)
        agree(got, root, "P", p, list(range(len(p))), dtype, "P in a slot used before (%d tokens)" % len(p))
    s1, s2 = eng.alloc_slot(), eng.alloc_slot()
    g1 = eng.step([s1, s2], [c[:50], b], [[49], [len(b) - 1]], to="host")
    g2 = eng.step([s1], [c[50:]], [list(range(40))], to="host")
    eng.free_slot(s1)
    eng.free_slot(s2)
    agree(np.concatenate([g1[:1], g2]), root, "P", c, [49] + list(range(50, 90)), dtype, "P cut in two, in a used slot")
    agree(g1[1:], root, "P", b, [len(b) - 1], dtype, "P beside it")
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_go_back_behind_a_run(root, dtype):
    """Two requests take turns and give back the pages of the runs they have left: each takes pages that the other filled, and a
    sequence holds no more than its run's pages."""
    eng, cfg, _ = engine(root, "long", dtype, max_batch=2, max_ctx=1024, max_tokens=2048)
    ps = prompts([700, 700], cfg["vocab"], 21)
    slots = [eng.alloc_slot() for _ in ps]
    got, at = [[], []], 0
    while at < 700:
        c = min(96 if at < 600 else 5, 700 - at)
        for i in (0, 1):
            got[i].append(eng.step([slots[i]], [ps[i][at:at + c]], [[0, c - 1]], to="host"))
        at += c
        (group,) = eng.stats()["groups"]
        assert group["pages_held"] <= 2 * 3, "%d pages held at %d tokens" % (group["pages_held"], at)
    for i in (0, 1):
        eng.free_slot(slots[i])
        places, at = [], 0
        while at < 700:
            c = min(96 if at < 600 else 5, 700 - at)
            places += [at, at + c - 1]
            at += c
        agree(np.concatenate(got[i]), root, "long", ps[i], places, dtype, "request %d of two that take turns" % i)
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(root, dtype):
    """Hundreds of single-token steps, through the ends of several runs: the states run on."""
    eng, cfg, _ = engine(root, "long", dtype)
    (p,) = prompts([10 + 420], cfg["vocab"], 12)
    s = eng.alloc_slot()
    eng.step([s], [p[:10]], [[]], to="host")
    got = [eng.step([s], [[tok]], [[0]], to="host") for tok in p[10:]]
    eng.free_slot(s)
    agree(np.concatenate(got), root, "long", p, list(range(10, 430)), dtype, "long decoding")


@pytest.mark.parametrize("name", ["P", "R"])
def test_greedy_generation(root, name):
    """Engine.generate (the library's scheduler, its decoder with captured steps, its sampler) chooses the tokens that the
    plain implementation chooses."""
    eng, cfg, t = engine(root, name, "float32", max_batch=3)
    ps = prompts([5, 23, 64, 9], cfg["vocab"], 13)
    out = eng.generate(ps, max_new_tokens=12, temperature=0.0, ignore_eos=True)
    for p, g in zip(ps, out):
        want = plain.greedy(cfg, t, p, 12)
        for i, (a, b) in enumerate(zip(g.tokens, want)):
            if a != b:
                lg = plain.forward(cfg, t, p + want[:i])[-1]
                top2 = np.sort(lg)[-2:]
                assert top2[1] - top2[0] < 1e-4, "%s: token %d is %d, plain chooses %d" % (name, i, a, b)
                break
    assert nothing_held(eng)


def test_bf16_generation_follows_the_step_function(root):
    """Captured one-token steps in bfloat16, over the end of a run of positions: every chosen token is the largest logit that the step
    function gives for the same tokens, or within rounding of it; and generating again repeats it."""
    eng, cfg, _ = engine(root, "R", "bfloat16", max_batch=4)
    ps = prompts([5, 23, 60, 95], cfg["vocab"], 14)
    a = eng.generate(ps, max_new_tokens=20, temperature=0.0, ignore_eos=True)
    b = eng.generate(ps, max_new_tokens=20, temperature=0.0, ignore_eos=True)
    assert [g.tokens for g in a] == [g.tokens for g in b]
    for p, g in zip(ps, a):
        assert len(g.tokens) == 20
        s = eng.alloc_slot()
        rows = eng.step([s], [p + g.tokens[:-1]], [list(range(len(p) - 1, len(p) + 19))], to="host")
        eng.free_slot(s)
        spread = np.sqrt((np.asarray(rows, dtype=np.float64) ** 2).mean())
        for row, tok in zip(rows, g.tokens):
            assert row.max() - row[tok] < 0.15 * spread
    assert nothing_held(eng)


def test_random_weights_draw_a_table(root):
    """Without a checkpoint: seeded weights, and a table whose rows differ and name every expert."""
    eng = Engine(config=models.CONFIGS["R"], seed=3, dtype="bfloat16", max_ctx=256, max_batch=2)
    out = eng.generate(prompts([40, 9], 512, 23), max_new_tokens=5, temperature=0.0, ignore_eos=True)
    assert all(len(g.tokens) == 5 for g in out)
    assert nothing_held(eng)


def test_the_command_line_generates(root):
    """bin/friday serves the design like any other: the folder's config.json names it."""
    d, cfg, t = model(root, "P")
    (p,) = prompts([20], cfg["vocab"], 16)
    out = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "friday"), d, "--dtype", "float32", "--ctx", "128", "--json", "--ignore-eos",
                          "--max-new-tokens", "6", "--prompt-ids", ",".join(map(str, p))], capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    tokens = json.loads(out.stdout.strip().splitlines()[-1])["tokens"]
    eng, _, _ = engine(root, "P", "float32")
    assert tokens == eng.generate([p], max_new_tokens=6, temperature=0.0, ignore_eos=True)[0].tokens
