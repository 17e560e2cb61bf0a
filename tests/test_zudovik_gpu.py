"""Zudovik through the engine against the plain implementation (tests/plain_zudovik.py), on small configurations of the tests'
own (tests/zudovik_models.py) with weights drawn here: each mechanism alone, whole prompts, decoding token by token, prompts
cut into portions down to two tokens, batches of unequal requests, slots and pages used again, keys far away and at page
borders with a standout key (also through a layer that reads another's keys), prompts around the chunks of the linear
attention, the first tokens of a sequence, long decoding, and greedy generation through Engine.generate and the command line.

float32 must agree with the plain implementation to summation order.  In bfloat16 a router's close call can go the other
way, and another expert is another function, not a rounding: the bfloat16 runs use folders whose corrections lie far apart,
and are compared with a bound relative to the logits' spread.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import harness
import plain_zudovik as plain
import tiny_configs
import zudovik_models as models
from friday_inference_engine_b200 import Engine

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [pytest.param("float32", id="f32"), pytest.param("bfloat16", id="bf16")]
STANDOUT_TOKEN = 7

_made = {}


def model(root, name, dtype, standout=False):
    clear = dtype != "float32"
    key = (str(root), name, clear, standout)
    if key not in _made:
        cfg = models.CONFIGS[name]
        t = models.tensors_of(cfg, np.random.default_rng(models.SEEDS[name]), clear_routing=clear)
        if standout:
            models.standout(cfg, t, STANDOUT_TOKEN)
        d = models.write_folder(os.path.join(str(root), "zudovik_%s_%d_%d" % (name, clear, standout)), cfg, t)
        _made[key] = (d,) + plain.load(d)
    return _made[key]


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("zudovik")


def engine(root, name, dtype, standout=False, **kw):
    d, cfg, t = model(root, name, dtype, standout)
    kw.setdefault("max_ctx", 1024)
    kw.setdefault("max_batch", 6)
    return Engine(model_path=d, dtype=dtype, **kw), cfg, t


_plain = {}


def plain_logits(root, name, prompt, dtype, standout=False):
    key = (str(root), name, tuple(prompt), dtype != "float32", standout)
    if key not in _plain:
        _, cfg, t = model(root, name, dtype, standout)
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
    for i in range(len(places)):
        ok, text = harness.bf16_ok(got[i], ref[places[i]], what, harness.BF16_WIDE)
        assert ok, "%s, place %d: %s" % (what, places[i], text)


def agree(got, root, name, prompt, places, dtype, what, standout=False):
    compare(got, plain_logits(root, name, prompt, dtype, standout), places, dtype, what)


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
@pytest.mark.parametrize("name", ["attention_only", "shared_keys_only", "lightning_only", "dense_only", "experts_only"])
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
@pytest.mark.parametrize("name,n", [("P", 150), ("Q", 70), ("R", 300), ("S", 200), ("T", 130), ("U", 260), ("V", 100)])
def test_whole_prompt(root, name, n, dtype):
    eng, cfg, _ = engine(root, name, dtype)
    (p,) = prompts([n], cfg["vocab"], 5)
    s = eng.alloc_slot()
    got = eng.step([s], [p], [list(range(n))], to="host")
    eng.free_slot(s)
    agree(got, root, name, p, list(range(n)), dtype, "%s whole %d" % (name, n))
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [31, 32, 33, 63, 64, 65, 127, 128, 129])
def test_prompts_around_chunks(root, n, dtype):
    """Lengths around the chunks of the linear attention (64 tokens) and around the step that starts to use them; then the
    sequence goes on from the state that was left."""
    eng, cfg, _ = engine(root, "R", dtype)
    (p,) = prompts([n + 3], cfg["vocab"], 15)
    s = eng.alloc_slot()
    got = [eng.step([s], [p[:n]], [list(range(n))], to="host")]
    for tok in p[n:]:
        got.append(eng.step([s], [[tok]], [[0]], to="host"))
    eng.free_slot(s)
    agree(np.concatenate(got), root, "R", p, list(range(n + 3)), dtype, "R, %d tokens and three more" % n)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mode", ["whole", "decode", "portions"])
def test_far_keys_with_a_standout_key(root, mode, dtype):
    """One token whose key outweighs all others, at the first places, at page borders, far back and right before the asking
    rows: in prompts, in decoding and in portions; the layers that read those keys later see it as well."""
    n, ask = 200, 150
    asking = [ask, ask + 1, n - 1]
    eng, cfg, t = engine(root, "far", dtype, standout=True, max_batch=2)
    (base,) = prompts([n], cfg["vocab"], 17, without=STANDOUT_TOKEN)
    without = plain_logits(root, "far", base, dtype, True)
    for marked in [0, 1, 63, 64, 127, 128, 149, 150]:
        p = list(base)
        p[marked] = STANDOUT_TOKEN
        ref = plain_logits(root, "far", p, dtype, True)
        s = eng.alloc_slot()
        if mode == "whole":
            got = eng.step([s], [p], [asking], to="host")
        elif mode == "decode":
            eng.step([s], [p[:ask - 3]], [[]], to="host")
            rows = [eng.step([s], [[tok]], [[0]], to="host") for tok in p[ask - 3:]]
            got = np.concatenate([rows[3], rows[4], rows[-1]])
        else:
            at, rows = 0, {}
            for c in [2, 61, 3, 64, 17, 2, 2, 30, 19]:
                out = eng.step([s], [p[at:at + c]], [list(range(c))], to="host")
                for i in range(c):
                    rows[at + i] = out[i:i + 1]
                at += c
            assert at == n
            got = np.concatenate([rows[a] for a in asking])
        eng.free_slot(s)
        compare(got, ref, asking, dtype, "marked token at %d, %s" % (marked, mode))
        spread = np.sqrt((ref ** 2).mean())
        assert np.sqrt(((ref[n - 1] - without[n - 1]) ** 2).mean()) > 0.2 * spread, "the marked token at %d hardly matters" % marked


def test_faults_would_show(root):
    """What the comparisons would see: the plain implementation with one mechanism changed a little differs from itself by far
    more than the float32 bound."""
    _, cfg, t = model(root, "P", "float32")
    (p,) = prompts([150], cfg["vocab"], 5)
    ref = plain_logits(root, "P", p, "float32")
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

    assert changed(layers__0__mixer__softcap=6.2) > bound
    assert changed(layers__0__mixer__rot__dims=10) > bound
    assert changed(layers__0__mixer__rot__base=9000.0) > bound
    assert changed(layers__1__mixer__decay__2=0.993) > bound
    assert changed(layers__1__mlp__expert__limit=0.85) > bound
    assert changed(layers__1__mlp__shared__limit=1.4) > bound
    assert changed(embedding__scale=2.55) > bound
    assert changed(norm__eps=3e-3) > bound
    assert scaled(l0__mix__sink=lambda x: x - 30.0) > bound
    assert scaled(l1__mlp__correction=lambda x: 0.0 * x) > bound
    assert scaled(l1__mlp__shared__sg=lambda x: 0.0 * x) > bound
    assert scaled(l2__mix__g=lambda x: 0.0 * x) > bound
    assert scaled(l3__mix__q__norm=lambda x: 0.0 * x + 1.0) > bound
    late = plain.forward(cfg, t, p[100:])                       # keys and state lost
    assert np.abs(late[-1] - ref[-1]).max() > bound


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "R", "S", "T", "U", "V"])
def test_prompt_then_token_by_token(root, name, dtype):
    eng, cfg, _ = engine(root, name, dtype)
    n, tail = (330, 150) if name == "R" else (110, 50)
    (p,) = prompts([n], cfg["vocab"], 6)
    s = eng.alloc_slot()
    got = [eng.step([s], [p[:n - tail]], [[n - tail - 1]], to="host")]
    for i in range(n - tail, n):
        got.append(eng.step([s], [[p[i]]], [[0]], to="host"))
    eng.free_slot(s)
    agree(np.concatenate(got), root, name, p, list(range(n - tail - 1, n)), dtype, "%s decode" % name)
    assert nothing_held(eng)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "S"])
def test_all_tokens_one_by_one(root, name, dtype):
    """From the very first token: states start at zero, the first row sees itself and the sink."""
    eng, cfg, _ = engine(root, name, dtype)
    (p,) = prompts([90], cfg["vocab"], 7)
    s = eng.alloc_slot()
    got = [eng.step([s], [[tok]], [[0]], to="host") for tok in p]
    eng.free_slot(s)
    agree(np.concatenate(got), root, name, p, list(range(90)), dtype, "%s one by one" % name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,cuts", [("P", [2, 3, 7, 64, 65, 9, 1, 1, 2]), ("R", [64, 2, 128, 100, 6]), ("Q", [1, 2, 30, 37, 3]),
                                       ("S", [5, 64, 3, 70, 2, 2]), ("T", [3, 2, 40, 1, 5, 66, 2]), ("U", [2, 130, 33, 2, 50])])
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
    """A prompt longer than the step function's pass: states and cache go from pass to pass, and a layer that reads another's
    keys finds those of the pass before and of its own."""
    eng, cfg, _ = engine(root, "R", dtype, prefill_chunk=64)
    (p,) = prompts([300], cfg["vocab"], 9)
    s = eng.alloc_slot()
    got = eng.step([s], [p], [list(range(300))], to="host")
    eng.free_slot(s)
    agree(got, root, "R", p, list(range(300)), dtype, "R in passes of 64")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "R"])
def test_batch_of_unequal_requests(root, name, dtype):
    """Requests of different lengths in one batch (one of a single token), then decoded together; the shorter ones end
    earlier.  Every request must come out as it does alone."""
    eng, cfg, _ = engine(root, name, dtype)
    lengths = [1, 70, 131, 40] if name == "P" else [1, 200, 90]
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


@pytest.mark.parametrize("form", ["grouped", "dense", "pairs"])
def test_forms_of_the_experts(root, form, monkeypatch):
    """The three ways a prompt's rows can run through the experts, with choices that are no expert of the table among them."""
    monkeypatch.setenv("FRIDAY_EXPERTS", form)
    eng, cfg, _ = engine(root, "R", "bfloat16")
    (p,) = prompts([150], cfg["vocab"], 18)
    s = eng.alloc_slot()
    got = eng.step([s], [p], [list(range(150))], to="host")
    eng.free_slot(s)
    agree(got, root, "R", p, list(range(150)), "bfloat16", "R, experts %s" % form)


@pytest.mark.parametrize("splits", ["1", "2", "5", "8", "11"])
def test_one_token_steps_in_splits(root, splits, monkeypatch):
    """A sequence's keys shared among CTAs, as a cluster and through memory, some of them with no key at all: caps, sinks and
    gates join once, whoever merges."""
    monkeypatch.setenv("FRIDAY_ATTN_SPLITS", splits)
    eng, cfg, _ = engine(root, "R", "bfloat16")
    ps = prompts([290, 40], cfg["vocab"], 19)
    slots = [eng.alloc_slot() for _ in ps]
    eng.step(slots, [p[:-3] for p in ps], [[], []], to="host")
    got = [eng.step(slots, [[p[len(p) - 3 + k]] for p in ps], [[0], [0]], to="host") for k in range(3)]
    for i, p in enumerate(ps):
        eng.free_slot(slots[i])
        agree(np.stack([g[i] for g in got]), root, "R", p, list(range(len(p) - 3, len(p))), "bfloat16", "R in %s splits, request %d" % (splits, i))
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_used_again(root, dtype):
    """A slot that held a long request is given to a short one: states start anew, stale pages are not read."""
    eng, cfg, _ = engine(root, "P", dtype, max_batch=2, max_ctx=256, max_tokens=512)
    a, b, c = prompts([200, 30, 90], cfg["vocab"], 11)
    for p in (a, b, c, b):
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
def test_long_decoding(root, dtype):
    """Hundreds of single-token steps: the states run on, the keys of the first tokens stay in sight."""
    eng, cfg, _ = engine(root, "R", dtype)
    (p,) = prompts([10 + 300], cfg["vocab"], 12)
    s = eng.alloc_slot()
    eng.step([s], [p[:10]], [[]], to="host")
    got = [eng.step([s], [[tok]], [[0]], to="host") for tok in p[10:]]
    eng.free_slot(s)
    agree(np.concatenate(got), root, "R", p, list(range(10, 310)), dtype, "R long decoding")


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


def test_bf16_generation_runs_and_repeats(root):
    eng, cfg, _ = engine(root, "R", "bfloat16", max_batch=4)
    ps = prompts([5, 23, 64, 9], cfg["vocab"], 14)
    a = eng.generate(ps, max_new_tokens=20, temperature=0.0, ignore_eos=True)
    b = eng.generate(ps, max_new_tokens=20, temperature=0.0, ignore_eos=True)
    assert [g.tokens for g in a] == [g.tokens for g in b]
    assert all(len(g.tokens) == 20 for g in a)
    assert nothing_held(eng)


def test_the_command_line_generates(root):
    """bin/friday serves the design like any other: the folder's config.json names it."""
    d, cfg, t = model(root, "P", "float32")
    (p,) = prompts([20], cfg["vocab"], 16)
    out = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "friday"), d, "--dtype", "float32", "--ctx", "128", "--json", "--ignore-eos",
                          "--max-new-tokens", "6", "--prompt-ids", ",".join(map(str, p))], capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    tokens = json.loads(out.stdout.strip().splitlines()[-1])["tokens"]
    eng, _, _ = engine(root, "P", "float32")
    assert tokens == eng.generate([p], max_new_tokens=6, temperature=0.0, ignore_eos=True)[0].tokens
