"""Zidepel models through the engine's own entry points (inference_forward_tokens, inference_forward_token,
inference_generate, the command line) against the plain float64 restatement (oracle/hybrid_oracle.py)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import _hybrid as T
from test_gpu_latent_model import run

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
o = T.o
N = 330
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module", params=T.FAMILIES)
def family(request, tmp_path_factory):
    folder, config, weights = T.build(tmp_path_factory, request.param)
    t = T.tokens(config, N, 1)
    return dict(name=request.param, folder=folder, config=config, weights=weights, tokens=t, want=o.forward(config, weights, t)[0])


@pytest.fixture(params=DTYPES)
def model(request, family, pkg):
    with pkg.DirModel(family["folder"], N, request.param) as m:
        m.dtype, m.limit = request.param, T.limit(family["name"], request.param)
        yield m


def good(m, got, want):
    e = T.errors(got, want)
    assert e.max() <= m.limit, (e.max(), int(e.argmax()))


def test_whole_prompt(model, family):
    good(model, run(model, family["tokens"], [N]), family["want"])
    assert model.position == N and model.lib.inference_state_model_type(model.state) == 3


def test_token_by_token(model, family):
    """Long decoding from nothing, and the whole prompt after it on the same state."""
    got = run(model, family["tokens"], [])
    good(model, got, family["want"])
    model.reset()
    assert T.errors(got, run(model, family["tokens"], [N])).max() <= 1.5 * model.limit


@pytest.mark.parametrize("portions", [[2] * 60, [1, 2, 3, 5, 8, 13, 21, 34, 55, 89], [64, 64, 64, 64], [7, 100, 31, 65, 2, 2], [129, 128], [15, 16, 17, 1, 63]])
def test_portions(model, family, portions):
    good(model, run(model, family["tokens"], portions), family["want"])


def test_first_tokens(model, family):
    for first in (1, 2, 3):
        model.reset()
        good(model, run(model, family["tokens"][:12], [first]), family["want"][:12])


def test_places_asked_for(model, family):
    t = family["tokens"]
    every = run(model, t[:90], [90])
    model.reset()
    some = [3, 0, 89, 64]
    got = np.array(model.feed(t[:90], some), dtype=np.float64)[:4 * model.vocab].reshape(4, -1)
    assert np.array_equal(got, every[some])
    model.reset()
    model.feed(t[:50])
    model.feed(t[50:51])
    good(model, np.array(model.feed(t[51:53], [1]), dtype=np.float64)[:model.vocab].reshape(1, -1), family["want"][52:53])


def test_a_sequence_after_another_equals_a_fresh_state(model, family, pkg):
    """Neither cache rows nor states of an earlier, longer sequence are seen; nor those of one generated before."""
    t, other = family["tokens"], T.tokens(family["config"], N, 5)
    run(model, other, [200, 2, 100])
    model.reset()
    again = run(model, t[:80], [33, 2, 20])
    model.generate(other[:60], 20, eos=[])
    model.reset()
    single = run(model, t[:20], [])
    with pkg.DirModel(family["folder"], N, model.dtype) as fresh:
        assert np.array_equal(again, run(fresh, t[:80], [33, 2, 20]))
        fresh.reset()
        assert np.array_equal(single, run(fresh, t[:20], []))


def test_the_cache_can_be_filled_and_not_overfilled(model, family):
    t = family["tokens"]
    run(model, t, [N - 2])
    assert model.position == N
    with pytest.raises(RuntimeError):
        model.feed([1])
    model.reset()
    model.feed(t[:N - 1])
    with pytest.raises(RuntimeError):
        model.feed([1, 2])
    assert model.position == N - 1                                    # a refused portion changes nothing
    good(model, run(model, t, [], start=N - 1), family["want"][N - 1:])


def test_positions_end_with_their_table(pkg, tmp_path):
    """More cache than learned positions: the sequence ends with the table."""
    config, ranks = o.model_config(32, 40, 2, [T.A(2, 1, 8, 8, 16), T.R(1, 8, 8, None, 4.0, 2)], max_positions=37)
    w = o.random_model(config, ranks, 2)
    t = T.tokens(config, 37, 1)
    want, _ = o.forward(config, w, t)
    folder = o.write_model(str(tmp_path / "m"), config, w)
    with pkg.DirModel(folder, 500, "float32") as m:
        m.limit = T.LIMIT["float32"]
        good(m, run(m, t, [20]), want)
        with pytest.raises(RuntimeError):
            m.feed([1])
        assert len(m.generate(t[:30], 50, eos=[])) == 8


def test_a_prompt_longer_than_one_pass_of_the_row_path(pkg, tmp_path):
    config, ranks = o.model_config(48, 64, 2, [T.R(2, 12, 8, None, 300.0, 3), T.A(2, 1, 16, 8, 40, temp=(0.25, 500))], loop=(0, 2, 2), max_positions=2300)
    w = o.random_model(config, ranks, 31)
    w["l0.mix.a2.b"] = o.bf16(w["l0.mix.a2.b"] + 3.0)                         # a state that reaches across the cut
    t = T.tokens(config, 2300, 6)
    want, _ = o.forward(config, w, t)
    folder = o.write_model(str(tmp_path / "m"), config, w)
    places = [0, 1, 63, 64, 1000, 2046, 2047, 2048, 2049, 2111, 2112, 2289]
    for dtype in DTYPES:
        with pkg.DirModel(folder, 2300, dtype) as m:
            got = np.array(m.feed(t[:2290], places), dtype=np.float64).reshape(len(places), -1)
            tail = run(m, t, [], start=2290)
            assert T.errors(np.concatenate([got, tail]), want[places + list(range(2290, 2300))]).max() <= T.LIMIT[dtype]


# ------------------------------------------------------------------ generation

def greedy(family, prompt, n):
    t, margins = list(prompt), []
    for _ in range(n):
        lg = o.forward(family["config"], family["weights"], t)[0][-1]
        top = np.sort(lg)[-2:]
        margins.append((top[1] - top[0]) / lg.std())
        t.append(int(lg.argmax()))
    return t[len(prompt):], margins


@pytest.mark.parametrize("length", [1, 2, 3, 70])
def test_greedy_generation(pkg, family, length):
    prompt = family["tokens"][:length]
    want, margins = greedy(family, prompt, 20)
    safe = next((i for i, m in enumerate(margins) if m < 1e-4), 20)   # beyond a near-tie the continuations may part
    with pkg.DirModel(family["folder"], 128, "float32") as m:
        got = m.generate(prompt, 20, eos=[])
        assert len(got) == 20 and got[:safe] == want[:safe] and safe >= 8
        assert m.generate(prompt, 20, eos=[]) == got                  # nothing of the first request is left
        for k in range(20):                                           # an end id anywhere in a group of ids read back
            stop = got[k]
            cut = m.generate(prompt, 20, eos=[stop])
            assert cut == got[:got.index(stop) + 1]
            assert m.position == length + len(cut) - 1
            # a request goes on where generation stopped, although forwards past the end id have run
            lg = np.array(m.feed(cut[-1:], [0]), dtype=np.float64)
            assert int(lg.argmax()) == (got + [int(lg.argmax())])[len(cut)]
            two = np.array(m.feed([5, 6], [1]), dtype=np.float64).reshape(1, -1)
            if k in (0, 7, 13):
                ref = o.forward(family["config"], family["weights"], list(prompt) + cut + [5, 6])[0][-1:]
                assert T.errors(two, ref).max() <= T.limit(family["name"], "float32")


def test_bfloat16_generation_follows_its_own_logits(pkg, family):
    prompt = family["tokens"][:50]
    with pkg.DirModel(family["folder"], 128, "bfloat16") as m:
        got = m.generate(prompt, 20, eos=[])
        m.reset()
        m.feed(prompt[:-1])
        for prev, tok in zip([prompt[-1]] + got, got):
            assert int(np.array(m.feed([prev], [0]), dtype=np.float32).argmax()) == tok


def test_launch_chaining_changes_nothing(pkg, family, monkeypatch):
    t = family["tokens"][:60]
    with pkg.DirModel(family["folder"], N, "bfloat16") as m:
        a = run(m, t, [20])
    monkeypatch.setenv("LLMB200_NO_PDL", "1")
    with pkg.DirModel(family["folder"], N, "bfloat16") as m:
        assert np.array_equal(a, run(m, t, [20]))


def test_measurement_hooks_leave_the_sequence_alone(pkg, family):
    with pkg.DirModel(family["folder"], N, "float32") as m:
        L, t = m.lib, family["tokens"]
        m.feed(t[:100])
        runs = o.order(family["config"])
        dense = sum(1 for i in runs if family["config"]["layers"][i]["mlp"])
        assert L.llmb200_state_graph_kernels(m.state, 1) == 3 * len(runs) + 2 * dense + 1
        n = C.c_int(0)
        for kind in range(6):
            assert L.llmb200_state_time_kind(m.state, kind, 2, C.byref(n)) >= 0
        lg = np.array(m.feed(t[100:103], [0, 1, 2]), dtype=np.float64).reshape(3, -1)         # states are where they were
        assert T.errors(lg, family["want"][100:103]).max() <= T.limit(family["name"], "float32")
        ms, launches = (C.c_float * 6)(), (C.c_int * 6)()
        assert L.llmb200_state_profile_token(m.state, ms, launches) == 0
        assert list(launches) == [len(runs)] * 3 + [dense] * 2 + [1]
        assert L.llmb200_state_run_device_steps(m.state, 5) > 0 and m.position == 109


# ------------------------------------------------------------------ parts in isolation, by weights

@pytest.mark.parametrize("what", ["no mixer", "no feed-forward", "streams swapped", "one stream read", "no positions"])
def test_parts_switched_off_by_their_weights(pkg, tmp_path, what):
    config, ranks = o.model_config(72, 88, 3, [T.A(3, 1, 12, 10, 40), T.R(2, 10, 12, None, 8.0, 4), T.A(2, 2, 8, 8, None)], loop=(1, 3, 2))
    w = o.random_model(config, ranks, 21)
    for name in list(w):
        if (what == "no mixer" and name.endswith("mix.o")) or (what == "no feed-forward" and name.endswith("mlp.down")) or (what == "no positions" and name == "pos"):
            w[name] = w[name] * 0
        if what == "streams swapped" and name.endswith("hc1.mix"):
            w[name] = np.roll(np.eye(3), 1, axis=1)
        if what == "one stream read" and name.endswith(".in"):
            w[name] = np.array([0.0, 1.0, 0.0])
    t = T.tokens(config, 50, 3)
    want, _ = o.forward(config, w, t)
    folder = o.write_model(str(tmp_path / "m"), config, w)
    for dtype in DTYPES:
        with pkg.DirModel(folder, 50, dtype) as m:
            m.limit = T.LIMIT[dtype]
            good(m, run(m, t, [23, 2]), want)


@pytest.mark.parametrize("loop,same", [(None, True), ((1, 1, 3), True), ((0, 3, 1), True), ((2, 3, 2), False), ((0, 1, 3), False)])
def test_loops_of_every_kind(pkg, tmp_path, loop, same):
    config, ranks = o.model_config(40, 56, 2, [T.R(2, 8, 12, 24, 4.0, 3), T.A(2, 1, 8, 16, None), T.A(4, 2, 8, 8, 32)], loop=loop)
    w = o.random_model(config, ranks, 5)
    t = T.tokens(config, 40, 2)
    want, _ = o.forward(config, w, t)
    assert np.array_equal(want, o.forward(dict(config, loop=None), w, t)[0]) == same
    with pkg.DirModel(o.write_model(str(tmp_path / "m"), config, w), 40, "float32") as m:
        m.limit = T.LIMIT["float32"]
        good(m, run(m, t, [25, 2]), want)


def test_a_far_key_decides(pkg, tmp_path):
    """One attention layer whose scores rest on the tokens alone: queries of token 1 score the key of token 0 far above all
    others, and token 0 occurs once, hundreds of tokens back. In a prompt, in a later portion, and decoded alone."""
    config, ranks = o.model_config(64, 48, 2, [T.A(2, 1, 32, 32, None, scale=1.0, cap=40.0, temp=None)], max_positions=700)
    w = o.random_model(config, ranks, 17)
    w["pos"] = w["pos"] * 0
    eps = config["norm"]["eps"]
    x = o.layer_norm(w["embed"], w["embed.norm"], w["embed.norm.b"], eps)
    h = o.layer_norm(w["l0.hc1.in"].sum() * x, w["l0.norm1"], w["l0.norm1.b"], eps)      # the mixer's input, token by token
    d = h[1] - h[0]
    swap = np.eye(64) - 2.0 * np.outer(d, d) / (d @ d)                # turns the input of token 1 into (nearly) that of token 0
    w["l0.mix.q"] = o.bf16(np.concatenate([w["l0.mix.k"] @ swap] * 2))
    w["l0.mix.q.norm"] = w["l0.mix.k.norm"] = np.ones(32)
    t = [int(v) for v in np.random.default_rng(3).integers(2, 48, 700)]
    marked = [400, 401, 620, 699]
    for i in marked:
        t[i] = 1
    t[9] = 0
    want, _ = o.forward(config, w, t)
    changed = t.copy()
    changed[9] = 5
    assert T.errors(o.forward(config, w, changed)[0], want)[marked].min() > 0.2         # the logits rest on the far key
    folder = o.write_model(str(tmp_path / "m"), config, w)
    for dtype in DTYPES:
        with pkg.DirModel(folder, 700, dtype) as m:
            m.limit = T.LIMIT[dtype]
            good(m, run(m, t, [300, 110, 200]), want)


def test_large_activations_keep_their_range(pkg, tmp_path):
    config, ranks = o.model_config(64, 80, 2, [T.A(2, 2, 16, 24, 64), T.R(2, 16, 16, 64, 8.0, 4)])
    w = o.random_model(config, ranks, 22)
    for name in ("l0.mlp.up", "l1.mlp.up"):
        w[name] = o.bf16(w[name] * 2e3)                               # squared: far outside binary16's range
    t = T.tokens(config, 40, 4)
    want, _ = o.forward(config, w, t)
    with pkg.DirModel(o.write_model(str(tmp_path / "m"), config, w), 40, "bfloat16") as m:
        m.limit = T.LIMIT["bfloat16"]
        good(m, run(m, t, [25, 5]), want)


# ------------------------------------------------------------------ refusals and the command line

def edited(tmp_path, change=None, drop=None, reshape=None):
    config, ranks = T.CONFIGS["mixed"]
    config = json.loads(json.dumps(config))
    w = o.random_model(config, ranks, 9)
    if change:
        change(config)
    if drop:
        del w[drop]
    if reshape:
        w[reshape] = w[reshape][:-1]
    return o.write_model(str(tmp_path / "m"), config, w)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][1].__setitem__("type", "other"), lambda c: c["layers"][1].__setitem__("mlp", {"kind": "sparse", "ff": 8}),
    lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 4), lambda c: c["layers"][1]["mixer"].__setitem__("softcap", -1.0),
    lambda c: c["layers"][1]["mixer"].__setitem__("q_temp", {"coef": 1.0}), lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mixer"].pop("tau"), lambda c: c["layers"][0]["mixer"].__setitem__("dim", 0), lambda c: c.pop("streams"),
    lambda c: c.__setitem__("streams", 9), lambda c: c.__setitem__("loop", {"start": 1, "stop": 5, "times": 2}),
    lambda c: c.__setitem__("loop", {"start": 2, "stop": 1, "times": 2}), lambda c: c.__setitem__("loop", {"start": 0, "stop": 1, "times": 0}),
    lambda c: c["norm"].pop("eps"), lambda c: c.__setitem__("max_positions", 511)])
def test_unusable_configurations_are_refused(lib, tmp_path, change):
    assert not lib.inference_state_create_from_dir(edited(tmp_path, change).encode(), 32, 2)


def test_missing_or_misshapen_tensors_are_refused(lib, tmp_path):
    for kw in (dict(drop="l1.hc2.mix"), dict(drop="final.norm.b"), dict(drop="l0.mix.a1"), dict(reshape="l0.mix.a2.b"), dict(reshape="l1.hc1.in"),
               dict(reshape="pos"), dict(reshape="l1.mlp.down")):
        assert not lib.inference_state_create_from_dir(edited(tmp_path, **kw).encode(), 32, 2), kw


def test_command_line(pkg, tmp_path):
    config, ranks = T.CONFIGS["odd"]
    w = o.random_model(config, ranks, 13)
    folder = o.write_model(str(tmp_path / "m"), config, w)
    t = [T.tokens(config, 60, s) for s in (1, 2)]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[0][:40], "want": [39, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[0][40:41], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": t[0][41:43], "want": [0, 1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": t[1][:1], "want": [0]}], "end": []},
             {"step": 4, "entries": [{"id": "b", "tokens": t[1][1:30], "want": [28]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    for dtype in DTYPES:
        r = subprocess.run([os.path.join(T.ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "60"],
                           input="\n".join(map(json.dumps, steps)), stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert r.stdout.split("\n") == [f"done {i}" for i in range(5)] + [""]
        full = [o.forward(config, w, x)[0] for x in t]
        for name, want in ((0, full[0][[39, 2]]), (2, full[0][[41, 42]]), (3, full[1][:1]), (4, full[1][[29]])):
            got = np.fromfile(out / f"{name}.f32", "<f4").reshape(-1, config["vocab"])
            assert T.errors(got, want).max() <= T.LIMIT[dtype]
            os.unlink(out / f"{name}.f32")
        assert not os.listdir(out)
    r = subprocess.run([sys.executable, os.path.join(T.ROOT, "bin", "generate"), "--model", folder, "--dtype", "float32", "--prompt", "3, 1,4",
                        "--max-new", "6", "--max-tokens", "32"], stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    with pkg.DirModel(folder, 32, "float32") as m:
        assert list(map(int, r.stdout.split(","))) == m.generate([3, 1, 4], 6)
