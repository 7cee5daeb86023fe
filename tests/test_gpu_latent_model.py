"""Morilorn models through the engine's own entry points (inference_forward_tokens, inference_forward_token,
inference_generate, the command line) against the plain float64 restatement (oracle/latent_oracle.py)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import _latent as T

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
o = T.o
N = 330          # longer than every window of the test models but one, and than the tiles of the kernels
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module", params=T.FAMILIES)
def family(request, tmp_path_factory):
    folder, config, weights = T.build(tmp_path_factory, request.param)
    t = T.tokens(config, N, 1)
    want, handed_on = o.forward(config, weights, t)
    return dict(folder=folder, config=config, weights=weights, tokens=t, want=want)


@pytest.fixture(params=DTYPES)
def model(request, family, pkg):
    with pkg.DirModel(family["folder"], N, request.param) as m:
        m.limit = T.LIMIT[request.param]
        yield m


def run(m, tokens, portions, start=0, decode=True):
    """Logits of every token, the sequence fed in portions (what is left over one by one)."""
    out, at = [], start
    for k in list(portions) + [1] * (len(tokens) - start - sum(portions)):
        out.append(np.array(m.feed(tokens[at:at + k], range(k)), dtype=np.float64).reshape(k, m.vocab))
        at += k
    return np.concatenate(out)


def good(m, got, want):
    e = T.errors(got, want)
    assert e.max() <= m.limit, (e.max(), int(e.argmax()))


def test_whole_prompt(model, family):
    good(model, run(model, family["tokens"], [N]), family["want"])
    assert model.position == N


def test_token_by_token(model, family):
    got = run(model, family["tokens"], [])
    good(model, got, family["want"])
    model.reset()
    whole = run(model, family["tokens"], [N])
    assert T.errors(got, whole).max() <= 1.5 * model.limit


@pytest.mark.parametrize("portions", [[2] * 60, [1, 2, 3, 5, 8, 13, 21, 34, 55, 89], [64, 64, 64, 64], [7, 100, 31, 65, 2, 2], [129, 128]])
def test_portions(model, family, portions):
    good(model, run(model, family["tokens"], portions), family["want"])


def test_first_tokens(model, family):
    for first in (1, 2, 3):
        model.reset()
        good(model, run(model, family["tokens"][:12], [first]), family["want"][:12])


def test_places_asked_for(model, family):
    """Any subset of places, in any order, equals the same rows of all places; none is fine too."""
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
    """Cache rows that an earlier, longer sequence left behind must not be seen."""
    t, other = family["tokens"], T.tokens(family["config"], N, 5)
    run(model, other, [200, 2, 100])
    model.reset()
    again = run(model, t[:80], [33, 2, 20])
    with pkg.DirModel(family["folder"], N, [k for k, v in model.DTYPES.items() if T.LIMIT[k] == model.limit][0]) as fresh:
        assert np.array_equal(again, run(fresh, t[:80], [33, 2, 20]))


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


def test_bad_input_is_refused(model):
    L = model.lib
    buf, one = (C.c_float * model.vocab)(), (C.c_uint32 * 2)(0, model.vocab)
    fp = C.cast(buf, C.POINTER(C.c_float))
    assert L.inference_forward_tokens(model.state, one, 2, None, 0, None) < 0          # an id outside the vocabulary
    assert L.inference_forward_tokens(model.state, one, 0, None, 0, None) < 0
    assert L.inference_forward_tokens(model.state, one, 1, (C.c_int * 1)(1), 1, fp) < 0
    assert L.inference_forward_tokens(model.state, one, 1, (C.c_int * 1)(0), 1, None) < 0
    assert not L.inference_forward_token(model.state, model.vocab)
    assert model.position == 0 and L.llmb200_state_error(model.state) == 0


def test_the_single_token_entry_point(model, family):
    t, rows = family["tokens"][:40], []
    for k in t:
        p = model.lib.inference_forward_token(model.state, k)
        rows.append(np.ctypeslib.as_array(p, shape=(model.vocab,)).astype(np.float64))
    good(model, np.stack(rows), family["want"][:40])
    assert model.lib.inference_state_model_type(model.state) == 2


def test_long_decoding(pkg, family):
    """A few prompt tokens, then one by one until every window has been passed several times over."""
    with pkg.DirModel(family["folder"], N, "float32") as m:
        m.limit = T.LIMIT["float32"]
        good(m, run(m, family["tokens"], [3]), family["want"])


def test_a_prompt_longer_than_one_pass_of_the_row_path(pkg, tmp_path):
    """2300 tokens: two passes inside one call, windows reaching across the cut; then decoding from there."""
    config = o.model_config(48, 64, [T.L(2, 12, 4, 8, 16, 90, 40), T.L(1, 8, 8, 16, 24, 2200, None)], groups=2)
    w = o.random_model(config, 31)
    t = T.tokens(config, 2300, 6)
    want, _ = o.forward(config, w, t)
    folder = o.write_model(str(tmp_path / "m"), config, w)
    places = [0, 1, 89, 90, 1000, 2046, 2047, 2048, 2049, 2136, 2137, 2138, 2199, 2200, 2280, 2289]
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
    want, margins = greedy(family, prompt, 24)
    safe = next((i for i, m in enumerate(margins) if m < 1e-4), 24)   # beyond a near-tie the continuations may part
    with pkg.DirModel(family["folder"], 128, "float32") as m:
        got = m.generate(prompt, 24, eos=[])
        assert len(got) == 24 and got[:safe] == want[:safe] and safe >= 8
        assert m.generate(prompt, 24, eos=[]) == got                  # nothing of the first request is left
        stop = got[5]
        cut = m.generate(prompt, 24, eos=[stop])
        assert cut == got[:got.index(stop) + 1]
        assert m.position == length + len(cut) - 1
        # a request goes on where generation stopped
        lg = np.array(m.feed(cut[-1:], [0]), dtype=np.float64)
        assert int(lg.argmax()) == (got + [None])[len(cut)]


def test_generation_stops_at_the_end_of_the_cache(pkg, family):
    with pkg.DirModel(family["folder"], 40, "bfloat16") as m:
        assert len(m.generate(family["tokens"][:30], 64, eos=[])) == 11
        with pytest.raises(RuntimeError):
            m.generate(family["tokens"][:41], 4)


def test_bfloat16_generation_follows_its_own_logits(pkg, family):
    prompt = family["tokens"][:50]
    with pkg.DirModel(family["folder"], 128, "bfloat16") as m:
        got = m.generate(prompt, 20, eos=[])
        m.reset()
        m.feed(prompt[:-1])
        for prev, tok in zip([prompt[-1]] + got, got):
            lg = np.array(m.feed([prev], [0]), dtype=np.float32)
            assert int(lg.argmax()) == tok


def test_launch_chaining_changes_nothing(pkg, family, monkeypatch):
    t = family["tokens"][:60]
    with pkg.DirModel(family["folder"], N, "bfloat16") as m:
        a = run(m, t, [20])
    monkeypatch.setenv("LLMB200_NO_PDL", "1")
    with pkg.DirModel(family["folder"], N, "bfloat16") as m:
        assert np.array_equal(a, run(m, t, [20]))


def test_measurement_hooks(pkg, family):
    with pkg.DirModel(family["folder"], N, "bfloat16") as m:
        L, t = m.lib, family["tokens"]
        m.feed(t[:100])
        ms, launches = (C.c_float * 6)(), (C.c_int * 6)()
        assert L.llmb200_state_profile_token(m.state, ms, launches) == 0
        layers, dense = family["config"]["layers"], sum(1 for x in family["config"]["layers"] if x["mlp"])
        assert list(launches) == [len(layers)] * 3 + [dense] * 2 + [1]
        assert L.llmb200_state_graph_kernels(m.state, 1) == 5 * len(layers) + 2 * dense + 1
        n = C.c_int(0)
        for kind in range(6):
            assert L.llmb200_state_time_kind(m.state, kind, 2, C.byref(n)) > 0 and n.value > 0
        m.reset()
        m.feed(t[:100])                                               # the timing loops leave no trace in a new sequence
        lg = np.array(m.feed(t[100:101], [0]), dtype=np.float64).reshape(1, -1)
        assert T.errors(lg, family["want"][100:101]).max() <= T.LIMIT["bfloat16"]
        assert L.llmb200_state_run_device_steps(m.state, 5) > 0 and m.position == 106


# ------------------------------------------------------------------ one layer's parts in isolation, by weights

@pytest.mark.parametrize("what", ["no mixer", "no feed-forward result", "depth: first only", "depth: one earlier layer"])
def test_parts_switched_off_by_their_weights(pkg, tmp_path, what):
    config = o.model_config(72, 88, [T.L(2, 12, 8, 10, 20, 9, 40), T.L(3, 10, 4, 12, 24, 17, None), T.L(2, 8, 8, 8, 16, 5, 56)], groups=2)
    w = o.random_model(config, 21)
    for i in range(3):
        if what == "no mixer":
            w[f"l{i}.mix.o"] *= 0
        if what == "no feed-forward result" and f"l{i}.mlp.down" in w:
            w[f"l{i}.mlp.down"] *= 0
        if what.startswith("depth"):
            w[f"l{i}.dwa"] *= 0
            w[f"l{i}.dwa"][0 if what.endswith("only") else i] = 1.0
    t = T.tokens(config, 50, 3)
    want, _ = o.forward(config, w, t)
    folder = o.write_model(str(tmp_path / "m"), config, w)
    for dtype in DTYPES:
        with pkg.DirModel(folder, 50, dtype) as m:
            m.limit = T.LIMIT[dtype]
            good(m, run(m, t, [23, 2]), want)


def test_large_activations_keep_their_range(pkg, tmp_path):
    """Values far outside binary16's range pass through the bfloat16 path."""
    config = o.model_config(64, 80, [T.L(2, 16, 8, 16, 24, 30, 64)], emb_scale=2e5)
    w = o.random_model(config, 22)
    w["l0.mlp.up"] = o.bf16(w["l0.mlp.up"] * 3e5)
    t = T.tokens(config, 40, 4)
    want, _ = o.forward(config, w, t)
    with pkg.DirModel(o.write_model(str(tmp_path / "m"), config, w), 40, "bfloat16") as m:
        m.limit = T.LIMIT["bfloat16"]
        good(m, run(m, t, [25, 5]), want)


# ------------------------------------------------------------------ refusals and the command line

def edited(tmp_path, change, drop=None, reshape=None):
    config = json.loads(json.dumps(T.CONFIGS["narrow"]))
    w = o.random_model(config, 9)
    change(config)
    if drop:
        del w[drop]
    if reshape:
        w[reshape] = w[reshape][:-1]
    return o.write_model(str(tmp_path / "m"), config, w)


@pytest.mark.parametrize("key,value", [("type", "other"), ("mlp", {"kind": "sparse", "ff": 8}), ("mlp", {"kind": "dense", "ff": 0})])
def test_unknown_layer_parts_are_refused(lib, tmp_path, key, value):
    folder = edited(tmp_path, lambda c: c["layers"][1].__setitem__(key, value))
    assert not lib.inference_state_create_from_dir(folder.encode(), 32, 2)


@pytest.mark.parametrize("key", ["heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"])
def test_a_missing_constant_is_refused(lib, tmp_path, key):
    folder = edited(tmp_path, lambda c: c["layers"][0]["mixer"].pop(key))
    assert not lib.inference_state_create_from_dir(folder.encode(), 32, 2)


def test_missing_or_misshapen_tensors_are_refused(lib, tmp_path):
    for kw in (dict(drop="l1.mix.uk"), dict(drop="final.norm"), dict(reshape="l0.rg1"), dict(reshape="l1.dwa"), dict(reshape="embed")):
        assert not lib.inference_state_create_from_dir(edited(tmp_path, lambda c: None, **kw).encode(), 32, 2), kw


def test_end_ids_come_from_the_configuration(pkg, tmp_path):
    config, prompt = T.CONFIGS["narrow"], [5, 9, 11]
    w = o.random_model(config, 9)
    with pkg.DirModel(o.write_model(str(tmp_path / "a"), config, w), 64, "float32") as m:
        free = m.generate(prompt, 20)
    assert len(free) == 20
    stop = free[6]
    with pkg.DirModel(o.write_model(str(tmp_path / "b"), dict(config, eos_token_id=[stop, 3]), w), 64, "float32") as m:
        got = m.generate(prompt, 20)
    ends = [i for i, t in enumerate(free) if t in (stop, 3)]
    assert got == free[:ends[0] + 1]


def test_command_line(pkg, tmp_path):
    config = T.CONFIGS["odd"]
    w = o.random_model(config, 13)
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
    bad = dict(steps[0], entries=[dict(steps[0]["entries"][0], id=i) for i in "ab"])
    r = subprocess.run([os.path.join(T.ROOT, "bin", "trace_run"), "--model", folder, "--out", str(out), "--max-tokens", "60"],
                       input=json.dumps(bad), stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=300)
    assert r.returncode != 0


def test_other_model_types_take_portions_too(pkg, lib, synth):
    """inference_forward_tokens on a Qwen3 state: token by token behind the same call."""
    sp = pkg.spec("tiny-qwen3", n_layers=2)
    model = synth.llmb200_synth_qwen3(C.byref(sp), 4)
    st = lib.inference_state_create(model, 64, 0)
    lib.metal_flush()
    synth.llmb200_synth_free_qwen3(model)
    ids = np.random.default_rng(0).integers(0, sp.vocab_size, 20)
    one = [np.ctypeslib.as_array(lib.inference_forward_token(st, int(t)), shape=(sp.vocab_size,)).copy() for t in ids]
    lib.inference_state_reset(st)
    got = np.zeros((2, sp.vocab_size), dtype=np.float32)
    rc = lib.inference_forward_tokens(st, (C.c_uint32 * 20)(*map(int, ids)), 20, (C.c_int * 2)(4, 19), 2, got.ctypes.data_as(pkg.c_float_p))
    assert rc == 0 and np.array_equal(got[0], one[4]) and np.array_equal(got[1], one[19]) and lib.llmb200_state_position(st) == 20
    lib.inference_state_free(st)
