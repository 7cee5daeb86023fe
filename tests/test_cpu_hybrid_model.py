"""Zidepel without a GPU: the restatement against independent forms of the same equations, and that its test inputs
show a wrong connection, decay, norm, factor or order."""
import ctypes as C
import json
import os

import numpy as np
import pytest

import _hybrid as T

o = T.o


def test_layer_norm_has_mean_and_spread_of_its_weights():
    x = np.random.default_rng(1).standard_normal((3, 50)) * 7 + 3
    y = o.layer_norm(x, np.full(50, 2.0), np.full(50, 5.0), 0.0)
    assert np.allclose(y.mean(axis=1), 5.0) and np.allclose(y.std(axis=1), 2.0)
    assert np.allclose(o.layer_norm(x, np.ones(50), np.zeros(50), 1e9), (x - x.mean(1, keepdims=True)) / np.sqrt(x.var(axis=1)[:, None] + 1e9))


def test_query_factor_steps_where_a_block_is_complete():
    f = o.query_temperature(13, {"coef": 0.5, "every": 4})
    assert np.allclose(f[:3], 1.0) and np.allclose(f[3:7], 1 + 0.5 * np.log(2)) and np.allclose(f[7:11], 1 + 0.5 * np.log(3)) and f[11] > f[10]
    assert np.allclose(o.query_temperature(3, {"coef": 2.0, "every": 1}), 1 + 2 * np.log([2, 3, 4]))


def test_attention_one_query_at_a_time():
    rng = np.random.default_rng(2)
    q, k, v = rng.standard_normal((9, 6, 10)) * 3, rng.standard_normal((9, 2, 10)), rng.standard_normal((9, 2, 4))
    got = o.attend(q, k, v, 0.7, 5.0)
    for i in range(9):
        for h in range(6):
            s = np.array([5.0 * np.tanh(0.7 * (q[i, h] @ k[j, h // 3]) / 5.0) for j in range(i + 1)])
            p = np.exp(s) / np.exp(s).sum()
            assert np.allclose(got[i, h], p @ v[: i + 1, h // 3])
    assert not np.allclose(got, o.attend(q, k, v, 0.7, None))


def test_decay_at_both_ends():
    assert np.allclose(o.decay(np.array([0.0, 40.0, -900.0]), 1.0), [0.5, 1.0, 0.0])
    assert np.allclose(o.decay(np.array([1.3, -2.0]), 4.0), (1 / (1 + np.exp([-1.3, 2.0]))) ** 0.25)


def test_recurrence_as_a_weighted_sum_over_earlier_tokens():
    rng = np.random.default_rng(3)
    q, k, v, a = rng.standard_normal((20, 6)), rng.standard_normal((20, 6)), rng.standard_normal((20, 5)), rng.uniform(0.2, 1.0, (20, 6))
    out, S = o.recurrence(q, k, v, a)
    for t in range(20):
        want = sum(((q[t] * k[s] * np.prod(a[s + 1:t + 1], axis=0)).sum()) * v[s] for s in range(t + 1))
        assert np.allclose(out[t], want)
    tail, S2 = o.recurrence(q[12:], k[12:], v[12:], a[12:], o.recurrence(q[:12], k[:12], v[:12], a[:12])[1])
    assert np.allclose(tail, out[12:]) and np.allclose(S, S2)


def test_one_stream_with_unit_connections_is_a_residual_sum():
    rng = np.random.default_rng(4)
    x, W = rng.standard_normal((1, 5, 8)), rng.standard_normal((8, 8))
    one = {"in": np.ones(1), "out": np.ones(1), "mix": np.ones((1, 1))}
    assert np.allclose(o.connect(x, one, lambda u: 2 * u, lambda h: h @ W), x + 2 * x @ W)


def test_connections_read_and_write_stream_by_stream():
    rng = np.random.default_rng(5)
    x, c = rng.standard_normal((3, 2, 4)), {"in": rng.standard_normal(3), "out": rng.standard_normal(3), "mix": rng.standard_normal((3, 3))}
    got = o.connect(x, c, lambda u: u, lambda h: h * h)
    u = sum(c["in"][s] * x[s] for s in range(3))
    for t in range(3):
        assert np.allclose(got[t], sum(c["mix"][s, t] * x[s] for s in range(3)) + c["out"][t] * u * u)


def test_order_of_runs():
    config = {"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 3}}
    assert o.order(config) == [0, 1, 2, 1, 2, 1, 2, 3, 4] and o.order(dict(config, loop=None)) == [0, 1, 2, 3, 4]


def test_appending_tokens_changes_nothing_before_them():
    config, ranks = T.CONFIGS["mixed"]
    w, t = o.random_model(config, ranks, 3), T.tokens(config, 60)
    assert np.allclose(o.forward(config, w, t)[0][:31], o.forward(config, w, t[:31])[0])


MISTAKES = ["loop", "mix transposed", "take", "spread", "norm bias", "embedding norm", "positions", "tau", "decay bias", "query factor", "factor step",
            "cap", "gate", "state", "eps", "key norm"]


@pytest.mark.parametrize("what", MISTAKES)
def test_a_planted_mistake_shows_far_above_the_limits(what, monkeypatch):
    """The inputs of the GPU tests would reveal each of these in the logits."""
    config, ranks = T.CONFIGS["mixed"]
    config = json.loads(json.dumps(config))
    w = o.random_model(config, ranks, 7)
    t = T.tokens(config, 90)
    right, _ = o.forward(config, w, t)
    mixers = [layer["mixer"] for layer in config["layers"]]
    if what == "loop":
        config["loop"]["times"] = 3
    for name in list(w):
        if what == "mix transposed" and name.endswith(".mix"):
            w[name] = w[name].T
        if (what == "take" and name.endswith(".in")) or (what == "spread" and name.endswith(".out")) or (what == "key norm" and name.endswith("k.norm")):
            w[name] = np.roll(w[name], 1)
        if (what == "norm bias" and name.endswith("norm1.b")) or (what == "decay bias" and name.endswith("a2.b")):
            w[name] = w[name] * 0.9
    if what == "embedding norm":
        w["embed.norm.b"] = w["embed.norm.b"] * 0
    if what == "positions":
        w["pos"] = np.roll(w["pos"], 1, axis=0)
    if what == "tau":
        mixers[2]["tau"] = 2.1
    if what == "query factor":
        mixers[1]["q_temp"] = None
    if what == "factor step":
        mixers[1]["q_temp"]["every"] = 8
    if what == "cap":
        mixers[3]["softcap"] = None
    if what == "gate":
        monkeypatch.setattr(o, "silu", lambda z: 1.0 / (1.0 + np.exp(-z)))
    if what == "eps":
        config["norm"]["eps"] = 1e-2
    if what == "state":                                               # the state is lost after forty tokens
        rec = o.recurrence
        monkeypatch.setattr(o, "recurrence", lambda q, k, v, a: (np.concatenate([rec(q[:40], k[:40], v[:40], a[:40])[0], rec(q[40:], k[40:], v[40:], a[40:])[0]]), None))
    wrong, _ = o.forward(config, w, t)
    e = T.errors(wrong, right)
    assert np.median(e[45:]) > 20 * T.LIMIT["float32"], e[45:]
    if what not in ("eps", "tau", "cap", "factor step"):
        assert e.max() > T.LIMIT["bfloat16"], e.max()


def test_tensor_dimensions_are_read_from_the_file(lib, tmp_path):
    config, ranks = T.CONFIGS["odd"]
    folder = o.write_model(str(tmp_path / "m"), config, o.random_model(config, ranks, 1))
    lib.llmb200_tensor_file_open.restype, lib.llmb200_tensor_file_open.argtypes = C.c_void_p, [C.c_char_p]
    lib.llmb200_tensor_file_close.restype, lib.llmb200_tensor_file_close.argtypes = None, [C.c_void_p]
    lib.llmb200_tensor_dim.restype, lib.llmb200_tensor_dim.argtypes = C.c_longlong, [C.c_void_p, C.c_char_p, C.c_int]
    f = lib.llmb200_tensor_file_open(os.path.join(folder, "model.safetensors").encode())
    dims = [lib.llmb200_tensor_dim(f, n, a) for n, a in ((b"l1.mix.a1", 0), (b"l1.mix.a1", 1), (b"l2.mix.a1", 0), (b"embed", 0), (b"l0.norm1", 0),
                                                        (b"l0.norm1", 1), (b"embed", -1), (b"nothing", 0))]
    lib.llmb200_tensor_file_close(f)
    assert dims == [9, 101, 17, 203, 101, -1, -1, -1]
