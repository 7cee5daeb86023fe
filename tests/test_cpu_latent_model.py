"""Morilorn without a GPU: the restatement against independent forms of the same equations, that its test inputs
show a wrong window, rotation or norm, and the host code that reads model folders."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import _latent as T

o = T.o
ROOT = T.ROOT


def test_rotation_is_a_complex_product():
    rng = np.random.default_rng(1)
    v, pos = rng.standard_normal((5, 3, 10)), np.array([0, 1, 7, 900, 4000])
    got = o.rotate(v, pos, 50.0, 8)
    z = v[..., 0:8:2] + 1j * v[..., 1:8:2]
    z = z * np.exp(1j * pos[:, None, None] * 50.0 ** (-np.arange(4) / 4.0))
    assert np.allclose(got[..., 0:8:2], z.real) and np.allclose(got[..., 1:8:2], z.imag)
    assert np.array_equal(got[..., 8:], v[..., 8:]) and np.array_equal(got[0], v[0])


def test_latent_attention_one_query_at_a_time():
    """The scores of the definition against the form with the query moved into the latent space."""
    rng = np.random.default_rng(2)
    mix = T.L(3, 10, 6, 5, 14, 4, None)["mixer"]
    n = 11
    c, kr_raw, q = rng.standard_normal((n, 14)), rng.standard_normal((n, 6)), rng.standard_normal((n, 3, 16))
    uk, uv = rng.standard_normal((30, 14)), rng.standard_normal((15, 14))
    kr = o.rotate(kr_raw, np.arange(n), mix["rot"]["base"], 6)
    got = o.attend(q, c, kr, mix, uk, uv)
    for i in range(n):
        for h in range(3):
            qn = uk[h * 10:(h + 1) * 10].T @ q[i, h, :10]
            qr = o.rotate(q[i:i + 1, h, 10:], np.array([i]), mix["rot"]["base"], 6)[0]
            js = list(range(max(0, i - 3), i + 1))
            s = np.array([(qn @ c[j] + qr @ kr[j]) * mix["scale"] for j in js])
            p = np.exp(s - s.max())
            p /= p.sum()
            assert np.allclose(got[i, h], uv[h * 5:(h + 1) * 5] @ (p @ c[js]))


def test_window_counts_the_token_itself():
    v = o.visible(6, 3)
    assert v[5].tolist() == [False, False, False, True, True, True] and v[1].tolist() == [True, True, False, False, False, False]
    assert o.visible(6, None)[5].all() and o.visible(6, 1).sum() == 6


def test_groups_are_normalised_apart():
    x = np.array([[3.0, 4.0, 0.5, 0.5]])
    y = o.group_rms(x, np.ones(4), 2, 0.0)
    assert np.allclose(y, [[3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 1.0, 1.0]])
    assert not np.allclose(y, o.group_rms(x, np.ones(4), 1, 0.0))


def test_appending_tokens_changes_nothing_before_them():
    config = T.CONFIGS["odd"]
    w = o.random_model(config, 3)
    t = T.tokens(config, 60)
    a, _ = o.forward(config, w, t)
    b, _ = o.forward(config, w, t[:31])
    assert np.allclose(a[:31], b)


@pytest.mark.parametrize("what", ["window+1", "window-1", "rotation", "groups", "depth", "gate", "alpha", "cap", "eps"])
def test_a_planted_mistake_shows_far_above_the_limits(what):
    """The inputs of the GPU tests would reveal each of these in the logits."""
    config = json.loads(json.dumps(T.CONFIGS["odd"]))
    w = o.random_model(config, 7)
    t = T.tokens(config, 90)
    right, _ = o.forward(config, w, t)
    w = dict(w)
    for i, layer in enumerate(config["layers"]):
        m = layer["mixer"]
        if what.startswith("window"):
            m["mask"]["size"] += int(what[6:])
        if what == "rotation":
            m["rot"]["base"] *= 1.5
        if what == "gate":
            w[f"l{i}.rg1.b"] = w[f"l{i}.rg1.b"] * 0
    if what == "groups":
        config["norm"]["groups"] = 1
    if what == "depth":
        w["l2.dwa"] = np.roll(w["l2.dwa"], 1)
    if what == "alpha":
        config["postln_alpha"] *= 1.3
    if what == "cap":
        config["logit_softcap"] *= 1.2
    if what == "eps":
        config["norm"]["eps"] = 3e-2
    wrong, _ = o.forward(config, w, t)
    e = T.errors(wrong, right)
    assert np.median(e[45:]) > 20 * T.LIMIT["float32"], e[45:]
    if what != "eps":
        assert e.max() > 1.0 * T.LIMIT["bfloat16"], e.max()


# ------------------------------------------------------------------ host code

@pytest.fixture()
def folder(tmp_path):
    config = T.CONFIGS["narrow"]
    w = o.random_model(config, 5)
    return o.write_model(str(tmp_path / "m"), config, w), w


def reader(lib):
    lib.llmb200_tensor_file_open.restype, lib.llmb200_tensor_file_open.argtypes = C.c_void_p, [C.c_char_p]
    lib.llmb200_tensor_file_close.restype, lib.llmb200_tensor_file_close.argtypes = None, [C.c_void_p]
    lib.llmb200_tensor_f32.restype = C.POINTER(C.c_float)
    lib.llmb200_tensor_f32.argtypes = [C.c_void_p, C.c_char_p, C.c_longlong, C.c_longlong]
    return lib


def test_tensor_file_reads_what_was_written(lib, folder):
    path, w = folder
    lib = reader(lib)
    f = lib.llmb200_tensor_file_open(os.path.join(path, "model.safetensors").encode())
    assert f
    for name, v in w.items():
        p = lib.llmb200_tensor_f32(f, name.encode(), v.shape[0], v.shape[1] if v.ndim == 2 else 0)
        assert p, name
        assert np.array_equal(np.ctypeslib.as_array(p, shape=v.shape), v.astype(np.float32)), name
    assert not lib.llmb200_tensor_f32(f, b"no such tensor", 4, 0)
    assert not lib.llmb200_tensor_f32(f, b"embed", 96, 63)             # another shape
    assert not lib.llmb200_tensor_f32(f, b"embed", 96, 0)              # another rank
    lib.llmb200_tensor_file_close(f)


def test_tensor_file_types_and_damage(lib, tmp_path):
    lib = reader(lib)
    h = np.array([0.0, -0.0, 1.5, -2.25, 65504.0, 6e-8, 3.1e-5, np.inf], dtype=np.float16)
    s = np.array([1e-30, -3.25, 7.0], dtype=np.float32)

    def put(name, header, data):
        text = json.dumps(header).encode()
        (tmp_path / name).write_bytes(len(text).to_bytes(8, "little") + text + data)
        return str(tmp_path / name).encode()

    f = lib.llmb200_tensor_file_open(put("a", {"__metadata__": {"k": "é\\\"\n"}, "h": {"dtype": "F16", "shape": [8], "data_offsets": [0, 16]},
                                               "s": {"dtype": "F32", "shape": [3, 1], "data_offsets": [16, 28]},
                                               "i": {"dtype": "I32", "shape": [3], "data_offsets": [16, 28]},
                                               "long": {"dtype": "F32", "shape": [4], "data_offsets": [16, 32]},
                                               "short": {"dtype": "F32", "shape": [3], "data_offsets": [16, 24]}}, h.tobytes() + s.tobytes()))
    assert f
    assert np.array_equal(np.ctypeslib.as_array(lib.llmb200_tensor_f32(f, b"h", 8, 0), shape=(8,)), h.astype(np.float32))
    assert np.array_equal(np.ctypeslib.as_array(lib.llmb200_tensor_f32(f, b"s", 3, 1), shape=(3,)), s)
    for bad in (b"i", b"long", b"short"):                              # unsupported type, past the end, wrong size
        assert not lib.llmb200_tensor_f32(f, bad, 4 if bad == b"long" else 3, 0)
    lib.llmb200_tensor_file_close(f)
    (tmp_path / "b").write_bytes((1 << 40).to_bytes(8, "little") + b"{}")
    (tmp_path / "c").write_bytes((3).to_bytes(8, "little") + b"{]}")
    (tmp_path / "d").write_bytes(b"123")
    for name in ("b", "c", "d", "missing"):
        assert not lib.llmb200_tensor_file_open(str(tmp_path / name).encode())


def test_json_reader(lib):
    class Node(C.Structure):
        pass
    Node._fields_ = [("type", C.c_int), ("number", C.c_double), ("string", C.c_char_p), ("key", C.c_char_p),
                     ("child", C.POINTER(Node)), ("next", C.POINTER(Node)), ("n", C.c_int)]
    lib.json_parse.restype, lib.json_parse.argtypes = C.POINTER(Node), [C.c_char_p, C.c_size_t, C.POINTER(C.c_size_t)]
    lib.json_free.restype, lib.json_free.argtypes = None, [C.POINTER(Node)]

    def value(p):
        v = p.contents
        kids, k = [], v.child
        while k:
            kids.append((k.contents.key, value(k)))
            k = k.contents.next
        return [None, bool(v.number), v.number, (v.string or b"").decode("utf-8"), [b for _, b in kids],
                {a.decode(): b for a, b in kids if a is not None}][v.type]

    def parse(text):
        raw = text.encode()
        p = lib.json_parse(raw, len(raw), None)
        if not p:
            return "invalid"
        out = value(p)
        lib.json_free(p)
        return out

    for text in ('{"a": [1, -2.5e3, true, false, null, "x"], "b": {"c": {}}, "d": []}', ' [ ] ', '"\\u00e9\\ud83d\\ude00\\n\\"\\\\"', "12",
                 json.dumps(T.CONFIGS["wide"])):
        assert parse(text) == json.loads(text), text
    for text in ('{"a": }', '{"a" 1}', "[1,]", "[1 2]", "", "nul", '"abc', "1.2.3", '{"a": 1} x', "[" * 80 + "]" * 80, '"\\x"', '"\\u12"'):
        assert parse(text) == "invalid", text


def test_unusable_folders_are_refused(lib, folder, tmp_path):
    path, _ = folder
    create = lib.inference_state_create_from_dir
    assert not create(str(tmp_path / "nowhere").encode(), 64, 2)
    assert not create(path.encode(), 0, 2) and not create(path.encode(), 64, 1)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump({"architecture": "Something else"}, f)
    assert not create(path.encode(), 64, 2)
    with open(os.path.join(path, "config.json"), "w") as f:
        f.write("{")
    assert not create(path.encode(), 64, 2)


def test_command_line_help():
    for name in ("trace_run", "generate"):
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", name), "--help"], stdout=subprocess.PIPE, text=True, timeout=60)
        assert r.returncode == 0 and "--model" in r.stdout
        assert os.access(os.path.join(ROOT, "bin", name), os.X_OK)
