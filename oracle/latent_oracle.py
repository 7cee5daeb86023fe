"""Plain restatement of a Morilorn model (test infrastructure): numpy in float64, one function per mechanism,
whole sequences at a time, no cache. Shares no code with the library.

A model is (config, weights): `config` as config.json holds it, `weights` a dict name -> float array. `random_model`
makes small ones, `write_model` puts one into a folder as the library reads it.
"""
import json
import os

import numpy as np


# ------------------------------------------------------------------ mechanisms

def logistic(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms(x, gamma, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gamma


def group_rms(x, gamma, groups, eps):
    """Equal consecutive parts, each over its own root mean square; the weight runs over the whole vector."""
    parts = np.split(x, groups, axis=-1)
    return np.concatenate([p / np.sqrt(np.mean(p * p, axis=-1, keepdims=True) + eps) for p in parts], axis=-1) * gamma


def rotate(v, positions, base, dims):
    """Pairs (2i, 2i+1) of the last axis, i < dims/2, turned by position * base^(-2i/dims); positions run over axis 0."""
    out = v.copy()
    for i in range(dims // 2):
        a = positions * base ** (-2.0 * i / dims)
        c, s = (f(a).reshape((-1,) + (1,) * (v.ndim - 2)) for f in (np.cos, np.sin))
        x, y = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = x * c - y * s, y * c + x * s
    return out


def visible(n, window):
    """[i, j]: position i may look at position j."""
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & ((d < window) if window else True)


def softmax(scores, mask):
    s = np.where(mask, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent(h, mix, w_dkv, gamma, eps):
    """The low-rank vector and the shared rotated key part of every position."""
    R = mix["kv_rank"]
    kv = h @ w_dkv.T
    return rms(kv[:, :R], gamma, eps), rotate(kv[:, R:], np.arange(len(h)), mix["rot"]["base"], mix["rot"]["dims"])


def attend(q, c, kr, mix, w_uk, w_uv):
    """q [n, heads, dim + rot_dim] (not rotated yet), c and kr of every position -> [n, heads, vdim]."""
    n, H, d = len(q), mix["heads"], mix["dim"]
    keys, values = (c @ w_uk.T).reshape(n, H, d), (c @ w_uv.T).reshape(n, H, mix["vdim"])
    qr = rotate(q[..., d:], np.arange(n), mix["rot"]["base"], mix["rot"]["dims"])
    mask = visible(n, mix["mask"]["size"] if mix.get("mask") else None)
    out = np.empty((n, H, mix["vdim"]))
    for h in range(H):
        scores = (q[:, h, :d] @ keys[:, h].T + qr[:, h] @ kr.T) * mix["scale"]
        out[:, h] = softmax(scores, mask) @ values[:, h]
    return out


def mixer(h, mix, w, eps):
    n = len(h)
    q = (h @ w["q"].T).reshape(n, mix["heads"], mix["dim"] + mix["rot_dim"])
    c, kr = latent(h, mix, w["dkv"], w["dkv.norm"], eps)
    o = attend(q, c, kr, mix, w["uk"], w["uv"]).reshape(n, -1)
    return (o * logistic(h @ w["g"].T)) @ w["o"].T


def feed_forward(h, w):
    return (gelu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def gated_postnorm(x, y, gate, bias, alpha, gamma, groups, eps):
    return group_rms(alpha * x + logistic(gate + bias) * y, gamma, groups, eps)


def depth_average(results, coef):
    return sum(c * r for c, r in zip(coef, results))


def softcap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens):
    """-> logits [n, vocab], and what every layer hands on."""
    eps, groups, alpha = config["norm"]["eps"], config["norm"]["groups"], config["postln_alpha"]
    w = weights
    x = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    results, handed_on = [x], []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        u = gated_postnorm(x, mixer(x, layer["mixer"], sub(w, p + "mix."), eps), x @ w[p + "rg1"].T, w[p + "rg1.b"], alpha,
                           w[p + "norm1"], groups, eps)
        if layer["mlp"]:
            u = gated_postnorm(u, feed_forward(u, sub(w, p + "mlp.")), u @ w[p + "rg2"].T, w[p + "rg2.b"], alpha, w[p + "norm2"],
                               groups, eps)
        results.append(u)
        x = depth_average(results, w[p + "dwa"])
        handed_on.append(x)
    logits = group_rms(x, w["final.norm"], groups, eps) @ w["head"].T
    return softcap(logits, config.get("logit_softcap")), handed_on


# ------------------------------------------------------------------ models

def bf16(x):
    """Nearest bfloat16 value (ties to even)."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32).astype(np.float64)


def layer_config(heads, dim, rot_dim, vdim, kv_rank, window, ff, scale=None, base=10000.0):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot_dim}, "scale": scale or (dim + rot_dim) ** -0.5},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model_config(width, vocab, layers, groups=1, eps=1e-5, alpha=1.5, emb_scale=4.0, cap=20.0):
    return {"architecture": "Morilorn", "vocab": vocab, "width": width, "embedding": {"scale": emb_scale},
            "norm": {"eps": eps, "groups": groups}, "postln_alpha": alpha, "logit_softcap": cap, "layers": layers}


def tensor_shapes(config):
    D, V = config["width"], config["vocab"]
    s = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        H, R = m["heads"], m["kv_rank"]
        s.update({p + "norm1": (D,), p + "rg1": (D, D), p + "rg1.b": (D,), p + "dwa": (i + 2,),
                  p + "mix.q": (H * (m["dim"] + m["rot_dim"]), D), p + "mix.dkv": (R + m["rot_dim"], D), p + "mix.dkv.norm": (R,),
                  p + "mix.uk": (H * m["dim"], R), p + "mix.uv": (H * m["vdim"], R), p + "mix.g": (H * m["vdim"], D),
                  p + "mix.o": (D, H * m["vdim"])})
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            s.update({p + "norm2": (D,), p + "rg2": (D, D), p + "rg2.b": (D,), p + "mlp.gate": (F, D), p + "mlp.up": (F, D),
                      p + "mlp.down": (D, F)})
    return s


def random_model(config, seed, sharp=2.0):
    """Weights that keep every part in play: scores of spread about `sharp` (single keys stand out), gates and depth
    weights away from their trivial values. All are bfloat16 values."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if len(shape) == 1:
            if leaf == "dwa":
                v = 0.25 * rng.standard_normal(shape)
                v[-1] += 1.0
            elif leaf == "b":
                v = 0.5 * rng.standard_normal(shape)
            else:
                v = 1.0 + 0.2 * rng.standard_normal(shape)
        else:
            v = rng.standard_normal(shape) * shape[1] ** -0.5
            if leaf == "q":
                v *= sharp
            if leaf == "embed":
                v = 0.3 * rng.standard_normal(shape)
            if leaf == "head":
                v *= 4.0
        w[name] = bf16(v)
    return w


def write_model(folder, config, weights):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    header, blobs, at = {}, [], 0
    for name, v in weights.items():
        raw = (np.ascontiguousarray(v, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for b in blobs:
            f.write(b)
    return folder
