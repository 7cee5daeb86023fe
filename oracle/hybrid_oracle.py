"""Plain restatement of a Zidepel model (test infrastructure): numpy in float64, one function per mechanism, whole
sequences at a time, no cache; the recurrence is a loop over tokens. Shares no code with the library.

A model is (config, weights): `config` as config.json holds it, `weights` a dict name -> float array. `random_model`
makes small ones; latent_oracle.write_model puts one into a folder as the library reads it.
"""
import importlib.util
import os

import numpy as np

_spec = importlib.util.spec_from_file_location("latent_oracle", os.path.join(os.path.dirname(os.path.abspath(__file__)), "latent_oracle.py"))
_latent = importlib.util.module_from_spec(_spec)
_spec.loader.exec_module(_latent)
bf16, write_model, sub = _latent.bf16, _latent.write_model, _latent.sub


# ------------------------------------------------------------------ mechanisms

def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def embedding(tokens, table, positions, w, b, eps):
    t = np.asarray(tokens)
    return layer_norm(table[t] + positions[: len(t)], w, b, eps)


def query_temperature(n, q_temp):
    """Factor of the query at positions 0 .. n-1."""
    if not q_temp:
        return np.ones(n)
    return np.array([1.0 + q_temp["coef"] * np.log(np.floor((p + 1) / q_temp["every"]) + 1.0) for p in range(n)])


def capped(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def causal_softmax(s):
    """Rows i of s [n, n] over columns j <= i."""
    n = len(s)
    s = np.where(np.arange(n)[:, None] >= np.arange(n)[None, :], s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def attend(q, k, v, scale, cap):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim] -> [n, H, vdim]; query head h reads key head h // (H / G)."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.empty((n, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        out[:, h] = causal_softmax(capped(q[:, h] @ k[:, g].T * scale, cap)) @ v[:, g]
    return out


def attention(h, mix, w, eps):
    n, H, G, d, dv = len(h), mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms_norm((h @ w["q"].T).reshape(n, H, d), w["q.norm"], eps) * query_temperature(n, mix.get("q_temp"))[:, None, None]
    k = rms_norm((h @ w["k"].T).reshape(n, G, d), w["k.norm"], eps)
    v = (h @ w["v"].T).reshape(n, G, dv)
    return attend(q, k, v, mix["scale"], mix.get("softcap")).reshape(n, -1) @ w["o"].T


def decay(z, tau):
    """logistic(z) ** (1 / tau)"""
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def recurrence(q, k, v, a, state=None):
    """One head: q, k, a [n, dim], v [n, vdim] -> outputs [n, vdim] and the last state."""
    S = np.zeros((q.shape[1], v.shape[1])) if state is None else state.copy()
    out = np.empty_like(v)
    for t in range(len(q)):
        S = a[t][:, None] * S + np.outer(k[t], v[t])
        out[t] = q[t] @ S
    return out, S


def silu(z):
    return z / (1.0 + np.exp(-z))


def linear_attention(h, mix, w, eps):
    n, H, d, dv = len(h), mix["heads"], mix["dim"], mix["vdim"]
    q, k = (h @ w["q"].T).reshape(n, H, d) * d ** -0.5, (h @ w["k"].T).reshape(n, H, d)
    v = (h @ w["v"].T).reshape(n, H, dv)
    a = decay((h @ w["a1"].T) @ w["a2"].T + w["a2.b"], mix["tau"]).reshape(n, H, d)
    o = np.stack([recurrence(q[:, i], k[:, i], v[:, i], a[:, i])[0] for i in range(H)], axis=1)
    return (rms_norm(o, w["norm"], eps).reshape(n, -1) * silu(h @ w["g"].T)) @ w["o"].T


def feed_forward(h, w):
    return np.maximum(h @ w["up"].T, 0.0) ** 2 @ w["down"].T


def connect(streams, w, norm, sublayer):
    """One sublayer between the streams [s, n, D]: read a combination, spread the result, mix the old ones."""
    y = sublayer(norm(np.tensordot(w["in"], streams, axes=(0, 0))))
    return np.einsum("st,snd->tnd", w["mix"], streams) + w["out"][:, None, None] * y[None]


def order(config):
    """Layer indexes in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


MIXERS = {"attention": attention, "gla": linear_attention}


def forward(config, weights, tokens):
    """-> logits [n, vocab], and the sum of the streams after every layer run."""
    eps, w, after = config["norm"]["eps"], weights, []
    x = embedding(tokens, w["embed"], w["pos"], w["embed.norm"], w["embed.norm.b"], eps)
    streams = np.stack([x] * config["streams"])
    for i in order(config):
        layer, p = config["layers"][i], f"l{i}."
        mixer = MIXERS[layer["type"]]
        streams = connect(streams, sub(w, p + "hc1."), lambda u: layer_norm(u, w[p + "norm1"], w[p + "norm1.b"], eps),
                          lambda h: mixer(h, layer["mixer"], sub(w, p + "mix."), eps))
        if layer["mlp"]:
            streams = connect(streams, sub(w, p + "hc2."), lambda u: layer_norm(u, w[p + "norm2"], w[p + "norm2.b"], eps),
                              lambda h: feed_forward(h, sub(w, p + "mlp.")))
        after.append(streams.sum(axis=0))
    return layer_norm(streams.sum(axis=0), w["final.norm"], w["final.norm.b"], eps) @ w["head"].T, after


# ------------------------------------------------------------------ models

def attention_layer(heads, kv_heads, dim, vdim, ff, scale=None, cap=25.0, temp=(0.3, 64)):
    mix = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "softcap": cap,
           "q_temp": {"coef": temp[0], "every": temp[1]} if temp else None}
    return {"type": "attention", "mixer": mix, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def gla_layer(heads, dim, vdim, ff, tau, rank):
    """`rank` is no key of a configuration: it is the shape of a tensor (tensor_shapes reads it)."""
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "_rank": rank}


def model_config(width, vocab, streams, layers, loop=None, eps=1e-5, max_positions=512):
    """-> config.json's content and the ranks of the layers' decays."""
    ranks = [layer.get("_rank") for layer in layers]
    clean = [{k: v for k, v in layer.items() if k != "_rank"} for layer in layers]
    return {"architecture": "Zidepel", "vocab": vocab, "width": width, "streams": streams, "max_positions": max_positions, "norm": {"eps": eps},
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None, "layers": clean}, ranks


def tensor_shapes(config, ranks):
    D, V, n = config["width"], config["vocab"], config["streams"]
    s = {"embed": (V, D), "pos": (config["max_positions"], D), "head": (V, D)}
    for name in ("embed.norm", "final.norm"):
        s.update({name: (D,), name + ".b": (D,)})
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        for q in range(1, 3 if layer["mlp"] else 2):
            s.update({f"{p}norm{q}": (D,), f"{p}norm{q}.b": (D,), f"{p}hc{q}.in": (n,), f"{p}hc{q}.out": (n,), f"{p}hc{q}.mix": (n, n)})
        s.update({p + "mix.q": (H * d, D), p + "mix.o": (D, H * dv)})
        if layer["type"] == "attention":
            G = m["kv_heads"]
            s.update({p + "mix.k": (G * d, D), p + "mix.v": (G * dv, D), p + "mix.q.norm": (d,), p + "mix.k.norm": (d,)})
        else:
            r = ranks[i]
            s.update({p + "mix.k": (H * d, D), p + "mix.v": (H * dv, D), p + "mix.g": (H * dv, D), p + "mix.norm": (dv,), p + "mix.a1": (r, D),
                      p + "mix.a2": (H * d, r), p + "mix.a2.b": (H * d,)})
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            s.update({p + "mlp.up": (F, D), p + "mlp.down": (D, F)})
    return s


def random_model(config, ranks, seed, sharp=1.2):
    """Weights that keep every part in play: scores of spread about sharp^2, decays from a token to hundreds, stream
    connections away from their trivial values. The recurrences' keys lean towards their queries, so that a head's result
    is not a difference of nearly equal numbers before its norm. All are bfloat16 values."""
    rng = np.random.default_rng(seed)
    n, w = config["streams"], {}
    for name, shape in tensor_shapes(config, ranks).items():
        leaf = name.split(".", 1)[1] if name[0] == "l" else name
        z = rng.standard_normal(shape)
        if leaf.endswith(".in"):
            v = 1.0 / n + 0.1 * z
        elif leaf.endswith(".out"):
            v = 1.0 + 0.3 * z
        elif leaf.startswith("hc"):
            v = 0.8 * np.eye(n) + 0.2 * n ** -0.5 * z
        elif leaf == "mix.a2.b":
            v = 2.0 + 2.0 * z
        elif leaf.endswith(".b"):
            v = 0.2 * z
        elif leaf in ("mix.q.norm", "mix.k.norm"):
            v = sharp * (1.0 + 0.3 * z)
        elif len(shape) == 1:
            v = 1.0 + 0.2 * z
        elif leaf in ("embed", "pos"):
            v = 0.5 * z
        else:
            v = z * shape[1] ** -0.5 * (2.0 if leaf == "head" else 1.0)
            if leaf == "mix.k" and config["layers"][int(name[1:name.index(".")])]["type"] == "gla":
                v = 0.7 * w[name[:-1] + "q"] + 0.7 * v
        w[name] = bf16(v)
    return w
