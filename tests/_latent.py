"""Small Morilorn models for the tests, made by oracle/latent_oracle.py."""
import importlib.util
import os

import numpy as np

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_spec = importlib.util.spec_from_file_location("latent_oracle", os.path.join(ROOT, "oracle", "latent_oracle.py"))
o = importlib.util.module_from_spec(_spec)
_spec.loader.exec_module(o)

L = o.layer_config
CONFIGS = {
    # sizes that are no multiples of 8, a layer without a feed-forward, different layers in one model
    "odd": o.model_config(102, 203, [L(3, 20, 12, 18, 37, 21, 130), L(5, 9, 6, 7, 50, 40, None, scale=0.3, base=500.0),
                                     L(2, 33, 4, 41, 29, 7, 67, base=100.0)], groups=3, eps=1e-4, alpha=2.5, emb_scale=3.0, cap=9.0),
    # one head, one group, window of one token next to a wide one
    "narrow": o.model_config(64, 96, [L(1, 16, 8, 24, 24, 1, 48), L(1, 8, 16, 8, 40, 300, 80)], groups=1, alpha=1.0, cap=30.0),
    # more heads than one block of the decode scores holds; latent and value sizes beyond one pass
    "wide": o.model_config(320, 520, [L(18, 40, 24, 72, 300, 150, 256), L(9, 64, 32, 136, 96, 33, 200)], groups=5, alpha=3.5, emb_scale=6.0),
    # smaller than every tile and than the narrowest tensor-core product
    "tiny": o.model_config(24, 30, [L(1, 4, 2, 3, 5, 6, 10), L(2, 3, 4, 1, 8, 33, 9, base=30.0)], groups=4, emb_scale=1.0, alpha=2.0, cap=5.0),
    # the last layer has no feed-forward
    "bare-end": o.model_config(80, 136, [L(4, 16, 16, 16, 32, 50, 96, base=1000.0), L(4, 24, 8, 32, 48, 64, None)], groups=2),
}
FAMILIES = list(CONFIGS)


def build(tmp_path_factory, name, seed=7):
    config = CONFIGS[name]
    weights = o.random_model(config, seed)
    return str(o.write_model(str(tmp_path_factory.mktemp(name)), config, weights)), config, weights


def tokens(config, n, seed=0):
    return np.random.default_rng(seed).integers(0, config["vocab"], n).tolist()


def errors(got, want):
    """Per position: rms difference of the logits, mean taken off, over the spread of the expected ones."""
    d = np.asarray(got, dtype=np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / want.std()


LIMIT = {"float32": 3e-5, "bfloat16": 4e-2}
