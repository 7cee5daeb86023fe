"""Small Zidepel models for the tests, made by oracle/hybrid_oracle.py."""
import importlib.util
import os

import numpy as np

from _latent import errors, tokens  # noqa: F401

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_spec = importlib.util.spec_from_file_location("hybrid_oracle", os.path.join(ROOT, "oracle", "hybrid_oracle.py"))
o = importlib.util.module_from_spec(_spec)
_spec.loader.exec_module(o)

A, R = o.attention_layer, o.gla_layer
CONFIGS = {
    # both mixers with and without a feed-forward, different sizes in one model, a looped range of both kinds
    "mixed": o.model_config(72, 150, 4, [R(3, 20, 18, None, 8.0, 5), A(6, 2, 24, 16, 120, cap=20.0, temp=(0.2, 7)),
                                         R(2, 16, 24, 70, 2.0, 3), A(4, 4, 16, 40, None, scale=0.3, cap=9.0, temp=(0.7, 100))], loop=(1, 3, 2)),
    # sizes that are no multiples of 8, one key/value head, no cap, no query factor, no loop
    "odd": o.model_config(101, 203, 2, [A(5, 1, 33, 41, 67, cap=None, temp=None), R(2, 37, 70, 50, 16.0, 9), R(1, 12, 5, None, 1.0, 17)], eps=1e-3),
    # one stream, heads of one group each, values wider than a block, decays of tau 1, the loop over everything
    "one-stream": o.model_config(128, 96, 1, [R(2, 64, 136, 96, 1.0, 16), A(2, 2, 128, 128, 64)], loop=(0, 2, 3)),
    # many query heads per key head, head sizes beyond one pass of the kernels
    "wide": o.model_config(320, 520, 3, [A(12, 2, 160, 264, 256, cap=50.0, temp=(0.1, 33)), R(4, 72, 260, None, 4.0, 24), A(9, 3, 40, 72, 200, temp=(0.2, 1))],
                           loop=(2, 3, 2)),
    # smaller than every tile, the most streams, a loop of one pass
    "tiny": o.model_config(24, 30, 8, [R(1, 3, 2, 9, 3.0, 1), A(2, 1, 4, 3, 10, temp=(2.0, 5)), A(1, 1, 2, 6, None)], loop=(0, 1, 1), max_positions=400),
}
FAMILIES = list(CONFIGS)
LIMIT = {"float32": 3e-5, "bfloat16": 5e-2}
WIDER = {"tiny": 3.0}      # norms over two or three numbers: their differences of nearly equal numbers magnify every rounding


def limit(name, dtype):
    return LIMIT[dtype] * WIDER.get(name, 1.0)


def build(tmp_path_factory, name, seed=8):
    config, ranks = CONFIGS[name]
    weights = o.random_model(config, ranks, seed)
    return str(o.write_model(str(tmp_path_factory.mktemp(name)), config, weights)), config, weights
