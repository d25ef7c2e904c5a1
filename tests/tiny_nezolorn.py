"""Tiny Nezolorn configurations for the tests.

They differ from one another in every size: width, vocabulary, the residual factor, rows and multipliers of the pair
embedding, query and key/value heads, head sizes, window and block lengths (blocks longer than the window among them),
rotated dimensions and their scaling, softmax scale, the two sides' factors, heads and sizes of the matrix memory and
its gates' cap, heads, sizes and thin rank of the delta rule, feed-forward sizes and none, and the order of the layers.
A side's factor of 0 leaves the other side alone.
"""
from __future__ import annotations

import copy
from pathlib import Path

import torch

from tiny_fivitar import judge, row_errors, trace_portions  # noqa: F401  (the same rules of judgement)

BANDS = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 96}


def _left(heads, kv, dim, size, pool, dims=None, base=10000.0, scaling=None, scale=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5,
         "mask": {"size": size, "pool": pool}}
    if dims is not None:
        m["rot"] = {"base": base, "dims": dims}
        if scaling is not None:
            m["rot"]["scaling"] = dict(scaling)
    return m


def _right(heads, dim, vdim, cap=15.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _parallel(left, right, ls=1.0, rs=1.0, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": ls, "right_scale": rs},
            "mlp": _dense(ff)}


def _delta(heads, dim, rank, ff=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim, "rank": rank}, "mlp": _dense(ff)}


def _dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def _pairs(buckets, prev, cur):
    return {"buckets": buckets, "mul_prev": prev, "mul_cur": cur}


TINY = {
    # each mechanism alone
    "window": dict(vocab=300, width=64, eps=1e-5, emb=4.0, mult=0.7, seed=61, std=0.1, norm_std=0.1, pairs=_pairs(97, 37, 11),
                   layers=[_parallel(_left(6, 3, 8, 20, 4, dims=6, base=100.0, scaling=BANDS, scale=0.9), _right(1, 8, 8), 1.3, 0.0)]),
    "blocks": dict(vocab=290, width=48, eps=1e-6, emb=3.0, mult=1.0, seed=62, std=0.12, norm_std=0.1, pairs=_pairs(50, 3, 11),
                   layers=[_parallel(_left(4, 2, 12, 5, 9, dims=12, base=40.0, scale=1.1), _right(1, 8, 8), 0.8, 0.0)]),
    "memory": dict(vocab=260, width=40, eps=1e-5, emb=3.0, mult=0.5, seed=63, std=0.15, norm_std=0.1, pairs=_pairs(33, 2, 5),
                   layers=[_parallel(_left(1, 1, 8, 8, 4), _right(3, 12, 20, cap=6.0), 0.0, 1.1)]),
    "delta": dict(vocab=270, width=48, eps=1e-5, emb=2.0, mult=0.6, seed=64, std=0.15, norm_std=0.1, pairs=_pairs(64, 17, 29),
                  layers=[_delta(3, 20, 6)]),
    "dense": dict(vocab=280, width=48, eps=1e-5, emb=2.0, mult=0.4, seed=65, std=0.1, norm_std=0.1, pairs=_pairs(512, 97, 13),
                  layers=[_delta(2, 16, 8, ff=100)]),
    # everything, in another order than any other configuration's
    "mix": dict(vocab=411, width=96, eps=2e-6, emb=9.0, mult=0.35, seed=66, std=0.08, norm_std=0.15, pairs=_pairs(301, 1009, 65537),
                layers=[_delta(4, 24, 10, ff=128),
                        _parallel(_left(6, 2, 16, 24, 6, dims=16, base=300.0, scaling=dict(BANDS, factor=8.0, low=0.5)), _right(5, 16, 40, cap=9.0), 1.2, 0.9, ff=160),
                        _parallel(_left(3, 3, 24, 33, 1, dims=10, base=5000.0), _right(2, 32, 24), 0.7, 1.4),
                        _delta(1, 40, 3),
                        _parallel(_left(4, 1, 8, 3, 16, dims=4, base=50.0), _right(2, 64, 32, cap=3.0), 1.0, 1.0, ff=64)]),
    # head sizes the tensor-core kernels take, a group of more than 16 query heads per key/value head, heads of 128
    "tc": dict(vocab=300, width=128, eps=1e-5, emb=3.0, mult=0.3, seed=67, std=0.05, norm_std=0.1, pairs=_pairs(200, 5, 3),
               layers=[_parallel(_left(4, 2, 64, 40, 8, dims=64, base=1000.0, scaling=BANDS), _right(2, 128, 64), 1.1, 0.8, ff=96),
                       _parallel(_left(2, 1, 128, 70, 5, dims=128, base=30000.0), _right(1, 64, 128), 0.9, 1.2, ff=64),
                       _delta(2, 64, 16, ff=64),
                       _parallel(_left(34, 2, 16, 17, 3, dims=8, base=70.0), _right(3, 16, 96), 1.0, 0.5)]),
    # prompts of a thousand tokens on pages of 64: windows and blocks that several tiles of keys and of blocks make up
    "long": dict(vocab=384, width=192, eps=1e-5, emb=2.0, mult=0.45, seed=68, std=0.06, norm_std=0.1, pairs=_pairs(700, 41, 6),
                 layers=[_parallel(_left(4, 2, 128, 100, 2, dims=128, base=10000.0, scaling=dict(BANDS, original=512)), _right(3, 32, 48), 1.0, 0.7, ff=256),
                         _delta(3, 48, 24, ff=160),
                         _parallel(_left(6, 3, 48, 190, 24, dims=32, base=900.0), _right(4, 24, 64, cap=12.0), 0.8, 1.1),
                         _parallel(_left(2, 2, 128, 64, 64, dims=64, base=250000.0), _right(2, 96, 32), 1.2, 1.0, ff=96)]),
    # sizes that are multiples of nothing the kernels like
    "odd": dict(vocab=263, width=50, eps=1e-5, emb=2.5, mult=0.9, seed=69, std=0.1, norm_std=0.1, pairs=_pairs(31, 7, 3),
                layers=[_parallel(_left(3, 3, 6, 11, 5, dims=2, base=40.0, scaling=dict(BANDS, factor=1.5)), _right(3, 10, 7, cap=4.5), 0.6, 1.7, ff=30),
                        _delta(3, 11, 5),
                        _parallel(_left(5, 1, 10, 7, 3), _right(1, 5, 33), 1.5, 0.4)]),
    # ones everywhere: one head, a window of one token, blocks of one token, one bucket, a thin rank of one
    "ones": dict(vocab=257, width=48, eps=1e-5, emb=1.0, mult=1.0, seed=70, std=0.1, norm_std=0.2, pairs=_pairs(1, 1, 1),
                 layers=[_delta(1, 8, 1, ff=48),
                         _parallel(_left(1, 1, 8, 1, 1, dims=8, base=10.0), _right(1, 4, 1, cap=1.0), 1.0, 1.0, ff=24)]),
}


def config_dict(name: str) -> dict:
    t = TINY[name]
    return {"architecture": "Nezolorn", "vocab": t["vocab"], "width": t["width"],
            "embedding": {"scale": t["emb"], "bigram": dict(t["pairs"])}, "norm": {"eps": t["eps"]},
            "residual_mult": t["mult"], "layers": copy.deepcopy(t["layers"])}


def make_config(name: str):
    from garlic_inference_b200.config import NezolornConfig
    return NezolornConfig.from_dict(config_dict(name))


def write_model(name: str, folder) -> Path:
    from garlic_inference_b200 import write_random_model
    t = TINY[name]
    return write_random_model(folder, make_config(name), seed=t["seed"], std=t["std"], norm_std=t["norm_std"])


def plain_logits(model_dir, requests, dtype=torch.float32) -> dict:
    import plain_nezolorn as plain
    cfg, weights = plain.read_model_dir(model_dir)
    return {rid: plain.forward(cfg, weights, toks, dtype).to(torch.float64).numpy() for rid, toks in requests.items()}


def plain_pair(model_dir, requests):
    """(float64 logits, float32 logits) of the plain model for every request."""
    return plain_logits(model_dir, requests, torch.float64), plain_logits(model_dir, requests, torch.float32)
