"""Small Badepel configurations for the tests, and helpers that make their model folders.

The configurations differ from one another in every size and option: the order and kinds of the layers, one to five residual
streams and none, head counts and groups (also one head, and as many key/value heads as query heads), key and value sizes
(equal, wider, narrower; multiples of 4 and of 16, and not), score caps that bite and none, windows of 1 to 130 and none, the
whole head rotated, a part of it, nothing, convolutions of 1 to 5 taps and none, decay exponents 1 / tau, dense and routed
feed-forwards (one and several choices, with and without a shared expert of another limit, also none at all).
"""

from __future__ import annotations

from pathlib import Path

import torch

from acorninfer_b200.config.model_config import (AttentionBesideLinearConfig, BadepelConfig, BadepelLayer, CappedExpertsConfig,
                                                 GatedLinearConfig, HeadDeltaConfig, RowNormAttentionConfig)
from acorninfer_b200.weights.random_init import write_random_model
from acorninfer_b200.weights.safetensors_io import SafetensorsFile, write_safetensors


def att(heads, kv_heads, dim, scale, vdim=None, conv=None, cap=None, window=None, rot=0, base=100.0):
    return RowNormAttentionConfig(heads, kv_heads, dim, vdim if vdim is not None else dim, scale, conv, cap, window, rot,
                                  base if rot else 10000.0)


def gla(heads, dim, vdim, tau=4.0, rank=5):
    return GatedLinearConfig(heads, dim, vdim, tau, rank)


def both(left, right, left_scale=1.0, right_scale=1.0):
    return AttentionBesideLinearConfig(left, right, left_scale, right_scale)


def delta(heads, kv_heads, dim, vdim, conv=None):
    return HeadDeltaConfig(heads, kv_heads, dim, vdim, conv)


def moe(ff, experts, top, limit, shared=None, shared_limit=None):
    return CappedExpertsConfig(ff, limit, experts, top, shared, shared_limit)


def L(mixer, ff=None):
    return BadepelLayer(mixer.kind, mixer, ff)


BAD_A = dict(page_size=8, seed=51, cfg=BadepelConfig(
    vocab_size=170, hidden_size=72, norm_eps=1e-6, streams=2, residual_mult=0.7, layers=(
        L(both(att(heads=4, kv_heads=2, dim=6, vdim=10, scale=0.5, conv=3, cap=3.0, window=9, rot=4), gla(3, 5, 7, rank=3), 0.8, 1.3), ff=50),
        L(delta(heads=4, kv_heads=2, dim=6, vdim=9, conv=4), ff=moe(20, 5, 2, 1.2, 14, 0.9)),
        L(both(att(heads=3, kv_heads=3, dim=12, scale=0.4), gla(2, 8, 4, tau=1.0), 1.1, 0.6), ff=None),
        L(delta(heads=2, kv_heads=2, dim=12, vdim=4, conv=1), ff=moe(9, 3, 3, 2.0)),
    )))

BAD_B = dict(page_size=4, seed=52, cfg=BadepelConfig(
    vocab_size=141, hidden_size=60, norm_eps=1e-5, streams=5, residual_mult=1.0, layers=(
        L(delta(heads=3, kv_heads=1, dim=8, vdim=12), ff=48),
        L(both(att(heads=5, kv_heads=1, dim=8, vdim=4, scale=0.6, conv=5, window=1, rot=8), gla(1, 12, 20, tau=9.0), 0.5, 2.0),
          ff=moe(16, 4, 4, 0.7, 8, 3.0)),
        L(delta(heads=1, kv_heads=1, dim=20, vdim=16, conv=2), ff=None),
    )))

# sizes at which the bfloat16 engine takes its tensor-core paths, with and without padded heads
BAD_C = dict(page_size=16, seed=60, cfg=BadepelConfig(
    vocab_size=330, hidden_size=256, norm_eps=1e-5, streams=4, residual_mult=0.4, layers=(
        L(delta(heads=4, kv_heads=2, dim=64, vdim=32, conv=4), ff=192),
        L(both(att(heads=4, kv_heads=2, dim=64, scale=0.12, conv=4, cap=20.0, window=24, rot=32), gla(4, 32, 64, tau=16.0, rank=16), 1.2, 0.9),
          ff=moe(64, 6, 2, 1.5, 64, 2.5)),
        L(both(att(heads=6, kv_heads=2, dim=40, vdim=56, scale=0.15, conv=2, cap=8.0, rot=40), gla(2, 64, 48), 0.7, 1.0),
          ff=moe(32, 9, 1, 1.0, 128, 1.1)),
        L(both(att(heads=2, kv_heads=1, dim=128, scale=0.1, window=40, rot=64, conv=3), gla(2, 128, 128, tau=8.0), 1.0, 1.0), ff=64),
        L(delta(heads=2, kv_heads=1, dim=128, vdim=128, conv=3), ff=moe(40, 7, 3, 2.0)),
    )))

BAD_LONG = dict(page_size=16, seed=54, cfg=BadepelConfig(
    vocab_size=600, hidden_size=96, norm_eps=1e-5, streams=3, residual_mult=0.6, layers=(
        L(both(att(heads=4, kv_heads=2, dim=32, scale=0.25, conv=4, cap=10.0, window=70, rot=16), gla(3, 16, 32), 0.9, 1.1),
          ff=moe(24, 6, 2, 1.5, 16, 1.0)),
        L(delta(heads=6, kv_heads=3, dim=32, vdim=24, conv=4), ff=64),
        L(both(att(heads=3, kv_heads=3, dim=16, vdim=24, scale=0.3, window=130, conv=2, rot=16), gla(2, 70, 36, tau=12.0), 1.2, 0.8)),
        L(delta(heads=2, kv_heads=1, dim=64, vdim=64, conv=2), ff=moe(32, 5, 1, 1.8)),
    )))

BADEPELS = {"bad_a": BAD_A, "bad_b": BAD_B, "bad_c": BAD_C}


def read_weights(model_dir: Path) -> dict[str, torch.Tensor]:
    f = SafetensorsFile(Path(model_dir) / "model.safetensors")
    return {n: f.tensor(n).clone() for n in f.entries}


def make_model_dir(tmp: Path, tiny: dict, sigma: float = 0.12, sigma_norm: float = 0.2) -> Path:
    """A folder of random weights.  The router's biases are spread wide, so that few choices of experts hang on a hair: under
    bfloat16 such a choice may fall the other way and, through the recurrent states, change every later position."""
    d = write_random_model(tmp, tiny["cfg"], tiny["seed"], sigma, sigma_norm)
    w = read_weights(d)
    for name in w:
        if name.endswith("router.b"):
            w[name] = w[name] * 8
    write_safetensors(d / "model.safetensors", w, {"format": "pt"})
    return d


def random_config(seed: int) -> BadepelConfig:
    """A configuration drawn at random: 2 to 5 layers with both kinds of mixer, sizes from lists that hold what real
    models have (heads of 32 to 128) beside odd ones."""
    import random
    rng = random.Random(seed)
    width = rng.choice([128, 160, 320, 512])
    n = rng.randint(2, 5)
    order = [rng.choice(["both", "delta"]) for _ in range(n)]
    at = rng.randrange(n)
    order[at], order[(at + 1) % n] = "both", "delta"
    layers = []
    for k in order:
        ff = rng.choice([None, 200, 256, moe(rng.choice([32, 48, 96]), rng.choice([4, 8, 12]), rng.choice([1, 2, 4]), rng.choice([1.0, 2.0, 7.0]),
                                             *rng.choice([(None, None), (32, 1.5), (64, 0.8)]))])
        if k == "delta":
            kv = rng.choice([1, 2, 3])
            layers.append(L(delta(kv * rng.choice([1, 2, 3]), kv, rng.choice([16, 32, 64, 96, 128, 20]), rng.choice([16, 32, 64, 128, 36]),
                                  conv=rng.choice([None, 2, 4, 4, 6])), ff))
            continue
        kv = rng.choice([1, 2, 4])
        d = rng.choice([32, 64, 96, 128, 40])
        left = att(kv * rng.choice([1, 2, 3, 4]), kv, d, d ** -0.5, vdim=rng.choice([d, d, d, 48, 80]), conv=rng.choice([None, 2, 4, 4]),
                   cap=rng.choice([None, 5.0, 30.0]), window=rng.choice([None, 16, 50, 128]), rot=rng.choice([0, d // 2, d]), base=rng.choice([1e3, 1e6]))
        right = gla(rng.choice([1, 2, 3, 8]), rng.choice([16, 32, 64, 128, 18]), rng.choice([32, 64, 128, 50]), tau=rng.choice([1.0, 8.0, 16.0]),
                    rank=rng.choice([4, 16, 24]))
        layers.append(L(both(left, right, rng.choice([1.0, 0.7, 1.4]), rng.choice([1.0, 0.5, 1.2])), ff))
    return BadepelConfig(vocab_size=rng.choice([300, 520, 1000]), hidden_size=width, norm_eps=rng.choice([1e-5, 1e-6]),
                         layers=tuple(layers), streams=rng.choice([None, 1, 2, 3, 4, 6]), residual_mult=rng.choice([1.0, 0.5, 0.31]))
