"""Small Zusolix configurations for the tests, and helpers that make their model folders.

The configurations differ from one another in every size and option: the order and kinds of the layers, head counts and
groups (also one head, and as many key/value heads as query heads), key and value sizes (equal, wider, narrower), score
caps that bite and none, query temperatures (spans of 1 to 40 positions, a negative coefficient, none), minGRU widths
below and above the model's and no multiple of 4, norms in 1 to 6 groups (parts that are and are not multiples of 128),
factors on the token rows and on a layer's results (also 1), dense and routed feed-forwards (one and several choices,
with and without a shared expert, also none at all), a single layer.
"""

from __future__ import annotations

from pathlib import Path

import torch

from acorninfer_b200.config.model_config import (InputWeightedExpertsConfig, MinGRUConfig, TemperedAttentionConfig, ZusolixConfig,
                                                 ZusolixLayer)
from acorninfer_b200.weights.random_init import write_random_model
from acorninfer_b200.weights.safetensors_io import SafetensorsFile


def att(heads, kv_heads, dim, scale, vdim=None, cap=None, coef=0.0, every=None):
    return TemperedAttentionConfig(heads, kv_heads, dim, vdim if vdim is not None else dim, scale, cap, coef, every)


def gru(width):
    return MinGRUConfig(width)


def moe(ff, experts, top, shared=None):
    return InputWeightedExpertsConfig(ff, experts, top, shared)


def L(mixer, ff=None):
    return ZusolixLayer(mixer.kind, mixer, ff)


ZUS_A = dict(page_size=8, seed=41, cfg=ZusolixConfig(
    vocab_size=170, hidden_size=72, norm_eps=1e-6, norm_groups=3, residual_mult=0.7, embedding_scale=3.0, layers=(
        L(att(heads=4, kv_heads=2, dim=6, vdim=10, scale=0.5, cap=3.0, coef=0.8, every=5), ff=50),
        L(gru(30), ff=moe(20, 5, 2, 14)),
        L(att(heads=3, kv_heads=3, dim=12, scale=0.3), ff=None),
        L(gru(101), ff=moe(9, 3, 3)),
    )))

ZUS_B = dict(page_size=4, seed=42, cfg=ZusolixConfig(
    vocab_size=141, hidden_size=60, norm_eps=1e-5, norm_groups=1, residual_mult=1.0, embedding_scale=1.0, layers=(
        L(gru(44), ff=48),
        L(gru(60), ff=None),
        L(att(heads=5, kv_heads=1, dim=8, vdim=4, scale=0.4, cap=1.0, coef=-0.1, every=1), ff=moe(16, 4, 4, 8)),
    )))

# sizes at which the bfloat16 engine takes its tensor-core paths
ZUS_C = dict(page_size=16, seed=43, cfg=ZusolixConfig(
    vocab_size=330, hidden_size=256, norm_eps=1e-5, norm_groups=2, residual_mult=0.3, embedding_scale=2.5, layers=(
        L(att(heads=4, kv_heads=2, dim=64, scale=0.15, cap=20.0, coef=0.25, every=16), ff=192),
        L(gru(320), ff=moe(64, 6, 2, 64)),
        L(att(heads=2, kv_heads=1, dim=128, scale=0.1, cap=8.0, coef=0.5, every=40), ff=moe(32, 9, 1, 128)),
        L(att(heads=8, kv_heads=1, dim=32, scale=0.2, coef=0.1, every=7), ff=64),
        L(gru(96), ff=moe(40, 7, 3)),
    )))

ZUS_LONG = dict(page_size=16, seed=44, cfg=ZusolixConfig(
    vocab_size=600, hidden_size=96, norm_eps=1e-5, norm_groups=6, residual_mult=0.6, embedding_scale=4.0, layers=(
        L(att(heads=4, kv_heads=2, dim=32, scale=0.25, cap=10.0, coef=0.4, every=48), ff=moe(24, 6, 2, 16)),
        L(gru(136), ff=64),
        L(att(heads=3, kv_heads=3, dim=16, vdim=24, scale=0.3, cap=25.0), ff=None),
        L(gru(50), ff=moe(32, 5, 1)),
    )))

ZUSES = {"zus_a": ZUS_A, "zus_b": ZUS_B, "zus_c": ZUS_C}


def read_weights(model_dir: Path) -> dict[str, torch.Tensor]:
    f = SafetensorsFile(Path(model_dir) / "model.safetensors")
    return {n: f.tensor(n).clone() for n in f.entries}


def make_model_dir(tmp: Path, tiny: dict, sigma: float = 0.12, sigma_norm: float = 0.2) -> Path:
    return write_random_model(tmp, tiny["cfg"], tiny["seed"], sigma, sigma_norm)


def random_config(seed: int) -> ZusolixConfig:
    """A configuration drawn at random: 2 to 6 layers with both kinds of mixer, sizes from lists that hold what real
    models have (heads of 32 to 128) beside odd ones."""
    import random
    rng = random.Random(seed)
    width = rng.choice([128, 160, 320, 512])
    n = rng.randint(2, 6)
    order = [rng.choice(["attention", "attention", "mingru"]) for _ in range(n)]
    order[rng.randrange(n)] = "attention"
    order[(order.index("attention") + 1) % n] = "mingru"
    layers = []
    for k in order:
        ff = rng.choice([None, 200, 256, moe(rng.choice([32, 48, 96]), rng.choice([4, 8, 12]), rng.choice([1, 2, 4]),
                                             rng.choice([None, 32, 64]))])
        if k == "mingru":
            layers.append(L(gru(rng.choice([width, 64, 200, 513, 768])), ff))
            continue
        kv = rng.choice([1, 2, 4])
        d = rng.choice([32, 64, 96, 128, 40])
        every = rng.choice([None, 1, 16, 50, 128])
        layers.append(L(att(kv * rng.choice([1, 2, 3, 4]), kv, d, d ** -0.5, vdim=rng.choice([d, d, d, 48]),
                            cap=rng.choice([None, 5.0, 30.0]), coef=rng.choice([0.1, 0.4]) if every else 0.0, every=every), ff))
    return ZusolixConfig(vocab_size=rng.choice([300, 520, 1000]), hidden_size=width, norm_eps=rng.choice([1e-5, 1e-6]),
                         layers=tuple(layers), norm_groups=rng.choice([1, 2, 4, 8]), residual_mult=rng.choice([1.0, 0.5, 0.31]),
                         embedding_scale=rng.choice([1.0, 3.0, 8.0]))
