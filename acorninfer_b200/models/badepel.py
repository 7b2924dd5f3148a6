"""Badepel as data: which parts each layer has, with which sizes, in which order.

The token rows as several equal residual streams; layers in the ``hyper`` arrangement (every sublayer reads a learned sum of
the streams through an RMS norm and writes back to all of them while a matrix mixes them; one plain stream where the
configuration names none).  A layer's mixer is ``side_by_side`` of ``attention`` with the options this design uses (biased
and convolved projections, a q/k norm over whole rows, neighbouring rotary pairs, capped scores, a window, a sink fixed at
zero) and ``gated_linear_attention``; or ``head_delta``.  Its feed-forward is ``gated`` with silu, ``routed_experts`` of the capped
form (a bias on the router's logits, weights over the chosen only) beside a shared expert, or absent.  The streams' sum goes
through the final norm to an output matrix of its own.

Tensor names: ``embed``, ``l<i>.norm1`` / ``norm2``, ``l<i>.hc1.*`` / ``hc2.*``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.model_config import (AttentionBesideLinearConfig, BadepelConfig, CappedExpertsConfig, HeadDeltaConfig,
                                   RowNormAttentionConfig)
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture

_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "q_norm": "q.norm",
                    "k_norm": "k.norm", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}
_FF_NAMES = {"gate": "gate", "up": "up", "down": "down"}


def _position(m: RowNormAttentionConfig, positions: dict) -> str | None:
    """Name of the position encoding for these rotary settings (made on first use)."""
    if m.rot_dims == 0:
        return None
    key = (m.dim, m.rot_dims, m.rot_base)
    for name, (k, _) in positions.items():
        if k == key:
            return name
    name = f"rot{len(positions)}"
    positions[name] = (key, PartSpec("rope", {"head_dim": m.dim, "rotary_dim": m.rot_dims, "theta": m.rot_base,
                                              "pairing": "interleaved", "exact": True}))
    return name


def badepel_spec(cfg: BadepelConfig) -> ModelSpec:
    W, eps = cfg.hidden_size, cfg.norm_eps
    positions: dict = {}
    layers = []

    def norm(name):
        return PartSpec("rmsnorm", {"width": W, "eps": eps, "tensor": ""}, name)

    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, AttentionBesideLinearConfig):
            a, r = m.left, m.right
            left = PartSpec("attention", {
                "hidden_size": W, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim, "value_dim": a.vdim,
                "position": _position(a, positions), "scale": a.scale, "qk_norm_eps": eps, "qk_norm_rows": True, "bias": True,
                "conv_taps": a.conv, "softcap": a.softcap, "window": a.window, "unit_sink": True, "pad_heads": True,
                "names": _ATTENTION_NAMES}, "left.")
            right = PartSpec("gated_linear_attention", {
                "hidden_size": W, "num_heads": r.heads, "dim": r.dim, "vdim": r.vdim, "tau": r.tau, "norm_eps": eps,
                "decay_rank": r.decay_rank}, "right.")
            mixer = PartSpec("side_by_side", {"left": left, "right": right, "left_scale": m.left_scale,
                                              "right_scale": m.right_scale}, p + "mix.")
        else:
            assert isinstance(m, HeadDeltaConfig)
            mixer = PartSpec("head_delta", {"hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "dim": m.dim,
                                            "vdim": m.vdim, "taps": m.conv, "norm_eps": eps}, p + "mix.")
        norms = {"mixer": norm(p + "norm1")}
        ff = None
        if isinstance(layer.ff, CappedExpertsConfig):
            f = layer.ff
            ff = PartSpec("routed_experts", {
                "hidden_size": W, "expert_size": f.ff, "num_experts": f.experts, "num_identity": 0, "top": f.top,
                "correction": False, "normalize": True, "activation": "capped_swish", "limit": f.limit, "shared_size": f.shared_ff,
                "shared_limit": f.shared_limit, "router_bias": True}, p + "mlp.")
        elif layer.ff is not None:
            ff = PartSpec("gated", {"hidden_size": W, "intermediate_size": layer.ff, "activation": "silu",
                                    "names": _FF_NAMES}, p + "mlp.")
        if ff is not None:
            norms["feed_forward"] = norm(p + "norm2")
        block = PartSpec("hyper", {"streams": cfg.streams or 1, "residual_scale": cfg.residual_mult,
                                   "learned": cfg.streams is not None}, p)
        layers.append(LayerSpec(block, mixer, ff, norms))
    # a layer without feed-forward has nothing that would read a second norm or a second set of stream factors
    spare = tuple(f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if layer.ff is None
                  for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix"))
    return ModelSpec(
        vocab_size=cfg.vocab_size, hidden_size=W, embedding="embed", layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=norm("final.norm"), head="head",
        positions={name: spec for name, (_, spec) in positions.items()}, streams=cfg.streams or 1, ignorable=spare)


register_architecture(BadepelConfig.architecture, BadepelConfig, badepel_spec)
