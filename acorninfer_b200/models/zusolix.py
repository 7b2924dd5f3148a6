"""Zusolix as data: which parts each layer has, with which sizes, in which order.

The token rows times a factor; layers in the ``parallel`` arrangement with a norm per sublayer and a factor on the sum of
both results (``x + m (mixer(norm1(x)) + ff(norm2(x)))``), the norms RMS norms in groups.  A layer's mixer is ``attention``
with the options this design uses (biased projections, no rotation, a query temperature, capped scores) or ``min_gru``;
its feed-forward is ``gated`` with silu, ``routed_experts`` with sigmoid scores on the experts' inputs beside a shared
expert with a gate, or absent.  After every layer the ``depth_average`` stream mix makes the stream that goes on.  The final
norm is one in groups too; the output matrix is the model's own.

Tensor names: ``embed``, ``l<i>.norm1`` / ``norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.dwa``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.model_config import InputWeightedExpertsConfig, MinGRUConfig, TemperedAttentionConfig, ZusolixConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture

_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b"}
_FF_NAMES = {"gate": "gate", "up": "up", "down": "down"}


def zusolix_spec(cfg: ZusolixConfig) -> ModelSpec:
    W = cfg.hidden_size
    layers = []

    def norm(name):
        return PartSpec("grouped_rmsnorm", {"width": W, "eps": cfg.norm_eps, "groups": cfg.norm_groups, "tensor": ""}, name)

    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, TemperedAttentionConfig):
            mixer = PartSpec("attention", {
                "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
                "position": None, "scale": m.scale, "bias": True, "softcap": m.softcap,
                "q_temp": None if m.temp_every is None else (m.temp_coef, m.temp_every), "names": _ATTENTION_NAMES}, p + "mix.")
        else:
            assert isinstance(m, MinGRUConfig)
            mixer = PartSpec("min_gru", {"hidden_size": W, "width": m.width}, p + "mix.")
        norms = {"mixer": norm(p + "norm1")}
        ff = None
        if isinstance(layer.ff, InputWeightedExpertsConfig):
            f = layer.ff
            ff = PartSpec("routed_experts", {
                "hidden_size": W, "expert_size": f.ff, "num_experts": f.experts, "num_identity": 0, "top": f.top,
                "correction": False, "scoring": "sigmoid", "weight_on": "input", "shared_size": f.shared_ff,
                "shared_gate": f.shared_ff is not None}, p + "mlp.")
        elif layer.ff is not None:
            ff = PartSpec("gated", {"hidden_size": W, "intermediate_size": layer.ff, "activation": "silu",
                                    "names": _FF_NAMES}, p + "mlp.")
        if ff is not None:
            norms["feed_forward"] = norm(p + "norm2")
        layers.append(LayerSpec(PartSpec("parallel", {"residual_scale": cfg.residual_mult}, p), mixer, ff, norms))
    return ModelSpec(
        vocab_size=cfg.vocab_size, hidden_size=W, embedding="embed", layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=norm("final.norm"), head="head",
        embedding_scale=cfg.embedding_scale,
        stream_mix=PartSpec("depth_average", {"names": tuple(f"l{i}.dwa" for i in range(len(layers)))}),
        # a layer without feed-forward has nothing that would read a second norm
        ignorable=tuple(f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if layer.ff is None))


register_architecture(ZusolixConfig.architecture, ZusolixConfig, zusolix_spec)
