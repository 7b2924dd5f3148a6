"""Zusolix without a GPU: its configuration, the model as data (parallel layers with two norms, the stream mix over
all layers' results), what its layers ask of the cache manager, and properties of the plain implementation."""

import copy
import math

import pytest
import torch

from acorninfer_b200.config.model_config import ConfigError, ZusolixConfig
from acorninfer_b200.kernels.ops import GRU_WALK_TOKENS, gru_walks
from acorninfer_b200.models.decoder import Decoder, expected_tensors
from acorninfer_b200.parts.base import TensorSpec
from acorninfer_b200.registry import config_from_dict, spec_for
from acorninfer_b200.weights.loader import check_names_and_shapes
from acorninfer_b200.weights.random_init import random_tensor
from acorninfer_b200.weights.safetensors_io import WeightsError
from tests.plain import zusolix as plain
from tests.tiny import random_tokens
from tests.zusolix_tiny import ZUS_A, ZUS_B, ZUSES, make_model_dir, random_config, read_weights


@pytest.mark.parametrize("name", list(ZUSES))
def test_config_round_trip_and_registry(name):
    cfg = ZUSES[name]["cfg"]
    raw = cfg.to_dict()
    assert raw["architecture"] == "Zusolix" and len(raw["layers"]) == len(cfg.layers)
    again = config_from_dict(raw)
    assert isinstance(again, ZusolixConfig) and again == cfg
    for seed in range(6):
        drawn = random_config(seed)
        assert config_from_dict(drawn.to_dict()) == drawn


def test_config_errors_name_the_key():
    raw = ZUS_A["cfg"].to_dict()
    for path, value, word in ((("layers", 0, "type"), "mamba", "type"), (("layers", 0, "mixer", "q_temp", "every"), 0, "every"),
                              (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"), (("layers", 0, "mixer", "softcap"), 0.0, "softcap"),
                              (("layers", 1, "mixer", "width"), 0, "width"), (("layers", 0, "mlp", "kind"), "sparse", "kind"),
                              (("layers", 1, "mlp", "router", "top"), 9, "top"), (("layers", 0, "mlp", "ff"), 0, "ff"),
                              (("norm", "groups"), 5, "groups"), (("norm", "eps"), 0.0, "eps")):
        bad = copy.deepcopy(raw)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            config_from_dict(bad)
    for path in (("layers", 0, "mixer", "scale"), ("layers", 1, "mixer", "width"), ("layers", 1, "mlp", "router"), ("width",)):
        bad = copy.deepcopy(raw)
        node = bad
        for k in path[:-1]:
            node = node[k]
        del node[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            config_from_dict(bad)
    # what a configuration leaves out does not exist: no temperature, no cap, no shared expert, no feed-forward, factors of 1
    lean = copy.deepcopy(raw)
    del lean["layers"][0]["mixer"]["q_temp"], lean["layers"][0]["mixer"]["softcap"], lean["layers"][1]["mlp"]["shared"]
    del lean["layers"][0]["mlp"], lean["residual_mult"], lean["embedding"], lean["norm"]["groups"]
    cfg = config_from_dict(lean)
    m = cfg.layers[0].mixer
    assert m.softcap is None and m.temp_every is None and cfg.layers[0].ff is None and cfg.layers[1].ff.shared_ff is None
    assert cfg.residual_mult == 1.0 and cfg.embedding_scale == 1.0 and cfg.norm_groups == 1
    names = expected_tensors(spec_for(cfg))
    assert "l0.norm2" not in names and "l1.mlp.shared.sg" not in names and "l1.mlp.router" in names


def test_model_as_data_and_cache_needs():
    cfg = ZUS_A["cfg"]
    spec = spec_for(cfg)
    assert [ls.mixer.kind for ls in spec.layers] == ["attention", "min_gru", "attention", "min_gru"]
    assert all(ls.block.kind == "parallel" and ls.block.params["residual_scale"] == 0.7 for ls in spec.layers)
    assert [ls.feed_forward.kind if ls.feed_forward else None for ls in spec.layers] == ["gated", "routed_experts", None, "routed_experts"]
    assert set(spec.layers[2].norms) == {"mixer"} and set(spec.layers[1].norms) == {"mixer", "feed_forward"}
    assert spec.stream_mix.kind == "depth_average" and spec.embedding_scale == 3.0 and spec.head == "head" and not spec.positions
    names = expected_tensors(spec)
    for n in ("embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.q.b", "l0.mix.v.b", "l0.mlp.gate", "l1.mix.z.b",
              "l1.mix.g", "l1.mlp.router", "l1.mlp.e4.down", "l1.mlp.shared.sg", "l3.dwa"):
        assert n in names, n
    for n in ("l2.norm2", "l1.mix.g.b", "l1.mlp.correction", "l1.mlp.e5.gate", "l3.mlp.shared.up", "l3.mlp.shared.sg", "l4.dwa"):
        assert n not in names, n
    assert [names[f"l{i}.dwa"].shape for i in range(4)] == [(2,), (3,), (4,), (5,)]
    assert names["l0.mix.v"].shape == (2 * 10, 72) and names["l0.mix.o"].shape == (72, 4 * 10)
    assert names["l1.mix.z"].shape == (30, 72) and names["l1.mix.o"].shape == (72, 30) and names["l1.mlp.shared.sg"].shape == (1, 72)
    dec = Decoder(spec, torch.float32, "cpu", page_size=8)
    kv, state = dec.cache_needs()
    assert sorted(kv) == [0, 2] and kv[0].head_dim == 6 and kv[0].value_dim == 10 and kv[0].window is None and kv[2].value_dim is None
    assert {i: s.shape for i, s in state.items()} == {1: (30,), 3: (101,)}
    assert dec.graph_safe
    # a second norm beside an absent feed-forward is not read: a folder may hold it; other strangers are errors
    shapes = {n: s.shape for n, s in names.items()}
    check_names_and_shapes(names, dict(shapes, **{"l2.norm2": (72,)}), dec.ignorable_tensors())
    with pytest.raises(WeightsError, match="l4.norm1"):
        check_names_and_shapes(names, dict(shapes, **{"l4.norm1": (72,)}), dec.ignorable_tensors())


def test_a_stream_mix_does_not_go_with_passes_that_take_the_tokens_in_again():
    from dataclasses import replace
    from acorninfer_b200.parts.base import ScheduleEntry
    spec = spec_for(ZUS_B["cfg"])
    bad = replace(spec, schedule=(ScheduleEntry(0), ScheduleEntry(1, add_embedding=True), ScheduleEntry(2)))
    with pytest.raises(ValueError, match="stream mix"):
        Decoder(bad, torch.float32, "cpu")


def test_coefficients_drawn_at_random_lean_on_the_newest_result():
    spec = TensorSpec((6,), "depth_average")
    t = random_tensor("l4.dwa", spec, 3, 0.02, 0.0, torch.float32)
    assert t.shape == (6,) and 0.6 < float(t[-1]) < 1.2 and float(t[:-1].abs().max()) < 0.5
    for a, b in ((0, 2), (2, 6), (5, 6)):          # any row range of a tensor can be drawn alone
        assert torch.equal(random_tensor("l4.dwa", spec, 3, 0.02, 0.0, torch.float32, rows=(a, b)), t[a:b])


def test_rows_of_the_recurrence_that_are_walked():
    assert gru_walks(1, 64) and gru_walks(GRU_WALK_TOKENS, 3) and not gru_walks(GRU_WALK_TOKENS + 1, 1) and not gru_walks(8192, 16)
    assert gru_walks(8192, 2000)                               # more chunks than a grid holds


def test_plain_implementation_properties(tmp_path):
    tiny = ZUS_A
    d = make_model_dir(tmp_path, tiny)
    w = read_weights(d)
    cfg = tiny["cfg"].to_dict()
    toks = random_tokens(40, tiny["cfg"].vocab_size, 5)
    layers: list = []
    full = plain.forward(cfg, w, toks, every_layer=layers)
    assert len(layers) == 4 and layers[0].shape == (40, 72)
    # causal: a prefix gives the same logits
    assert (plain.forward(cfg, w, toks[:17]) - full[:17]).abs().max() < 1e-9
    # a norm in groups: every part has unit root mean square, whatever the others hold
    x = torch.randn(3, 12, dtype=torch.float64)
    x[:, 4:8] *= 100.0
    y = plain.grouped_norm(x, torch.ones(12, dtype=torch.float64), 1e-12, 3)
    assert (y.reshape(3, 3, 4).pow(2).mean(-1) - 1).abs().max() < 1e-9
    # the temperature steps where a whole span of positions lies behind
    f = plain.query_temperature(range(12), {"coef": 0.5, "every": 4})
    assert f[:3].tolist() == [1.0, 1.0, 1.0] and f[3].item() == pytest.approx(1 + 0.5 * math.log(2)) and f[6] == f[3] < f[7]
    # a closed gate keeps the state, an open one takes the candidate
    c = torch.tensor([[5.0], [7.0]], dtype=torch.float64)
    s = plain.gated_recurrence(torch.tensor([[1.0], [0.0]], dtype=torch.float64), c)
    assert s.tolist() == [[5.0], [5.0]]
    assert plain.candidate(torch.tensor([0.0, -1e-9, 2.0], dtype=torch.float64)).tolist() == pytest.approx([0.5, 0.5, 2.5])
    # every coefficient counts: without the token rows' share the logits differ
    other = dict(w, **{"l3.dwa": w["l3.dwa"].clone()})
    other["l3.dwa"][0] += 1.0
    assert (plain.forward(cfg, other, toks) - full).abs().max() > 0.05
