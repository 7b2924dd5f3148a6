"""Badepel without a GPU: its configuration, the model as data (several residual streams, attention beside linear attention,
padded heads), what its layers ask of the cache manager, and properties of the plain implementation."""

import copy
import math

import pytest
import torch

from acorninfer_b200.config.model_config import BadepelConfig, ConfigError
from acorninfer_b200.models.decoder import Decoder, expected_tensors
from acorninfer_b200.parts.base import TensorSpec
from acorninfer_b200.parts.recurrent_heads import stack_rows
from acorninfer_b200.registry import config_from_dict, spec_for
from acorninfer_b200.weights.loader import check_names_and_shapes
from acorninfer_b200.weights.random_init import random_tensor
from acorninfer_b200.weights.safetensors_io import WeightsError
from tests.badepel_tiny import BAD_A, BAD_B, BAD_C, BADEPELS, make_model_dir, random_config, read_weights
from tests.plain import badepel as plain
from tests.tiny import random_tokens

F64 = torch.float64


@pytest.mark.parametrize("name", list(BADEPELS))
def test_config_round_trip_and_registry(name):
    cfg = BADEPELS[name]["cfg"]
    raw = cfg.to_dict()
    assert raw["architecture"] == "Badepel" and len(raw["layers"]) == len(cfg.layers)
    again = config_from_dict(raw)
    assert isinstance(again, BadepelConfig) and again == cfg
    for seed in range(8):
        drawn = random_config(seed)
        assert config_from_dict(drawn.to_dict()) == drawn


def test_config_errors_name_the_key():
    raw = BAD_A["cfg"].to_dict()
    for path, value, word in ((("layers", 0, "type"), "mamba", "type"), (("layers", 0, "mixer", "left", "mask", "size"), 0, "mask.size"),
                              (("layers", 0, "mixer", "left", "kv_heads"), 3, "kv_heads"), (("layers", 0, "mixer", "left", "softcap"), 0.0, "softcap"),
                              (("layers", 0, "mixer", "left", "rot", "dims"), 8, "rot.dims"), (("layers", 0, "mixer", "left", "conv"), 0, "conv"),
                              (("layers", 0, "mixer", "right", "tau"), 0.0, "tau"), (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
                              (("layers", 0, "mlp", "kind"), "sparse", "kind"), (("layers", 1, "mlp", "router", "top"), 9, "top"),
                              (("layers", 1, "mlp", "shared", "limit"), 0.0, "limit"), (("layers", 0, "mlp", "ff"), 0, "ff"),
                              (("streams",), 0, "streams"), (("streams",), 99, "streams"), (("norm", "eps"), 0.0, "eps")):
        bad = copy.deepcopy(raw)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            config_from_dict(bad)
    for path in (("layers", 0, "mixer", "left", "scale"), ("layers", 0, "mixer", "left_scale"), ("layers", 0, "mixer", "right", "tau"),
                 ("layers", 1, "mixer", "vdim"), ("layers", 1, "mlp", "expert", "limit"), ("width",)):
        bad = copy.deepcopy(raw)
        node = bad
        for k in path[:-1]:
            node = node[k]
        del node[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            config_from_dict(bad)
    # what a configuration leaves out does not exist: no window, cap, rotation, convolution, shared expert, feed-forward, streams
    lean = copy.deepcopy(raw)
    left = lean["layers"][0]["mixer"]["left"]
    del left["mask"], left["softcap"], left["rot"], left["conv"], lean["layers"][1]["mlp"]["shared"], lean["layers"][0]["mlp"]
    del lean["streams"], lean["residual_mult"]
    cfg = config_from_dict(lean)
    m = cfg.layers[0].mixer.left
    assert m.softcap is None and m.window is None and m.conv is None and m.rot_dims == 0
    assert cfg.layers[0].ff is None and cfg.layers[1].ff.shared_ff is None and cfg.streams is None and cfg.residual_mult == 1.0
    names = expected_tensors(spec_for(cfg))
    for n in ("l0.norm2", "l0.hc1.in", "l0.mix.left.q.conv", "l1.mlp.shared.up"):
        assert n not in names, n


def test_model_as_data_and_cache_needs():
    cfg = BAD_A["cfg"]
    spec = spec_for(cfg)
    assert [ls.mixer.kind for ls in spec.layers] == ["side_by_side", "head_delta", "side_by_side", "head_delta"]
    assert all(ls.block.kind == "hyper" and ls.block.params["residual_scale"] == 0.7 and ls.block.params["streams"] == 2 for ls in spec.layers)
    assert [ls.feed_forward.kind if ls.feed_forward else None for ls in spec.layers] == ["gated", "routed_experts", None, "routed_experts"]
    assert set(spec.layers[2].norms) == {"mixer"} and spec.streams == 2 and spec.head == "head" and len(spec.positions) == 1
    names = expected_tensors(spec)
    for n in ("embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.hc2.mix", "l0.mix.left.q.b", "l0.mix.left.v.conv", "l0.mix.right.a2.b",
              "l1.mix.A_log", "l1.mix.k.conv", "l1.mlp.router.b", "l1.mlp.e4.down", "l1.mlp.shared.gate", "l2.hc1.out"):
        assert n in names, n
    for n in ("l2.norm2", "l2.hc2.in", "l1.mlp.correction", "l1.mlp.e5.gate", "l3.mlp.shared.up", "l2.mix.left.q.conv", "l1.mix.q.b"):
        assert n not in names, n
    assert names["l0.mix.left.q.norm"].shape == (24,) and names["l0.mix.left.k.norm"].shape == (12,) and names["l0.mix.left.v"].shape == (20, 72)
    assert names["l0.mix.left.o"].shape == (72, 40) and names["l0.hc1.mix"].shape == (2, 2) and names["l1.mix.norm"].shape == (9,)
    dec = Decoder(spec, torch.float32, "cpu", page_size=8)
    kv, state = dec.cache_needs()
    assert sorted(kv) == [0, 2] and kv[0].head_dim == 6 and kv[0].value_dim == 10 and kv[0].window == 9 and kv[2].window is None
    conv = 2 * (24 + 12 + 20)                                    # two projected rows of 56 channels
    assert state[0].shape == (conv + 108,)                       # 3 heads of 5 x 7, up to a multiple of 4
    assert state[2].shape == (2 * 8 * 4,) and state[1].shape == (4 * 6 * 9 + 3 * (2 * 2 * 6 + 4 * 9),) and state[3].shape == (2 * 12 * 4,)
    left, right = dec.blocks[0].mixer.sides[0][1], dec.blocks[0].mixer.sides[1][1]
    assert left.state_base == 0 and right.state_base == conv
    assert dec.graph_safe
    # factors and a norm beside an absent feed-forward are not read: a folder may hold them; other strangers are errors
    shapes = {n: tuple(4 if k is None else k for k in s.shape) for n, s in names.items()}
    check_names_and_shapes(names, dict(shapes, **{"l2.norm2": (72,), "l2.hc2.mix": (2, 2)}), dec.ignorable_tensors())
    with pytest.raises(WeightsError, match="l4.norm1"):
        check_names_and_shapes(names, dict(shapes, **{"l4.norm1": (72,)}), dec.ignorable_tensors())


def test_streams_want_an_arrangement_that_takes_them():
    from dataclasses import replace
    from acorninfer_b200.parts.base import ScheduleEntry
    spec = spec_for(BAD_B["cfg"])
    with pytest.raises(ValueError, match="streams"):
        Decoder(replace(spec, streams=None), torch.float32, "cpu")
    with pytest.raises(ValueError, match="streams"):
        Decoder(replace(spec, schedule=(ScheduleEntry(0), ScheduleEntry(1, add_embedding=True), ScheduleEntry(2))), torch.float32, "cpu")


def test_heads_are_padded_for_the_tensor_core_kernels_only(tmp_path):
    """Under bfloat16 heads of 40 keys and 56 values become heads of 64 in the kernels' eyes: the checkpoint's shapes stay,
    zeros stand in the padded rows of q, k, v and the padded columns of o, and the norms count the real entries."""
    d = make_model_dir(tmp_path, BAD_C)
    w = read_weights(d)
    for dtype, width in ((torch.bfloat16, 64), (torch.float32, None)):
        dec = Decoder(spec_for(BAD_C["cfg"]), dtype, "cpu", page_size=16)
        dec.bind({n: t.to(dtype) for n, t in w.items()})
        side = dec.blocks[2].mixer
        a = side.sides[0][1]
        assert a.tensor_specs()["q"].shape == (6 * 40, 256) and a.tensor_specs()["q.norm"].shape == (240,)
        if width is None:
            assert (a.d, a.dv) == (40, 56)
            continue
        assert (a.d, a.dv) == (64, 64) and a.cache_needs().kv.head_dim == 64 and a.cache_needs().kv.value_dim is None
        q = a.w_qkv[:6 * 64].view(6, 64, 256)
        assert torch.equal(q[:, :40].reshape(240, 256), w["l2.mix.left.q"]) and not q[:, 40:].any()
        v = a.w_qkv[8 * 64:10 * 64].view(2, 64, 256)
        assert torch.equal(v[:, :56].reshape(112, 256), w["l2.mix.left.v"]) and not v[:, 56:].any()
        o = side.w_o[:, :6 * 64].view(256, 6, 64)
        assert torch.equal(o[..., :56].reshape(256, 336), w["l2.mix.left.o"]) and not o[..., 56:].any()
        assert not a.bias32[:6 * 64].view(6, 64)[:, 40:].any() and not a.q_norm32.view(6, 64)[:, 40:].any()
        assert side.w_in.shape[0] % 8 == 0 and side.first_in % 8 == 0


def test_projections_side_by_side_in_one_matrix():
    g = torch.Generator().manual_seed(0)
    a, b = torch.randn(3, 5, generator=g), torch.randn(4, 5, generator=g)
    w = stack_rows([a, b], (0, 8), torch.float32)
    assert w.shape == (16, 5) and torch.equal(w[:3], a) and torch.equal(w[8:12], b) and not w[3:8].any() and not w[12:].any()


def test_stream_matrices_drawn_at_random_lean_on_the_identity():
    spec = TensorSpec((4, 4), "stream_mix")
    t = random_tensor("l1.hc1.mix", spec, 3, 0.02, 0.0, torch.float32)
    assert float((t - 0.8 * torch.eye(4)).abs().max()) < 0.8 and float(t.diagonal().min()) > 0.2
    for a, b in ((0, 1), (1, 4), (3, 4)):          # any row range of a tensor can be drawn alone
        assert torch.equal(random_tensor("l1.hc1.mix", spec, 3, 0.02, 0.0, torch.float32, rows=(a, b)), t[a:b])


def test_plain_implementation_properties(tmp_path):
    d = make_model_dir(tmp_path, BAD_A)
    w = read_weights(d)
    cfg = BAD_A["cfg"].to_dict()
    toks = random_tokens(40, BAD_A["cfg"].vocab_size, 5)
    layers: list = []
    full = plain.forward(cfg, w, toks, every_layer=layers)
    assert len(layers) == 4 and layers[0].shape == (40, 72)
    # causal: a prefix gives the same logits
    assert (plain.forward(cfg, w, toks[:17]) - full[:17]).abs().max() < 1e-9
    g = torch.Generator().manual_seed(2)
    R = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    # the sink: shares sum to less than one, and a single key of score 0 gets half
    ok = plain.visible(3, None)
    p = plain.softmax_plus_one(R(3, 3), ok)
    assert float(p.sum(-1).max()) < 1.0 and plain.softmax_plus_one(torch.zeros(1, 1, dtype=F64), ok[:1, :1]).item() == pytest.approx(0.5)
    assert plain.softmax_plus_one(torch.full((1, 1), -800.0, dtype=F64), ok[:1, :1]).item() == 0.0
    assert plain.visible(5, 2).sum(-1).tolist() == [1, 2, 2, 2, 2]
    # the rotation turns neighbours: lengths of pairs stay, position 0 is untouched, scores hang on the distance alone
    x = R(1, 1, 8).expand(6, 1, 8)
    y = plain.rotate_neighbours(x, {"base": 50.0, "dims": 4})
    assert torch.allclose(y[0], x[0]) and torch.allclose(y[..., 4:], x[..., 4:])
    assert torch.allclose(y[..., 0] ** 2 + y[..., 1] ** 2, x[..., 0] ** 2 + x[..., 1] ** 2)
    assert (y[1, 0] @ y[3, 0]).item() == pytest.approx((y[2, 0] @ y[4, 0]).item())
    # a convolution with the newest tap alone is a scaling; the oldest tap alone is a delay
    u, taps = R(5, 2), torch.tensor([[0.0, 0.0, 2.0], [3.0, 0.0, 0.0]], dtype=F64)
    y = plain.short_conv(u, taps)
    assert torch.allclose(y[:, 0], 2 * u[:, 0]) and torch.allclose(y[2:, 1], 3 * u[:3, 1]) and not y[:2, 1].any()
    # linear attention without decay is a sum over the past; the delta rule with strength one stores what it last saw
    q, k, v = R(6, 1, 4), R(6, 1, 4), R(6, 1, 3)
    o, _ = plain.gla_recurrence(q, k, v, torch.ones(6, 1, 4, dtype=F64))
    want = torch.tril(q[:, 0] @ k[:, 0].T) @ v[:, 0]
    assert torch.allclose(o[:, 0], want)
    kk = plain.unit(k)
    o, _ = plain.delta_recurrence(kk, kk, v, torch.ones(6, 1, dtype=F64), torch.full((6, 1), 0.5, dtype=F64))
    assert (o - v).abs().max() < 1e-4
    # equal streams under equal factors stay equal; the matrix is [from, to]
    xs = [R(2, 3), R(2, 3)]
    new = plain.write_streams(xs, torch.tensor([[0.0, 1.0], [0.0, 0.0]], dtype=F64), torch.tensor([0.0, 2.0], dtype=F64), torch.ones(2, 3, dtype=F64))
    assert not new[0].any() and torch.allclose(new[1], xs[0] + 2.0)
    # one stream with the factors of a plain sum is a plain residual stream
    one = {**w, **{n: torch.ones_like(w[n][:1]) for n in w if ".hc" in n and ".mix" not in n},
           **{n: torch.ones_like(w[n][:1, :1]) for n in w if ".hc" in n and n.endswith(".mix")}}
    a = plain.forward({**cfg, "streams": 1}, one, toks)
    b = plain.forward({k: v for k, v in cfg.items() if k != "streams"}, w, toks)
    assert (a - b).abs().max() < 1e-9 and math.isfinite(float(a.sum()))
