"""Badepel on the GPU against the plain implementation (``tests/plain/badepel.py``, float64).

Whole models of several small configurations, replayed whole, with a decoded tail, in portions down to two tokens,
and mixed with other requests in a pool so small that pages and slots are used again; every mechanism alone (a small
model, or its kernel with inputs made so that a fault would show); long decoding; greedy generation through the public
entry point and the scheduler.

Errors are relative: the root mean square over the vocabulary of the difference of the logits (mean taken off) over
the standard deviation of the plain model's logits.  Under bfloat16 a token whose router logits put the last chosen
expert less than ``CLOSE`` above the first one left out may go to another expert than in float64 (the whole position
then differs); such positions, which the plain implementation names, are left out.
"""

import math

import numpy as np
import pytest
import torch

from acorninfer_b200.config.model_config import BadepelConfig
from tests import traces
from tests.badepel_tiny import BAD_LONG, BADEPELS, L, att, both, delta, gla, make_model_dir, moe, random_config, read_weights
from tests.paged import rows_layout, scatter_to_pages
from tests.plain import badepel as plain
from tests.tiny import random_tokens

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {"float32": 4e-5, "bfloat16": 0.1}
CLOSE = 0.1
LENGTHS = [45, 38, 61, 50, 33, 29]


def rel_err(got, ref):
    d = np.asarray(got, np.float64) - np.asarray(ref, np.float64)
    d = d - d.mean()
    return math.sqrt((d ** 2).mean()) / float(np.std(ref))


class Ref(dict):
    """request -> float64 logits [T, vocab]; ``close``: the (request, position) pairs whose choice of experts
    hangs on less than ``CLOSE``."""

    close: set = frozenset()


def plain_logits(cfg, w, reqs, close_gap=CLOSE):
    ref = Ref()
    close = set()
    for rid, toks in reqs.items():
        gaps: list = []
        ref[rid] = plain.forward(cfg.to_dict(), w, toks, router_gaps=gaps).numpy()
        close |= {(rid, t) for run in gaps for t, g in enumerate(run) if g < close_gap}
    ref.close = close
    return ref


@pytest.fixture(scope="module", params=list(BADEPELS))
def case(request, tmp_path_factory):
    tiny = BADEPELS[request.param]
    d = make_model_dir(tmp_path_factory.mktemp(request.param), tiny)
    reqs = {f"r{i}": random_tokens(n, tiny["cfg"].vocab_size, 5100 + i) for i, n in enumerate(LENGTHS)}
    return tiny, d, reqs, plain_logits(tiny["cfg"], read_weights(d), reqs)


def run_cut(tiny, model_dir, steps, dtype, max_requests=4, watch=None):
    from acorninfer_b200.engine.runner import ModelRunner
    from acorninfer_b200.replay import TraceSession

    pool = traces.max_live_tokens(steps)
    runner = ModelRunner.from_model_dir(model_dir, dtype=dtype, num_blocks=-(-pool // tiny["page_size"]),
                                        page_size=tiny["page_size"], max_requests=max_requests, max_step_tokens=4096)
    session = TraceSession(runner)

    def step(msg):
        if watch is None:
            return session.step(msg)
        out = session.step(dict(msg, end=[]))
        watch(session, msg)
        session.step({"entries": [], "end": msg["end"]})
        return out

    got = traces.collect(step, steps)
    runner.manager.assert_balanced()
    return got, runner


def check(got, ref, dtype, what, tol=None):
    """Every position within the tolerance; in bfloat16 a single position may come to twice the tolerance as long
    as the mean over all positions stays below a third of it: a fault moves many positions, rounding few."""
    errs = {key: rel_err(row, ref[key[0]][key[1]]) for key, row in got.items()}
    tol = tol or TOL[dtype]
    close = getattr(ref, "close", set()) if dtype == "bfloat16" else set()
    mean = float(np.mean([e for k, e in errs.items() if k not in close]))
    assert len(close & set(errs)) <= 0.5 * len(errs), f"{what}: too many close calls for the test to mean much"
    worst = max((k for k in errs if k not in close), key=errs.get)
    if dtype == "bfloat16":
        assert errs[worst] < 2 * tol and mean < tol / 3, f"{what}: {worst}: {errs[worst]:.3e}, mean {mean:.3e}"
    else:
        assert errs[worst] < tol, f"{what}: {worst}: {errs[worst]:.3e}, mean {mean:.3e}"


CUTS = {
    "whole": traces.whole,
    "decode_tail": lambda r: traces.decode_tail(r, tail=24),
    "portions": lambda r: traces.portions(r, sizes=(7, 2, 5, 3, 16, 2, 11, 4)),
    "mixed": lambda r: traces.mixed(r, max_live=4, seed=3, stagger=2),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cut", list(CUTS))
def test_cut_matches_plain(case, cut, dtype):
    tiny, d, reqs, ref = case
    got, runner = run_cut(tiny, d, CUTS[cut](reqs), dtype)
    assert len(got) == sum(len(t) for t in reqs.values())
    check(got, ref, dtype, cut)
    if cut == "decode_tail":
        assert runner.graph_replays >= len(reqs) * 10        # single-token steps replay captured graphs


def test_cuts_agree_with_each_other_float32(case):
    """The logits at a position do not depend on how the tokens were cut into steps, on what else was
    in the batch or on which pages and slots held them, beyond rounding."""
    tiny, d, reqs, _ = case
    base, _ = run_cut(tiny, d, traces.whole(reqs), "float32")
    for cut in ("decode_tail", "portions", "mixed"):
        other, _ = run_cut(tiny, d, CUTS[cut](reqs), "float32")
        for key, row in base.items():
            assert rel_err(other[key], row) < 1e-5, f"{cut}: {key}"


def test_mixed_trace_uses_pages_and_slots_again(case):
    tiny, d, reqs, _ = case
    steps = CUTS["mixed"](reqs)
    pages: dict = {}
    slots: dict = {}

    def watch(session, msg):
        for rid, rc in session.live.items():
            slots.setdefault(rc.slot, set()).add(rid)
            for table in rc.tables:
                for page in table:
                    pages.setdefault(page, set()).add(rid)

    run_cut(tiny, d, steps, "float32", watch=watch)
    assert len(slots) <= 4 and sum(1 for users in slots.values() if len(users) >= 2) >= 1, slots
    assert sum(1 for users in pages.values() if len(users) >= 2) >= 2, pages


def test_branches_of_a_captured_step_change_nothing(case):
    """Decoding four requests at a time from captured graphs, whose layers run attention and linear attention (and the shared
    expert and the routed ones) as branches side by side, against the same steps launched one by one."""
    from acorninfer_b200.engine.batch import StepEntry
    from acorninfer_b200.engine.runner import ModelRunner
    tiny, d, reqs, _ = case
    for dtype, tol in (("float32", 1e-6), ("bfloat16", 1e-3)):
        out = {}
        for graph in (True, False):
            runner = ModelRunner.from_model_dir(d, dtype=dtype, num_blocks=96, page_size=tiny["page_size"], max_requests=4,
                                                max_step_tokens=256, decode_graph=graph)
            rcs = [runner.open(f"g{i}") for i in range(4)]
            toks = [reqs[f"r{i}"][:28] for i in range(4)]
            runner.step([StepEntry(rc, t[:5], [4]) for rc, t in zip(rcs, toks)])
            out[graph] = torch.stack([runner.step([StepEntry(rc, [t[j]], [0]) for rc, t in zip(rcs, toks)]).clone()
                                      for j in range(5, 28)])
            assert (runner.graph_replays > 10) == graph
        assert (out[True] - out[False]).abs().max() < tol * max(1.0, float(out[False].abs().max())), dtype


def test_first_step_of_one_token_and_requests_left_out(case):
    """A request whose first step is a single token (recurrences from the zero state, a softmax of one key and the sink), then
    portions beside another request that decodes and is left out of some steps."""
    tiny, d, reqs, ref = case
    a, b = reqs["r0"], reqs["r1"]
    steps = [{"entries": [{"id": "r0", "tokens": a[:1], "want": [0]}], "end": []},
             {"entries": [{"id": "r0", "tokens": a[1:3], "want": [0, 1]}, {"id": "r1", "tokens": b[:9], "want": list(range(9))}], "end": []},
             {"entries": [{"id": "r1", "tokens": b[9:10], "want": [0]}], "end": []},
             {"entries": [{"id": "r0", "tokens": a[3:20], "want": []}, {"id": "r1", "tokens": b[10:11], "want": []}], "end": []},
             {"entries": [{"id": "r0", "tokens": a[20:], "want": list(range(len(a) - 20))}], "end": ["r0"]},
             {"entries": [{"id": "r1", "tokens": b[11:], "want": list(range(len(b) - 11))}], "end": ["r1"]}]
    for i, s in enumerate(steps):
        s["step"] = i
    for dtype in ("float32", "bfloat16"):
        got, _ = run_cut(tiny, d, steps, dtype)
        check(got, ref, dtype, "first token alone")


def test_long_decoding_float32(case):
    tiny, d, _, _ = case
    toks = random_tokens(190, tiny["cfg"].vocab_size, 79)
    ref = plain_logits(tiny["cfg"], read_weights(d), {"long": toks})
    got, _ = run_cut(tiny, d, traces.decode_tail({"long": toks}, tail=170), "float32")
    check(got, ref, "float32", "long decoding")


def test_long_requests_over_pages_and_segments(tmp_path):
    """Requests of a few hundred tokens over pages of 16: several chunks of keys in the tensor-core kernels, windows
    that pass, several segments and chunks of the recurrences, portions that end at and around their edges."""
    tiny = BAD_LONG
    reqs = {f"L{i}": random_tokens(n, tiny["cfg"].vocab_size, 710 + i) for i, n in enumerate([330, 260, 150])}
    cuts = {"whole": traces.whole, "decode_tail": lambda r: traces.decode_tail(r, tail=60),
            "portions": lambda r: traces.portions(r, sizes=(128, 3, 2, 129, 29, 16, 2, 70)),
            "mixed": lambda r: traces.mixed(r, max_live=3, seed=5, max_portion=80, stagger=1)}
    d = make_model_dir(tmp_path, tiny)
    ref = plain_logits(tiny["cfg"], read_weights(d), reqs)
    for dtype in ("float32", "bfloat16"):
        for cut, build in cuts.items():
            got, runner = run_cut(tiny, d, build(reqs), dtype)
            assert len(got) == sum(len(t) for t in reqs.values())
            check(got, ref, dtype, f"long, {cut}")


@pytest.mark.parametrize("seed", [1, 4, 6, 12, 13])
def test_configurations_drawn_at_random(seed, tmp_path):
    """Models whose sizes are drawn from what real models have, requests of up to 200 tokens, whole, with a decoded
    tail and mixed in a small pool, float32 and bfloat16."""
    import random
    tiny = dict(cfg=random_config(seed), page_size=16, seed=seed)
    d = make_model_dir(tmp_path, tiny, sigma=0.06, sigma_norm=0.1)
    w = read_weights(d)
    rng = random.Random(seed)
    lengths = [rng.randint(140, 200), rng.randint(60, 120), rng.randint(2, 60), 1, rng.randint(60, 100)]
    reqs = {f"q{i}": random_tokens(n, tiny["cfg"].vocab_size, seed * 10 + i) for i, n in enumerate(lengths)}
    ref = plain_logits(tiny["cfg"], w, reqs, close_gap=0.08)          # smaller weights than above: smaller router logits
    for dtype, tol in (("float32", 6e-5), ("bfloat16", 0.15)):
        for cut, steps in (("whole", traces.whole(reqs)), ("decode_tail", traces.decode_tail(reqs, tail=40)),
                           ("mixed", traces.mixed(reqs, max_live=4, seed=seed, max_portion=90, stagger=1))):
            got, _ = run_cut(tiny, d, steps, dtype)
            check(got, ref, dtype, f"seed {seed}, {cut}", tol=tol)


def follows_plain(cfg, w, prompt, ids, slack, excuse_close=False):
    gaps: list = []
    logits = plain.forward(cfg.to_dict(), w, ids[:-1], router_gaps=gaps)
    close = {t for run in gaps for t, g in enumerate(run) if g < CLOSE} if excuse_close else set()
    return all(float(logits[i - 1].max() - logits[i - 1][ids[i]]) <= slack * float(logits.std()) for i in range(len(prompt), len(ids))
               if i - 1 not in close)


@pytest.mark.parametrize("dtype,slack", [("float32", 1e-4), ("bfloat16", 0.3)])
def test_greedy_generation_through_the_engine(case, dtype, slack):
    """``generate``: the scheduler with a token budget (prompts cut into portions beside decoding
    requests), sampling on the device, a step ahead of the host."""
    from acorninfer_b200 import generate
    tiny, d, _, _ = case
    cfg = tiny["cfg"]
    w = read_weights(d)
    prompts = [random_tokens(n, cfg.vocab_size, 910 + n) for n in (1, 14, 23, 6, 31)]
    outs = generate(d, prompts, max_new_tokens=12, temperature=0.0, dtype=dtype, page_size=tiny["page_size"],
                    num_blocks=64, max_running=3, chunked_budget=10, watermark_blocks=0, eos_ids=())
    for p, ids in zip(prompts, outs):
        assert len(ids) == len(p) + 12 and follows_plain(cfg, w, p, ids, slack, dtype == "bfloat16"), (dtype, len(p))


def test_preemption_recomputes_float32(case):
    """So few pages that requests are preempted and recomputed from their first token."""
    from acorninfer_b200.generation import build_engine, generate_with_engine
    tiny, d, _, _ = case
    cfg = tiny["cfg"]
    prompts = [random_tokens(n, cfg.vocab_size, 50 + n) for n in (20, 18, 13)]
    pages = -(-36 // tiny["page_size"]) * 2 + 1
    tight = build_engine(d, dtype="float32", page_size=tiny["page_size"], num_blocks=pages, watermark_blocks=0, max_running=3)
    got = generate_with_engine(tight, prompts, max_new_tokens=16, eos_ids=())
    w = read_weights(d)
    for p, a in zip(prompts, got):
        assert len(a) == len(p) + 16 and follows_plain(cfg, w, p, a, 1e-4)


def test_replay_program_serves_the_design(tmp_path):
    """``bin/trace_run`` as a program on a Badepel folder: it picks the model by ``config.json``, runs a mixed trace in
    a pool sized for the live requests and writes the logits asked for."""
    import json
    import subprocess
    import sys
    from pathlib import Path
    tiny = BADEPELS["bad_b"]
    d = make_model_dir(tmp_path / "model", tiny)
    reqs = {f"t{i}": random_tokens(n, tiny["cfg"].vocab_size, 300 + i) for i, n in enumerate([35, 48, 21, 66, 40])}
    ref = plain_logits(tiny["cfg"], read_weights(d), reqs)
    steps = traces.mixed(reqs, seed=4)
    out = tmp_path / "out"
    root = Path(__file__).resolve().parent.parent
    proc = subprocess.run(
        [sys.executable, str(root / "bin" / "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out),
         "--max-tokens", str(traces.max_live_tokens(steps))],
        input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    V = tiny["cfg"].vocab_size

    def read_step(msg):
        f = out / f"{msg['step']}.f32"
        return np.fromfile(f, dtype="<f4").reshape(-1, V) if f.exists() else None

    check(traces.collect(read_step, steps), ref, "float32", "trace_run")


# ------------------------------------------------------------------ one mechanism at a time


def _solo(mixer, ff=None, width=48, vocab=90, streams=2, mult=1.0, more=()):
    return BadepelConfig(vocab_size=vocab, hidden_size=width, norm_eps=1e-5, streams=streams, residual_mult=mult,
                         layers=(L(mixer, ff),) + tuple(more))


_TINY = gla(1, 4, 4, rank=2)
_SMALL = both(att(heads=1, kv_heads=1, dim=4, scale=0.5), _TINY)
_DELTA = delta(heads=1, kv_heads=1, dim=8, vdim=8, conv=2)
SOLOS = {
    "attention, nothing but keys": _solo(both(att(heads=3, kv_heads=3, dim=10, scale=0.6), _TINY, 1.0, 0.3)),
    "attention, values wider than keys": _solo(both(att(heads=4, kv_heads=2, dim=6, vdim=22, scale=0.5, rot=6), _TINY)),
    "attention, values narrower, one head": _solo(both(att(heads=1, kv_heads=1, dim=16, vdim=3, scale=0.5, conv=2), _TINY)),
    "attention, a cap that bites": _solo(both(att(heads=2, kv_heads=1, dim=8, scale=2.0, cap=0.5, rot=2), _TINY)),
    "attention, 9 query heads a key head, a window": _solo(both(att(heads=9, kv_heads=1, dim=16, scale=0.4, window=4), _TINY)),
    "attention, 6 taps, the token itself only": _solo(both(att(heads=2, kv_heads=2, dim=32, scale=0.3, conv=6, window=1, rot=14), _TINY)),
    "attention, heads of 130": _solo(both(att(heads=2, kv_heads=1, dim=130, scale=0.1, conv=3, rot=130), _TINY)),
    "linear attention, wide heads": _solo(both(att(heads=1, kv_heads=1, dim=4, scale=0.5), gla(2, 132, 8, tau=2.0), 0.2, 1.0)),
    "linear attention, heads of 3 and 5": _solo(both(att(heads=1, kv_heads=1, dim=4, scale=0.5), gla(5, 3, 5, rank=1), 0.2, 1.0)),
    "linear attention, wide values": _solo(both(att(heads=1, kv_heads=1, dim=4, scale=0.5), gla(1, 16, 200, tau=1.0), 0.2, 1.0)),
    "delta rule, no convolution": _solo(delta(heads=2, kv_heads=2, dim=8, vdim=8)),
    "delta rule, three heads a key head": _solo(delta(heads=6, kv_heads=2, dim=10, vdim=6, conv=3)),
    "delta rule, heads of 136 and 130": _solo(delta(heads=2, kv_heads=1, dim=136, vdim=130, conv=4)),
    "delta rule, wide values, 7 taps": _solo(delta(heads=1, kv_heads=1, dim=64, vdim=200, conv=7)),
    "delta rule twice": _solo(_DELTA, more=(L(delta(heads=3, kv_heads=3, dim=4, vdim=12, conv=4), ff=20),)),
    "gated feed-forward, widths no multiple of 8": _solo(_DELTA, ff=37, width=44),
    "experts: one choice of seven, no shared expert": _solo(_DELTA, ff=moe(11, 7, 1, 1.0)),
    "experts: all three chosen, a wide shared expert": _solo(_DELTA, ff=moe(8, 3, 3, 0.5, 40, 2.0)),
    "experts: two of thirteen": _solo(_SMALL, ff=moe(24, 13, 2, 7.0, 8, 0.3), width=40),
    "one plain stream": _solo(_DELTA, ff=16, streams=None, mult=0.4),
    "one stream with factors": _solo(_SMALL, ff=16, streams=1, mult=1.3),
    "eight streams, a width of 50": _solo(_DELTA, ff=16, width=50, streams=8, mult=0.5),
    "four streams, five layers without feed-forward": _solo(_SMALL, more=(L(_DELTA), L(_SMALL), L(_DELTA), L(_SMALL)), mult=0.8, streams=4),
}


@pytest.mark.parametrize("name", list(SOLOS))
def test_mechanism_alone(name, tmp_path):
    tiny = dict(cfg=SOLOS[name], page_size=4, seed=7)
    d = make_model_dir(tmp_path, tiny, sigma=0.3)
    w = read_weights(d)
    reqs = {f"s{i}": random_tokens(n, tiny["cfg"].vocab_size, 70 + i) for i, n in enumerate([26, 17, 9])}
    ref = plain_logits(tiny["cfg"], w, reqs)
    for cut in ("whole", "portions", "mixed", "decode_tail"):
        steps = {"portions": traces.portions(reqs, sizes=(3, 2, 6, 2)), "decode_tail": traces.decode_tail(reqs, tail=8)}.get(cut) \
            or CUTS[cut](reqs)
        got, _ = run_cut(tiny, d, steps, "float32")
        check(got, ref, "float32", f"{name}, {cut}")
    got, _ = run_cut(tiny, d, CUTS["mixed"](reqs), "bfloat16")
    check(got, ref, "bfloat16", f"{name}, mixed, bfloat16", tol=0.2)


def test_no_mechanism_is_optional(tmp_path):
    """Each constant and each small tensor of a model changes the plain model's logits by far more than the tolerance:
    a run that agrees with the plain model has not left it out."""
    import copy
    tiny = BADEPELS["bad_a"]
    d = make_model_dir(tmp_path, tiny)
    w = read_weights(d)
    cfg = tiny["cfg"].to_dict()
    toks = random_tokens(30, tiny["cfg"].vocab_size, 3)
    full = plain.forward(cfg, w, toks).numpy()

    def differs(c, ww):
        return max(rel_err(a, b) for a, b in zip(plain.forward(c, ww, toks).numpy(), full)) > 30 * TOL["float32"]

    left = ("layers", 0, "mixer", "left")
    for path, value in (((*left, "mask", "size"), 10), ((*left, "mask", "size"), 8), ((*left, "softcap"), None), ((*left, "scale"), 0.45),
                        ((*left, "rot", "dims"), 2), ((*left, "rot", "base"), 120.0), (("layers", 0, "mixer", "left_scale"), 1.0),
                        (("layers", 0, "mixer", "right_scale"), 1.0), (("layers", 0, "mixer", "right", "tau"), 5.0),
                        (("layers", 1, "mlp", "router", "top"), 1), (("layers", 1, "mlp", "shared"), None),
                        (("layers", 1, "mlp", "shared", "limit"), 1.2), (("layers", 1, "mlp", "expert", "limit"), 0.9),
                        (("residual_mult",), 1.0)):
        other = copy.deepcopy(cfg)
        node = other
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        assert differs(other, w), path
    for name in [n for n in w if n.endswith((".b", "dt_bias", "A_log", ".in", ".out", ".mix")) and n != "embed"] + ["l0.mix.right.a1"]:
        assert differs(cfg, dict(w, **{name: torch.zeros_like(w[name])})), name
    for name in [n for n in w if n.endswith(".norm") or ".norm" in n]:
        assert differs(cfg, dict(w, **{name: torch.ones_like(w[name])})), name
    for name in [n for n in w if n.endswith(".conv")]:
        for j in range(w[name].shape[1]):
            one = w[name].clone()
            one[:, j] += 0.5
            assert differs(cfg, dict(w, **{name: one})), (name, j)
    for name in [n for n in w if n.endswith("hc1.mix")]:
        assert differs(cfg, dict(w, **{name: w[name].t().contiguous()})), name           # [from, to], not the other way round


def ops():
    from acorninfer_b200.kernels import ops as o
    return o


def _rand(g, *shape, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("width,n", [(12, 1), (72, 2), (50, 3), (256, 3), (1028, 4), (2048, 4), (4096, 2), (4608, 4), (96, 5), (130, 8)])
def test_hyper_norm(width, n, dtype, tol):
    """Streams that lie apart and streams that are all the same rows; no pending result, a plain one, experts with and without
    weights and a shared one; in place and into memory of its own, all rows or some of them (one twice); the plain sum."""
    o = ops()
    g = torch.Generator().manual_seed(width + n)
    eps = 1e-5
    d64 = lambda t: t.double()
    dev = lambda t: None if t is None else t.to(DEV)
    for T in (7, 200):
        top = 2
        w, mix, put, take = _rand(g, width), _rand(g, n, n), _rand(g, n), _rand(g, n)
        a, extra = _rand(g, T, width, dtype=dtype), _rand(g, T, width, dtype=dtype)
        y = _rand(g, T * top, width, dtype=dtype)
        slot_of = torch.randperm(T * top, generator=g).view(T, top).to(torch.int32)
        wts = torch.rand(T, top, generator=g)
        picked = d64(y)[slot_of.long()]
        experts = lambda ex, ws: o.ExpertsPending(dev(y), dev(slot_of), dev(ex), None, dev(ws))
        pend = [(None, None), (dev(a), d64(a)), (experts(None, wts), (picked * d64(wts)[..., None]).sum(1)),
                (experts(extra, wts), (picked * d64(wts)[..., None]).sum(1) + d64(extra)), (experts(extra, None), picked.sum(1) + d64(extra))]
        rows = torch.tensor([3, 0, 3, 6], dtype=torch.int32)
        for k, (result, add) in enumerate(pend):
            for same in (False, True):
                x = _rand(g, 1 if same else n, T, width)
                xs = [d64(x[0 if same else s]) for s in range(n)]
                new = xs if result is None else plain.write_streams(xs, d64(mix), 0.7 * d64(put), add)
                pending = None if result is None else (result, dev(mix), dev(put), 0.7)
                for tk in (take, None):
                    u = plain.read_streams(new, d64(tk) if tk is not None else torch.ones(n, dtype=torch.float64))
                    want = plain.rms_norm(u, d64(w), eps)
                    bound = tol * max(1.0, float(want.abs().max()))
                    bundle = o.StreamBundle(dev(x), n, pending)
                    got = bundle.read(dev(tk), dev(w), eps, dtype, rows=dev(rows))
                    assert (got.double().cpu() - want[rows.long()]).abs().max() < bound, (k, same)
                    assert torch.equal(bundle.x32.cpu(), x) and bundle.pending is pending           # rows: nothing else is written
                    got = bundle.read(dev(tk), dev(w), eps, dtype)
                    assert (got.double().cpu() - want).abs().max() < bound, (k, same)
                    if result is not None:
                        assert bundle.pending is None and bundle.x32.shape[0] == n
                        err = max(float((bundle.x32[t].double().cpu() - new[t]).abs().max() / new[t].abs().max()) for t in range(n))
                        assert err < 4e-6, (k, same)
                    else:
                        assert torch.equal(bundle.x32.cpu(), x)


def _conv_rows(lens, before, u, taps):
    """Every row's convolution given the inputs before it: [rows] of [len, C] (float64)."""
    out, at = [], 0
    for n, past in zip(lens, before):
        out.append(plain.short_conv(torch.cat([past, u[at:at + n]]), taps)[past.shape[0]:])
        at += n
    return torch.cat(out)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("nq,nkv,d,dv,rot,taps", [(3, 1, 10, 6, 4, 3), (4, 2, 32, 32, 32, 4), (4, 2, 32, 20, 6, 2), (2, 2, 130, 20, 0, 7),
                                                  (16, 4, 128, 128, 64, 4), (5, 5, 12, 8, 12, 1), (8, 1, 64, 64, 30, None), (40, 8, 128, 128, 128, 3)])
def test_qk_row_norm_across_steps(nq, nkv, d, dv, rot, taps, dtype, tol):
    """Bias, convolution across a step's border (from the request's memory), the norm over whole rows, the rotation and the
    cache write, in steps of rows of many and of one token, over scattered pages and slots; long enough that a block of the
    kernel walks several tokens and crosses from one row into the next; padded heads count their real entries only."""
    o = ops()
    g = torch.Generator().manual_seed(d + nq)
    P, C, eps = 4, (nq + nkv) * d + nkv * dv, 1e-5
    T_all = 620 if d == 128 and nq == 16 else 60
    lens = [T_all - 22, 1, 3, 18]
    befores = [0, 9, 2, 30]
    NP = sum(-(-(b + n) // P) for b, n in zip(befores, lens)) + 2
    lay = rows_layout(befores, lens, P, NP, seed=d)
    T = lay["num_tokens"]
    memory = max((taps or 1) - 1, 0)
    state_off, slots = 8, [5, 2, 0, 3]
    state = _rand(g, 7, state_off + memory * C + (-(memory * C)) % 4)
    rows = _rand(g, T, C + 8, dtype=dtype)
    bias, wq, wk = _rand(g, C), 1 + 0.3 * _rand(g, nq * d), 1 + 0.3 * _rand(g, nkv * d)
    conv_w = _rand(g, C, taps, scale=0.6) if taps else None
    freq = torch.tensor([0.7 ** i for i in range(rot // 2)])
    q_count = nq * d - 3
    k_pages = torch.zeros(NP, nkv, P, d, dtype=dtype, device=DEV)
    v_pages = torch.zeros(NP, nkv, P, dv, dtype=dtype, device=DEV)
    q = torch.empty(T, nq * d, dtype=dtype, device=DEV)
    sd = state.to(DEV)
    starts = torch.tensor(np.cumsum([0] + lens), dtype=torch.int32, device=DEV)
    slot_t = torch.tensor(slots, dtype=torch.int32, device=DEV)
    conv = o.ShortConv(conv_w.to(DEV), sd, state_off, starts, slot_t, update_single=True) if taps else None
    table = o.rope_table(lay["positions"], freq.to(DEV)) if rot else None
    dev_rows = rows.to(DEV)[:, :C]
    o.qk_row_norm(dev_rows, wq.to(DEV), wk.to(DEV), table, lay["positions"], lay["token_row"], lay["block_table"], lay["page_base"],
                  k_pages, v_pages, nq, nkv, d, dv, True, eps, q, bias32=bias.to(DEV), conv=conv, q_count=q_count, v_scale=0.6)
    if memory:
        o.conv_state_update(dev_rows, sd, state_off, starts, slot_t, len(lens), C, taps, skip_single=True, bias32=bias.to(DEV))
    u = rows[:, :C].double() + bias.double()
    past = [state[s, state_off:state_off + memory * C].double().view(memory, C) for s in slots]
    x = _conv_rows(lens, past, u, conv_w.double()) if taps else u
    pos = lay["positions"].cpu()

    def turned(rows_, heads):
        y = rows_.view(T, heads, d).clone()
        ang = pos.double()[:, None] * freq.double()
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        a, b = y[..., 0:rot:2].clone(), y[..., 1:rot:2].clone()
        y[..., 0:rot:2], y[..., 1:rot:2] = a * c - b * s, b * c + a * s
        return y

    xq, xk = x[:, :nq * d], x[:, nq * d:(nq + nkv) * d]
    want_q = turned(xq / torch.sqrt((xq * xq).sum(-1, keepdim=True) / q_count + eps) * wq.double(), nq).reshape(T, -1)
    want_k = turned(plain.rms_norm(xk, wk.double(), eps), nkv)
    want_v = 0.6 * x[:, (nq + nkv) * d:].reshape(T, nkv, dv)
    bound = lambda t: tol * max(1.0, float(t.abs().max()))
    assert (q.double().cpu() - want_q).abs().max() < bound(want_q)
    t = 0
    for r, (b, n) in enumerate(zip(befores, lens)):
        for i in range(n):
            page, slot = lay["tables"][r][(b + i) // P], (b + i) % P
            assert (k_pages[page, :, slot].double().cpu() - want_k[t]).abs().max() < bound(want_k)
            assert (v_pages[page, :, slot].double().cpu() - want_v[t]).abs().max() < bound(want_v)
            t += 1
    if memory:
        at = 0
        for s, n, before in zip(slots, lens, past):
            kept = torch.cat([before, u[at:at + n]])[-memory:]
            assert (sd[s, state_off:state_off + memory * C].double().cpu().view(memory, C) - kept).abs().max() < 1e-5 * float(kept.abs().max())
            at += n
        untouched = [s for s in range(7) if s not in slots]
        assert torch.equal(sd[untouched].cpu(), state[untouched])


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("H,KH,dim,vdim,taps", [(4, 2, 6, 9, 3), (6, 3, 32, 24, 4), (2, 1, 128, 128, 4), (3, 3, 12, 20, 1), (2, 2, 136, 8, 6), (4, 1, 64, 64, None)])
def test_delta_rule_across_steps(H, KH, dim, vdim, taps, dtype, tol):
    """The delta rule's mixer kernels over rows of very unequal length, then every row's next tokens one by one (the kernel
    for a token at once where the sizes allow it, the general ones otherwise), from states that were there before, in
    scattered slots; beside other tokens of the same step or alone."""
    o = ops()
    g = torch.Generator().manual_seed(dim)
    C, eps = 2 * KH * dim + H * vdim, 1e-5
    gate_col = C + (-C) % 8
    beta_col = gate_col + H * vdim + (-(H * vdim)) % 8
    width = beta_col + 2 * H + (-(2 * H)) % 8
    S_size, memory = H * dim * vdim, max((taps or 1) - 1, 0)
    s_off = 4
    conv_off = s_off + S_size + (-S_size) % 4
    slots, lens, tail = [3, 0, 4], [150, 2, 37], 5
    stride = conv_off + memory * C
    state = _rand(g, 6, stride + (-stride) % 4, scale=0.5)
    rows = [_rand(g, n + tail, width, dtype=dtype) for n in lens]
    a_log, dt_bias, norm_w = _rand(g, H) - 1.0, _rand(g, H), _rand(g, vdim)
    conv_w = _rand(g, C, taps, scale=0.6) if taps else None
    dv = lambda t: None if t is None else t.to(DEV)
    sd = state.to(DEV)
    outs = [torch.empty(n + tail, H * vdim) for n in lens]

    def run(parts, ids):
        n = [p.shape[0] for p in parts]
        x = torch.cat(parts).to(DEV)
        starts = torch.tensor(np.cumsum([0] + n), dtype=torch.int32, device=DEV)
        rows_of = torch.repeat_interleave(torch.arange(len(n)), torch.tensor(n)).to(torch.int32).to(DEV)
        slot_t = torch.tensor([slots[i] for i in ids], dtype=torch.int32, device=DEV)
        ins = o.delta_heads_prep(x, beta_col, beta_col + H, dv(conv_w), sd, conv_off, dv(a_log), dv(dt_bias), rows_of, starts, slot_t,
                                 H, KH, dim, vdim, update_single=True)
        if memory and max(n) > 1:
            o.conv_state_update(x, sd, conv_off, starts, slot_t, len(n), C, taps, skip_single=True)
        gate = x[:, gate_col:gate_col + H * vdim]
        y = torch.empty((x.shape[0], H * vdim + 8), dtype=dtype, device=DEV)[:, :H * vdim]
        if max(n) == 1 and o.recurrent_step_ok(dim, vdim, (sd, sd.stride(0), s_off), (gate, y)):
            o.recurrent_step(sd, s_off, slot_t, gate, dv(norm_w), eps, y, H, dim, vdim, 0.9, delta=ins)
        else:
            q, k, v, beta, dec, log_dec = ins
            r = o.delta_rule(q, k, v, beta, dec, sd, starts, slot_t, len(n), longest_row=max(n), state_off=s_off, log_g=log_dec)
            o.gated_norm(r.view(x.shape[0], -1), gate, dv(norm_w.repeat(H)), eps, H, False, y, 0.9, silu=True)
        return torch.split(y.float().cpu(), n)

    for i, part in enumerate(run([r[:n] for r, n in zip(rows, lens)], [0, 1, 2])):
        outs[i][:lens[i]] = part
    for j in range(tail):
        order = [2, 0, 1] if j % 2 else [0, 1, 2]
        for i, part in zip(order, run([rows[i][lens[i] + j:lens[i] + j + 1] for i in order], order)):
            outs[i][lens[i] + j] = part[0]
    group = torch.arange(H) // (H // KH)
    for i, r in enumerate(rows):
        u = r[:, :C].double()
        past = state[slots[i], conv_off:conv_off + memory * C].double().view(memory, C)
        x = plain.silu(plain.short_conv(torch.cat([past, u]), conv_w.double())[memory:]) if taps else plain.silu(u)
        T = x.shape[0]
        q = (plain.unit(x[:, :KH * dim].reshape(T, KH, dim)) * dim ** -0.5)[:, group]
        k = plain.unit(x[:, KH * dim:2 * KH * dim].reshape(T, KH, dim))[:, group]
        v = x[:, 2 * KH * dim:].reshape(T, H, vdim)
        beta = plain.sigmoid(r[:, beta_col:beta_col + H].double())
        dec = torch.exp(-torch.exp(a_log.double()) * plain.softplus(r[:, beta_col + H:beta_col + 2 * H].double() + dt_bias.double()))
        want, S = plain.delta_recurrence(q, k, v, beta, dec, state[slots[i], s_off:s_off + S_size].double().view(H, dim, vdim))
        y = plain.rms_norm(want, norm_w.double(), eps).reshape(T, -1) * plain.silu(r[:, gate_col:gate_col + H * vdim].double()) * 0.9
        assert (outs[i].double() - y).abs().max() < tol * max(1.0, float(y.abs().max())), i
        assert (sd[slots[i], s_off:s_off + S_size].double().cpu().view(H, dim, vdim) - S).abs().max() < 2e-5 * max(1.0, float(S.abs().max()))
        if memory:
            kept = torch.cat([past, u])[-memory:]
            assert (sd[slots[i], conv_off:conv_off + memory * C].double().cpu().view(memory, C) - kept).abs().max() < 1e-6
    untouched = [s for s in range(6) if s not in slots]
    assert torch.equal(sd[untouched].cpu(), state[untouched]) and torch.equal(sd[:, :s_off].cpu(), state[:, :s_off])


def test_delta_rule_long_memory():
    """A write at the first token, hardly any decay and no later write to the same key: hundreds of tokens on, across every
    chunk and segment of the recurrence and in another step, the read-out still is what was written."""
    o = ops()
    g = torch.Generator().manual_seed(5)
    H, KH, dim, vdim = 2, 1, 32, 24
    for T, cut in ((700, 0), (700, 1), (700, 63), (700, 64), (700, 65), (700, 128), (700, 333), (2, 1)):
        basis = torch.linalg.qr(_rand(g, dim, dim).double())[0]
        k = basis[1 + torch.randint(0, dim - 1, (T,), generator=g)].unsqueeze(1)          # [T, 1, dim], never basis[0] but at the start
        k[0, 0] = basis[0]
        q = basis[0].expand(T, 1, dim).contiguous()
        v, beta = _rand(g, T, H, vdim).double(), torch.rand(T, H, generator=g).double()
        dec = torch.full((T, H), 0.9995, dtype=torch.float64)
        state = torch.zeros(3, H * dim * vdim, device=DEV)
        f = lambda t: t.float().contiguous().to(DEV)
        got = []
        for a, b in (((0, cut), (cut, T)) if cut else ((0, T),)):
            got.append(o.delta_rule(f(q[a:b]), f(k[a:b]), f(v[a:b]), f(beta[a:b]), f(dec[a:b]), state,
                                    torch.tensor([0, b - a], dtype=torch.int32, device=DEV), torch.tensor([1], dtype=torch.int32, device=DEV), 1,
                                    longest_row=b - a, log_g=f(dec[a:b].log())).double().cpu())
        got = torch.cat(got)
        want = beta[0][:, None] * v[0] * (0.9995 ** torch.arange(T, dtype=torch.float64))[:, None, None]
        assert (got - want).abs().max() < 2e-5 * float(want.abs().max()), (T, cut)


@pytest.mark.parametrize("H,KH,dim,vdim", [(4, 2, 8, 12), (3, 3, 32, 20), (2, 1, 64, 64), (6, 3, 96, 80), (2, 2, 128, 128), (1, 1, 128, 200)])
def test_delta_chunks(H, KH, dim, vdim):
    """The delta rule over chunks of tokens against the loop over tokens and against the kernel that walks them: rows that end
    on and around a chunk's edge, many and unequal rows in one step, keys that repeat (a system far from the identity),
    decays from none to those that leave nothing, states that were there before."""
    o = ops()
    g = torch.Generator().manual_seed(dim + vdim)
    for lens in ([64], [65, 1, 63], [1, 200, 2, 128, 129, 5, 64, 192], [330]):
        T, slots = sum(lens), list(np.random.default_rng(len(lens)).permutation(10)[:len(lens)])
        base = _rand(g, KH, dim)
        k = plain.unit((_rand(g, T, KH, dim, scale=0.4) + base).double())          # neighbouring keys are alike
        q = plain.unit(_rand(g, T, KH, dim).double()) * dim ** -0.5
        v, beta = _rand(g, T, H, vdim).double(), torch.rand(T, H, generator=g).double()
        log_g = -torch.exp(_rand(g, T, H, scale=2.0).double() - 3.0)
        log_g[T // 2] = -90.0
        state = _rand(g, 10, H * dim * vdim + 4)
        f = lambda t: t.float().contiguous().to(DEV)
        starts = torch.tensor(np.cumsum([0] + lens), dtype=torch.int32, device=DEV)
        slot_t = torch.tensor(slots, dtype=torch.int32, device=DEV)
        got, ends = {}, {}
        for how in ("chunks", "walk"):
            sd = state.to(DEV)
            if how == "chunks":
                out = o.delta_chunk(f(q), f(k), f(v), f(beta), f(log_g), sd, starts, slot_t, len(lens), state_off=4)
            else:
                out = o.delta_rule(f(q), f(k), f(v), f(beta), f(log_g.exp()), sd, starts, slot_t, len(lens), state_off=4)
            got[how], ends[how] = out.double().cpu(), sd.double().cpu()
        group, at = torch.arange(H) // (H // KH), 0
        for r, n in enumerate(lens):
            rows = slice(at, at + n)
            want, S = plain.delta_recurrence(q[rows][:, group], k[rows][:, group], v[rows], beta[rows], log_g[rows].exp(),
                                             state[slots[r], 4:].double().view(H, dim, vdim))
            for how in got:
                assert (got[how][rows] - want).abs().max() < 3e-5 * float(want.abs().max()), (lens, r, how)
                assert (ends[how][slots[r], 4:].view(H, dim, vdim) - S).abs().max() < 3e-5 * float(S.abs().max()), (lens, r, how)
            at += n
        untouched = [s for s in range(10) if s not in slots]
        assert torch.equal(ends["chunks"][untouched], state[untouched].double()) and torch.equal(ends["chunks"][:, :4], state[:, :4].double())


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("H,dim,vdim,tau", [(3, 5, 7, 1.0), (4, 32, 64, 16.0), (2, 128, 128, 4.0), (2, 140, 20, 8.0), (8, 64, 128, 16.0), (1, 16, 200, 2.0)])
def test_linear_attention_across_steps(H, dim, vdim, tau, dtype, tol):
    """Gated linear attention over long rows (over chunks of tokens, or walked in segments), short ones and single tokens in
    one step, then tokens one by one; decays from none to those that leave nothing between two tokens."""
    o = ops()
    g = torch.Generator().manual_seed(dim + vdim)
    Hd, Hv, eps = H * dim, H * vdim, 1e-5
    gate_col = 2 * Hd + Hv + (-(2 * Hd + Hv)) % 8
    width = gate_col + Hv + (-Hv) % 8
    S_size, s_off = Hd * vdim, 8
    norm_w, bias = _rand(g, vdim), _rand(g, Hd)
    took = set()
    for lens, slots, chunks in (([400], [2], False), ([400], [2], True), ([190, 1, 33], [4, 0, 1], True), ([64, 65, 1, 129, 63], [4, 0, 1, 5, 2], True)):
        tail = 4
        state = _rand(g, 6, s_off + S_size + (-S_size) % 4, scale=0.5)
        rows = [_rand(g, n + tail, width, dtype=dtype) for n in lens]
        zs = [_rand(g, n + tail, Hd, scale=2.0) + 2.0 for n in lens]
        zs[0][20:23] -= 400.0
        zs[0][::7] += 30.0
        sd = state.to(DEV)
        outs = [torch.empty(n + tail, Hv) for n in lens]

        def run(parts, zparts, ids):
            n = [p.shape[0] for p in parts]
            x, z = torch.cat(parts).to(DEV), torch.cat(zparts).to(DEV)
            starts = torch.tensor(np.cumsum([0] + n), dtype=torch.int32, device=DEV)
            slot_t = torch.tensor([slots[i] for i in ids], dtype=torch.int32, device=DEV)
            gate = x[:, gate_col:gate_col + Hv]
            y = torch.empty((x.shape[0], Hv + 16), dtype=dtype, device=DEV)[:, 8:8 + Hv]
            if max(n) == 1 and (Hd % 2 == 0) and o.recurrent_step_ok(dim, vdim, (sd, sd.stride(0), s_off), (x, gate, y)):
                o.recurrent_step(sd, s_off, slot_t, gate, norm_w.to(DEV), eps, y, H, dim, vdim, 1.3, linear=(x, z, bias.to(DEV), tau))
            else:
                if chunks and o.linear_chunk_ok(max(n), x, z, sd, s_off, len(n), H, dim, vdim):
                    took.add("chunks")
                    r = o.linear_chunk(x, z, bias.to(DEV), tau, sd, starts, slot_t, len(n), H, dim, vdim, state_off=s_off)
                else:
                    q, k, v, al = o.linear_heads_prep(x, z, bias.to(DEV), tau, H, dim, vdim)
                    r = o.delta_rule(q, k, v, None, al, sd, starts, slot_t, len(n), longest_row=max(n), state_off=s_off)
                o.gated_norm(r.view(x.shape[0], -1), gate, norm_w.repeat(H).to(DEV), eps, H, False, y, 1.3, silu=True)
            return torch.split(y.float().cpu(), n)

        ids = list(range(len(lens)))
        for i, part in enumerate(run([r[:n] for r, n in zip(rows, lens)], [z[:n] for z, n in zip(zs, lens)], ids)):
            outs[i][:lens[i]] = part
        for j in range(tail):
            at = [lens[i] + j for i in ids]
            for i, part in enumerate(run([r[a:a + 1] for r, a in zip(rows, at)], [z[a:a + 1] for z, a in zip(zs, at)], ids)):
                outs[i][at[i]] = part[0]
        for i, (r, z) in enumerate(zip(rows, zs)):
            T = r.shape[0]
            r64 = r.double()
            al = torch.exp(-plain.softplus(-(z.double() + bias.double())) / tau).view(T, H, dim)
            want, S = plain.gla_recurrence(r64[:, :Hd].reshape(T, H, dim) * dim ** -0.5, r64[:, Hd:2 * Hd].reshape(T, H, dim),
                                           r64[:, 2 * Hd:2 * Hd + Hv].reshape(T, H, vdim), al, state[slots[i], s_off:s_off + S_size].double().view(H, dim, vdim))
            y = plain.rms_norm(want, norm_w.double(), eps).reshape(T, -1) * plain.silu(r64[:, gate_col:gate_col + Hv]) * 1.3
            assert (outs[i].double() - y).abs().max() < tol * max(1.0, float(y.abs().max())), (lens, i)
            assert (sd[slots[i], s_off:s_off + S_size].double().cpu().view(H, dim, vdim) - S).abs().max() < 2e-5 * max(1.0, float(S.abs().max()))
        untouched = [s for s in range(6) if s not in slots]
        assert torch.equal(sd[untouched].cpu(), state[untouched]) and torch.equal(sd[:, :s_off].cpu(), state[:, :s_off])
    assert took or dim % 4 or vdim % 4 or dim > 128


def test_sink_at_zero_where_one_key_decides():
    """A window, a cap and one added to the denominator in every attention kernel: a spiked key just inside or just outside
    the window of a prompt's rows and of decoded tokens, at page borders and far back; where all other scores are low, the
    sink takes its share, which leaving it out would double."""
    o = ops()
    g = torch.Generator().manual_seed(21)
    P, i32 = 16, dict(dtype=torch.int32, device=DEV)
    befores, qlens = [0, 499, 300, 63, 64], [180, 1, 130, 1, 1]
    for dtype, tol, kernel, d, dv, nq, nkv in ((torch.float32, 2e-5, "plain", 24, 10, 6, 3), (torch.bfloat16, 2e-2, "mma", 64, 64, 6, 2),
                                               (torch.bfloat16, 2e-2, "mma", 96, 96, 8, 1), (torch.bfloat16, 2e-2, "tc", 128, 128, 8, 2),
                                               (torch.bfloat16, 2e-2, "plain", 40, 56, 4, 1)):
        NP = sum(-(-(b + q) // P) for b, q in zip(befores, qlens)) + 3
        lay = rows_layout(befores, qlens, P, NP, seed=d)
        for window in (48, 65, None):
            edge = (window or 700) - 1
            # the decoded tokens' spikes: just inside (row 1), just outside (row 3 keeps none visible but the low ones)
            spikes = {0: (0, 63, 64, 130), 1: (499 - edge,) if window else (3,), 2: (300 - edge - 1 if window else 15, 299), 3: (63 - edge - 1,) if window and window < 63 else (0,),
                      4: (64,) if window else ()}
            k_pages = torch.zeros(NP, nkv, P, d, dtype=dtype, device=DEV)
            v_pages = torch.zeros(NP, nkv, P, dv, dtype=dtype, device=DEV)
            full = []
            for r, (b, n) in enumerate(zip(befores, qlens)):
                S = b + n
                k, v, q = _rand(g, S, nkv, d, scale=0.2), _rand(g, S, nkv, dv), _rand(g, S, nq, d, scale=0.2)
                k[:, :, d - 1] = -2.5                                    # every ordinary score about -5
                for j in spikes[r]:
                    if j >= 0:
                        k[j, :, d - 1] = 6.0
                q[:, :, d - 1] = 4.0
                k, v, q = k.to(dtype), v.to(dtype), q.to(dtype)
                scatter_to_pages(k_pages, lay["tables"][r], k, P)
                scatter_to_pages(v_pages, lay["tables"][r], v, P)
                full.append((q.double(), k.double(), v.double()))
            q_new = torch.cat([f[0][b:] for f, b in zip(full, befores)]).to(dtype).to(DEV).contiguous().view(-1, nq * d)
            common = (k_pages, v_pages, lay["block_table"], lay["page_base"])
            T, scale, zero = lay["num_tokens"], 0.5, torch.zeros(nq, device=DEV)
            starts = np.cumsum([0] + qlens)
            for cap in (None, 20.0):
                want, without = [], []
                for (fq, fk, fv), b in zip(full, befores):
                    S = fq.shape[0]
                    s = torch.einsum("ihd,jhd->hij", fq, fk.repeat_interleave(nq // nkv, 1)) * scale
                    s = cap * torch.tanh(s / cap) if cap else s
                    ok = plain.visible(S, window)
                    fold = lambda p: torch.einsum("hij,jhd->ihd", p, fv.repeat_interleave(nq // nkv, 1))[b:]
                    want.append(fold(plain.softmax_plus_one(s, ok)))
                    without.append(fold(torch.softmax(s.masked_fill(~ok, -math.inf), -1)))
                want, without = torch.cat(want), torch.cat(without)
                assert (want - without).abs().max() > 0.1
                for splits in (1, 3):
                    if kernel == "plain":
                        out = o.attention_plain(q_new, nq * d, *common, lay["token_row"], lay["positions"], T, nq, nkv, d, scale, window,
                                                value_dim=dv, softcap=cap, sink32=zero)
                    else:
                        out = torch.zeros((T, nq * dv), dtype=dtype, device=DEV)
                        step = 128 if kernel == "tc" else 64
                        tiles = torch.tensor([(r, q0) for r, n in enumerate(qlens) if n > 1 for q0 in range(0, n, step)], **i32)
                        fn = o.attention_prefill_tc if kernel == "tc" else o.attention_prefill
                        fn(q_new, nq * d, *common, torch.tensor(starts, **i32), torch.tensor(befores, **i32), tiles, T, nq, nkv, d, scale,
                           window, out=out, softcap=cap, sink32=zero)
                        singles = torch.tensor([int(starts[r]) for r, n in enumerate(qlens) if n == 1], **i32)
                        o.attention_decode(q_new, nq * d, *common, lay["token_row"], lay["positions"], T, nq, nkv, d, scale, window, splits,
                                           token_list=singles, out=out, use_tma=False, softcap=cap, sink32=zero)
                    got = out.float().cpu().view(-1, nq, dv)
                    assert (got - want).abs().max() < tol * max(1.0, float(want.abs().max())), (kernel, d, window, cap, splits)


@pytest.mark.parametrize("T,N,top", [(1, 5, 2), (9, 5, 2), (40, 12, 1), (3, 7, 7), (129, 33, 3), (700, 8, 4)])
def test_router_bias_and_weights_over_the_chosen(T, N, top):
    """A bias on the router's logits decides the choice; the weights are the softmax over the chosen logits alone."""
    o = ops()
    g = torch.Generator().manual_seed(T)
    z, bias = _rand(g, T, N, scale=2.0), _rand(g, N, scale=3.0)
    z[0] += 50.0
    full = z.double() + bias.double()
    best = torch.topk(full, top, dim=-1)
    want = torch.softmax(best.values, -1)
    idx, wts, offsets, slot_of, slot_token, _ = o.moe_route_plan(z.to(DEV), None, top, 1, 1, True, "softmax", bias32=bias.to(DEV))
    assert torch.equal(idx.cpu().long(), best.indices) and (wts.cpu().double() - want).abs().max() < 2e-5
    off = offsets.cpu().long()
    assert torch.equal(off[1:] - off[:-1], torch.bincount(best.indices.flatten(), minlength=N))
    idx2, wts2 = o.moe_route(z.to(DEV), None, top, 1, 1, True, "softmax", bias32=bias.to(DEV))
    assert torch.equal(idx2, idx) and (wts2 - wts).abs().max() < 1e-6


def test_gated_norm_with_silu():
    """The norm of a head's read-out with one weight and a silu gate, in the form a warp a head and in the general one."""
    o = ops()
    g = torch.Generator().manual_seed(3)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        for H, vdim in ((4, 64), (2, 128), (3, 256), (1, 20), (5, 6), (2, 260)):
            y, gate, w = _rand(g, 9, H * vdim), _rand(g, 9, H * vdim + 16, dtype=dtype), _rand(g, vdim)
            out = torch.empty(9, H * vdim + 8, dtype=dtype, device=DEV)[:, :H * vdim]
            o.gated_norm(y.to(DEV), gate.to(DEV)[:, 8:8 + H * vdim], w.repeat(H).to(DEV), 1e-5, H, False, out, 0.7, silu=True)
            want = plain.rms_norm(y.double().view(9, H, vdim), w.double(), 1e-5).reshape(9, -1) * plain.silu(gate[:, 8:8 + H * vdim].double()) * 0.7
            assert (out.double().cpu() - want).abs().max() < tol * max(1.0, float(want.abs().max())), (H, vdim)


def test_a_table_of_angles_is_made_again_in_captured_steps(tmp_path):
    """Decoded tokens of a rotated layer replayed from a captured graph turn by their own positions."""
    tiny = BADEPELS["bad_c"]
    d = make_model_dir(tmp_path, tiny)
    w = read_weights(d)
    toks = random_tokens(40, tiny["cfg"].vocab_size, 12)
    ref = plain_logits(tiny["cfg"], w, {"g": toks})
    got, runner = run_cut(tiny, d, traces.decode_tail({"g": toks}, tail=36), "float32")
    assert runner.graph_replays >= 20
    check(got, ref, "float32", "captured angles")
