"""Zusolix on the GPU against the plain implementation (``tests/plain/zusolix.py``, float64).

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

from acorninfer_b200.config.model_config import ZusolixConfig
from tests import traces
from tests.paged import rows_layout, scatter_to_pages
from tests.plain import zusolix as plain
from tests.tiny import random_tokens
from tests.zusolix_tiny import ZUS_LONG, ZUSES, L, att, gru, make_model_dir, moe, random_config, read_weights

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


@pytest.fixture(scope="module", params=list(ZUSES))
def case(request, tmp_path_factory):
    tiny = ZUSES[request.param]
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
    """Decoding four requests at a time from captured graphs, whose layers run their two sublayers (and the shared expert) as
    branches side by side, against the same steps launched one by one."""
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
    """A request whose first step is a single token (a recurrence from the zero state, a softmax of one key), then
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
    """Requests of a few hundred tokens over pages of 16: several chunks of keys in the tensor-core kernels, several
    segments of the recurrence, portions that end at and around a segment's edge."""
    tiny = ZUS_LONG
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


@pytest.mark.parametrize("seed", [1, 4, 6, 9])
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
    ref = plain_logits(tiny["cfg"], w, reqs, close_gap=0.04)          # smaller weights than above: smaller router logits
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
    """``bin/trace_run`` as a program on a Zusolix folder: it picks the model by ``config.json``, runs a mixed trace in
    a pool sized for the live requests and writes the logits asked for."""
    import json
    import subprocess
    import sys
    from pathlib import Path
    tiny = ZUSES["zus_b"]
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


def _solo(mixer, ff=None, width=48, vocab=90, groups=1, mult=1.0, emb=1.0, more=()):
    return ZusolixConfig(vocab_size=vocab, hidden_size=width, norm_eps=1e-5, norm_groups=groups, residual_mult=mult,
                         embedding_scale=emb, layers=(L(mixer, ff),) + tuple(more))


_SMALL = att(heads=1, kv_heads=1, dim=4, scale=0.5)
SOLOS = {
    "attention, nothing but keys": _solo(att(heads=3, kv_heads=3, dim=10, scale=0.6)),
    "attention, values wider than keys": _solo(att(heads=4, kv_heads=2, dim=6, vdim=22, scale=0.5)),
    "attention, values narrower, one head": _solo(att(heads=1, kv_heads=1, dim=16, vdim=3, scale=0.5)),
    "attention, a cap that bites": _solo(att(heads=2, kv_heads=1, dim=8, scale=2.0, cap=0.5)),
    "attention, 9 query heads a key head, a temperature": _solo(att(heads=9, kv_heads=1, dim=16, scale=0.4, coef=0.7, every=4)),
    "attention, a temperature that steps at every position": _solo(att(heads=2, kv_heads=2, dim=32, scale=0.3, cap=6.0, coef=0.5, every=1)),
    "attention, heads of 130": _solo(att(heads=2, kv_heads=1, dim=130, scale=0.1, coef=0.3, every=9)),
    "minGRU as wide as the model": _solo(gru(48)),
    "minGRU, one channel": _solo(gru(1)),
    "minGRU, 531 channels": _solo(gru(531), emb=2.0),
    "minGRU twice": _solo(gru(16), more=(L(gru(36), ff=20),)),
    "gated feed-forward, widths no multiple of 8": _solo(_SMALL, ff=37, width=44),
    "experts: one choice of seven, no shared expert": _solo(_SMALL, ff=moe(11, 7, 1)),
    "experts: all three chosen, a wide shared expert": _solo(_SMALL, ff=moe(8, 3, 3, 40)),
    "experts: two of thirteen": _solo(_SMALL, ff=moe(24, 13, 2, 8), width=40),
    "a norm in parts of one entry": _solo(_SMALL, ff=16, width=12, groups=12),
    "a norm in four parts, small results": _solo(_SMALL, ff=16, groups=4, mult=0.1, emb=5.0),
    "five layers without feed-forward": _solo(_SMALL, more=(L(gru(9)), L(_SMALL), L(gru(12)), L(_SMALL)), mult=0.8),
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
    tiny = ZUSES["zus_a"]
    d = make_model_dir(tmp_path, tiny)
    w = read_weights(d)
    cfg = tiny["cfg"].to_dict()
    toks = random_tokens(30, tiny["cfg"].vocab_size, 3)
    full = plain.forward(cfg, w, toks).numpy()

    def differs(c, ww):
        return max(rel_err(a, b) for a, b in zip(plain.forward(c, ww, toks).numpy(), full)) > 100 * TOL["float32"]

    for path, value in ((("layers", 0, "mixer", "q_temp", "coef"), 0.0), (("layers", 0, "mixer", "q_temp", "every"), 6),
                        (("layers", 0, "mixer", "softcap"), None), (("layers", 0, "mixer", "scale"), 0.45), (("norm", "groups"), 1),
                        (("residual_mult",), 1.0), (("embedding", "scale"), 1.0), (("layers", 1, "mlp", "router", "top"), 1),
                        (("layers", 1, "mlp", "shared"), None)):
        other = copy.deepcopy(cfg)
        node = other
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        assert differs(other, w), path
    for name in ("l0.mix.q.b", "l0.mix.v.b", "l1.mix.z.b", "l1.mix.x.b", "l1.mlp.shared.sg", "l1.mlp.router"):
        assert differs(cfg, dict(w, **{name: torch.zeros_like(w[name])})), name
    for name in ("l0.dwa", "l1.dwa", "l2.dwa", "l3.dwa"):
        for j in range(w[name].numel()):
            one = w[name].clone()
            one[j] = 0.0
            assert differs(cfg, dict(w, **{name: one})), (name, j)


def ops():
    from acorninfer_b200.kernels import ops as o
    return o


def _rand(g, *shape, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("width,groups", [(12, 3), (72, 1), (96, 4), (256, 2), (512, 1), (1280, 10), (2048, 4), (4608, 4), (130, 130)])
def test_stream_norm(width, groups, dtype, tol):
    """Pending results of every kind, the sum over earlier streams, and one or two norms in groups, with parts of very
    unequal size, in place and into memory of its own, all rows or some of them (one twice)."""
    o = ops()
    g = torch.Generator().manual_seed(width)
    T, top, eps = 7, 2, 1e-5
    d64 = lambda t: t.double()
    part = torch.repeat_interleave(torch.logspace(-1, 1, groups), width // groups)
    w1, w2 = _rand(g, width), _rand(g, width)
    dev = lambda t: None if t is None else t.to(DEV)
    a, b, extra = (_rand(g, T, width, dtype=dtype) for _ in range(3))
    y = _rand(g, T * top, width, dtype=dtype)
    slot_of = torch.randperm(T * top, generator=g).view(T, top).to(torch.int32)
    zwide = _rand(g, T, 5)
    experts = y.double()[slot_of.long()].sum(1)
    gated = experts + torch.sigmoid(zwide.double()[:, 3:4]) * d64(extra)
    zdev = zwide.to(DEV)[:, 3:4]
    E = lambda ex, z: o.ExpertsPending(dev(y), dev(slot_of), dev(ex), z)
    cases = [(None, 0.0), (dev(a), d64(a)), (o.DeltaPair(dev(a), dev(b), 0.4), 0.4 * (d64(a) + d64(b))),
             (o.DeltaPair(dev(a), None, -1.5), -1.5 * d64(a)), (o.DeltaPair(dev(a), E(None, None), 0.7), 0.7 * (d64(a) + experts)),
             (o.DeltaPair(dev(a), E(extra, None), 1.0), d64(a) + experts + d64(extra)),
             (o.DeltaPair(dev(a), E(extra, zdev), 0.5), 0.5 * (d64(a) + gated))]
    rows = torch.tensor([3, 0, 3, 6], dtype=torch.int32)

    def norms_of(x, which):
        return [plain.grouped_norm(x, d64(w), eps, groups) for w in which]

    for n in (None, 0, 1, 2, 5, 9):                 # earlier streams; None: no history
        for k, (delta, add) in enumerate(cases):
            x = _rand(g, T, width) * part
            which = ((w1, w2), (w1,), ())[(k + (n or 0)) % 3]
            specs = tuple((dev(w), eps, groups) for w in which)
            hist = coef = None
            v = d64(x) + add
            new = v
            if n is not None:
                hist = _rand(g, n + 1, T, width) * part
                coef = _rand(g, n + 1)
                new = sum((c * h for c, h in zip(d64(coef[:n]), d64(hist[:n]))), torch.zeros_like(v)) + d64(coef[n]) * v
            scale_of = lambda t: max(1.0, float(t.abs().max()))
            xd, hd = dev(x), dev(hist)
            got = o.stream_norm(xd, delta, specs, dtype, rows=dev(rows), history=hd, coef32=dev(coef))
            assert torch.equal(xd.cpu(), x) and (hist is None or torch.equal(hd.cpu(), hist))      # rows: nothing else is written
            for have, want in zip(got, norms_of(new[rows.long()], which)):
                assert (have.float().cpu() - want).abs().max() < tol * scale_of(want), (n, k)
            for out in (None, torch.full((T, width), 9.0, device=DEV)):
                xd, hd = dev(x), dev(hist)
                got = o.stream_norm(xd, delta, specs, dtype, history=hd, coef32=dev(coef), x_out=out)
                res = xd if out is None else out
                if out is not None:
                    assert torch.equal(xd.cpu(), x)
                assert (res.cpu() - new).abs().max() < 2e-6 * (3 + (n or 0)) * scale_of(new), (n, k)
                assert len(got) == len(which)
                for have, want in zip(got, norms_of(new, which)):
                    assert (have.float().cpu() - want).abs().max() < tol * scale_of(want), (n, k)
                if n is not None:
                    assert (hd.cpu()[n] - v).abs().max() < 4e-6 * scale_of(v) and torch.equal(hd.cpu()[:n], hist[:n])
            if n is not None:                        # a history without room for the new result
                xd = dev(x)
                o.stream_norm(xd, delta, (), dtype, history=dev(hist[:n].contiguous()), coef32=dev(coef))
                assert (xd.cpu() - new).abs().max() < 2e-6 * (3 + n) * scale_of(new)


def test_grouped_norm_part_takes_pending_results():
    """The norm as a part of its own: what is still to be added goes into the stream, rows chosen or all."""
    from acorninfer_b200.parts.base import BuildContext
    from acorninfer_b200.parts.norms import GroupedRMSNorm
    o = ops()
    g = torch.Generator().manual_seed(8)
    for width, groups in ((20, 5), (384, 3)):
        w, x, a, b = _rand(g, width), _rand(g, 6, width), _rand(g, 6, width), _rand(g, 6, width)
        norm = GroupedRMSNorm(BuildContext(torch.float32, torch.device(DEV), 16), width, 1e-6, groups, "")
        norm.bind({"": w.to(DEV)})
        xd = x.to(DEV)
        got = norm.add_forward(xd, o.DeltaPair(a.to(DEV), b.to(DEV), 0.3))
        new = x.double() + 0.3 * (a.double() + b.double())
        assert (xd.cpu() - new).abs().max() < 1e-5
        assert (got.cpu() - plain.grouped_norm(new, w.double(), 1e-6, groups)).abs().max() < 1e-5
        rows = torch.tensor([5, 2], dtype=torch.int32, device=DEV)
        got = norm.forward(xd, rows=rows)
        assert (got.cpu() - plain.grouped_norm(new[[5, 2]], w.double(), 1e-6, groups)).abs().max() < 1e-5


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("width", [4, 7, 64, 132, 530, 1024])
def test_min_gru_kernel(width, dtype, tol):
    """Rows of very unequal length in one step (one token to several segments), states that were there before, slots in
    any order; gates mostly closed, so that a state lives through several segments; then the same tokens in two
    steps cut at several places."""
    o = ops()
    g = torch.Generator().manual_seed(width)
    bias = torch.cat([_rand(g, width) - 3.5, _rand(g, width)])
    slots, off = 9, 4

    def reference(rows, start):
        out = []
        for p, s in zip(rows, start):
            z = torch.sigmoid(p[:, :width].double() + bias[:width].double())
            c = plain.candidate(p[:, width:2 * width].double() + bias[width:].double())
            st = plain.gated_recurrence(z, c, s.double())
            out.append((st * plain.silu(p[:, 2 * width:].double()), st[-1]))
        return out

    def run(parts, state, slot_ids, longest):
        starts = torch.tensor(np.cumsum([0] + [p.shape[0] for p in parts]), dtype=torch.int32, device=DEV)
        y = o.min_gru(torch.cat(parts).to(DEV), bias.to(DEV), state, off, starts,
                      torch.tensor(slot_ids, dtype=torch.int32, device=DEV), len(parts), longest_row=longest)
        return [t.float().cpu() for t in torch.split(y, [p.shape[0] for p in parts])]

    for lens in ([1, 1, 1], [7, 1, 9], [32, 2, 8, 31], [33, 1, 8], [128, 127, 9], [129, 1, 128], [300, 2, 40, 257], [2048, 130], [2300]):
        if sum(lens) > 1000 and width > 140:
            continue
        rows = [_rand(g, n, 3 * width, dtype=dtype) for n in lens]
        ids = [7, 2, 5, 0][:len(lens)]
        state = _rand(g, slots, off + width + 3 + (-(off + width + 3)) % 4).to(DEV)
        before = state.cpu().clone()
        want = reference(rows, [before[i, off:off + width] for i in ids])
        got = run(rows, state, ids, max(lens))
        for r, (have, (y, s)) in enumerate(zip(got, want)):
            assert (have - y).abs().max() < tol * max(1.0, float(y.abs().max())), (lens, r)
            assert (state.cpu()[ids[r], off:off + width] - s).abs().max() < 2e-5 * max(1.0, float(s.abs().max())), (lens, r)
        after = state.cpu()
        touched = torch.zeros_like(after, dtype=torch.bool)
        for i in ids:
            touched[i, off:off + width] = True
        assert torch.equal(after[~touched], before[~touched])
        for cut in (1, 2, 33, 127, 128, 130):
            if cut >= lens[0]:
                continue
            st = before.to(DEV)
            head = run([rows[0][:cut]], st, [ids[0]], cut)[0]
            tail = run([rows[0][cut:]], st, [ids[0]], lens[0] - cut)[0]
            assert (torch.cat([head, tail]) - want[0][0]).abs().max() < tol * max(1.0, float(want[0][0].abs().max())), (lens, cut)


def test_query_temperature_at_the_edges_of_its_spans():
    """qk_rope_kv with biases and a temperature (the form with four channels a lane and the general one), alone and after
    a norm and a rotation: queries at the last position before a step, at the step, far out; keys and values untouched."""
    o = ops()
    g = torch.Generator().manual_seed(4)
    P, coef = 4, 0.6
    freq0 = torch.zeros(0, device=DEV)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 3e-2)):
        for nq, nkv, d, dv in ((3, 1, 10, 6), (4, 2, 32, 32), (2, 2, 130, 20), (2, 1, 128, 128), (4, 4, 64, 12)):
            for every in (1, 3, 8, 100000):
                befores, qlens = [every - 2 if 2 <= every < 50 else 0, 5, 2 * every - 1 if every < 50 else 60], [4, 3, 1]
                lay = rows_layout(befores, qlens, P, 40, seed=d)
                T = lay["num_tokens"]
                C = (nq + nkv) * d + nkv * dv
                rows, bias = _rand(g, T, C, dtype=dtype), _rand(g, C)
                k_pages = torch.zeros(40, nkv, P, d, dtype=dtype, device=DEV)
                v_pages = torch.zeros(40, nkv, P, dv, dtype=dtype, device=DEV)
                q = torch.empty(T, nq * d, dtype=dtype, device=DEV)
                common = (lay["positions"], lay["token_row"], lay["block_table"], lay["page_base"], k_pages, v_pages, nq, nkv, d)
                o.qk_rope_kv(rows.to(DEV), None, None, freq0, *common, 0, False, 0.0, value_dim=dv, bias32=bias.to(DEV), q_out=q,
                             q_temp=(coef, every))
                x = rows.double() + bias.double()
                f = plain.query_temperature(lay["positions"].tolist(), {"coef": coef, "every": every})
                want = x[:, :nq * d] * f[:, None]
                assert (q.float().cpu() - want).abs().max() < tol * 3
                t = 0
                for r, (b, n) in enumerate(zip(befores, qlens)):
                    for i in range(n):
                        page, slot = lay["tables"][r][(b + i) // P], (b + i) % P
                        assert (k_pages[page, :, slot].float().cpu().reshape(-1) - x[t, nq * d:(nq + nkv) * d]).abs().max() < tol * 3
                        assert (v_pages[page, :, slot].float().cpu().reshape(-1) - x[t, (nq + nkv) * d:]).abs().max() < tol * 3
                        t += 1
                if d % 2 or dv != d:
                    continue
                # after norm and rotation, and with the norm after the rotation (no biases)
                inv = torch.tensor([0.3 ** i for i in range(d // 2)])
                for after in (False, True):
                    buf = rows.to(DEV).clone()
                    wq = _rand(g, d)
                    o.qk_rope_kv(buf, wq.to(DEV), wq.to(DEV), inv.to(DEV), *common, d, True, 1e-5, q_temp=(coef, every), norm_after=after)
                    base = rows.to(DEV).clone()
                    o.qk_rope_kv(base, wq.to(DEV), wq.to(DEV), inv.to(DEV), *common, d, True, 1e-5, norm_after=after)
                    ratio = buf[:, :nq * d].double().cpu() - base[:, :nq * d].double().cpu() * f[:, None]
                    assert ratio.abs().max() < tol * 6


def test_capped_scores_where_one_far_key_decides():
    """Capped scores over all earlier keys in every attention kernel: a spiked key at the first position, at page and chunk
    borders and far back decides a prompt's rows and a decoded token; without the cap the result is another."""
    o = ops()
    g = torch.Generator().manual_seed(11)
    P, i32 = 16, dict(dtype=torch.int32, device=DEV)
    befores, qlens = [0, 699, 300, 63, 64], [200, 1, 130, 1, 1]
    spikes = {0: (0, 63, 64, 130), 1: (3,), 2: (15, 299), 3: (0,), 4: (64,)}
    for dtype, tol, kernel, d, dv, nq, nkv in ((torch.float32, 2e-5, "plain", 24, 10, 6, 3), (torch.bfloat16, 2e-2, "mma", 64, 64, 6, 2),
                                               (torch.bfloat16, 2e-2, "mma", 96, 96, 4, 4), (torch.bfloat16, 2e-2, "tc", 128, 128, 8, 2),
                                               (torch.bfloat16, 2e-2, "plain", 40, 56, 4, 1)):
        NP = sum(-(-(b + q) // P) for b, q in zip(befores, qlens)) + 3
        lay = rows_layout(befores, qlens, P, NP, seed=d)
        k_pages = torch.zeros(NP, nkv, P, d, dtype=dtype, device=DEV)
        v_pages = torch.zeros(NP, nkv, P, dv, dtype=dtype, device=DEV)
        full = []
        for r, (b, n) in enumerate(zip(befores, qlens)):
            S = b + n
            k, v, q = _rand(g, S, nkv, d, scale=0.3), _rand(g, S, nkv, dv), _rand(g, S, nq, d, scale=0.3)
            for j in spikes[r]:
                k[j, :, d - 1] = 6.0
            q[:, :, d - 1] = 4.0
            k, v, q = k.to(dtype), v.to(dtype), q.to(dtype)
            scatter_to_pages(k_pages, lay["tables"][r], k, P)
            scatter_to_pages(v_pages, lay["tables"][r], v, P)
            full.append((q.double(), k.double(), v.double()))
        q_new = torch.cat([f[0][b:] for f, b in zip(full, befores)]).to(dtype).to(DEV).contiguous().view(-1, nq * d)
        common = (k_pages, v_pages, lay["block_table"], lay["page_base"])
        T, scale = lay["num_tokens"], 0.5
        starts = np.cumsum([0] + qlens)
        last = None
        for cap in (None, 30.0, 12.0):
            want = []
            for (fq, fk, fv), b in zip(full, befores):
                S = fq.shape[0]
                seen = torch.tril(torch.ones(S, S, dtype=torch.bool))
                s = torch.einsum("ihd,jhd->hij", fq, fk.repeat_interleave(nq // nkv, 1)) * scale
                p = torch.softmax(plain.capped(s, cap).masked_fill(~seen, -math.inf), -1)
                want.append(torch.einsum("hij,jhd->ihd", p, fv.repeat_interleave(nq // nkv, 1))[b:])
            want = torch.cat(want)
            for splits in (1, 3):
                if kernel == "plain":
                    out = o.attention_plain(q_new, nq * d, *common, lay["token_row"], lay["positions"], T, nq, nkv, d, scale, None,
                                            value_dim=dv, softcap=cap)
                else:
                    out = torch.zeros((T, nq * dv), dtype=dtype, device=DEV)
                    step = 128 if kernel == "tc" else 64
                    tiles = torch.tensor([(r, q0) for r, n in enumerate(qlens) if n > 1 for q0 in range(0, n, step)], **i32)
                    fn = o.attention_prefill_tc if kernel == "tc" else o.attention_prefill
                    fn(q_new, nq * d, *common, torch.tensor(starts, **i32), torch.tensor(befores, **i32), tiles, T, nq, nkv, d, scale,
                       None, out=out, softcap=cap)
                    singles = torch.tensor([int(starts[r]) for r, n in enumerate(qlens) if n == 1], **i32)
                    o.attention_decode(q_new, nq * d, *common, lay["token_row"], lay["positions"], T, nq, nkv, d, scale, None, splits,
                                       token_list=singles, out=out, use_tma=False, softcap=cap)
                got = out.float().cpu().view(-1, nq, dv)
                assert (got - want).abs().max() < tol, (kernel, d, cap, splits)
            if last is not None:
                assert (got - last).abs().max() > 0.02
            last = got


@pytest.mark.parametrize("T,N,top", [(1, 5, 2), (9, 5, 2), (40, 12, 1), (3, 7, 7), (128, 64, 6), (129, 33, 3), (700, 8, 4), (5, 300, 2)])
def test_sigmoid_scores_ranking_and_grouping(T, N, top):
    """Scores that are sigmoids of their own logits, chosen by the logits (also where the sigmoids are equal in float32),
    grouped by expert with the weights by slot: the fused kernel of small steps and the two kernels of large ones."""
    o = ops()
    g = torch.Generator().manual_seed(T)
    wide = _rand(g, T, N + 3, scale=2.0)
    wide[0, :N] += 60.0                                  # every sigmoid of this row rounds to one
    z = wide.to(DEV)[:, :N]
    s = torch.sigmoid(wide[:, :N].double())
    best = torch.topk(wide[:, :N], top, dim=-1).indices
    for fused in (True, False):
        if fused:
            idx, wts, offsets, slot_of, slot_token, slot_wts = o.moe_route_plan(z, None, top, 1, 1, scoring="sigmoid", by_slot=True)
        else:
            idx, wts = o.moe_route(z, None, top, 1, 1, scoring="sigmoid")
            offsets, slot_of, slot_token, slot_wts = o.moe_plan(idx, N, wts)
        idx, slot_of, slot_token = idx.cpu().long(), slot_of.cpu().long(), slot_token.cpu().long()
        assert torch.equal(idx, best)
        assert (wts.cpu().double() - s.gather(1, best)).abs().max() < 1e-6
        assert torch.equal(slot_of.flatten().sort().values, torch.arange(T * top))
        assert torch.equal(slot_token[slot_of], torch.arange(T)[:, None].expand(T, top))
        assert torch.equal(slot_wts.cpu()[slot_of], wts.cpu())
        off = offsets.cpu().long()
        assert torch.equal(off[1:] - off[:-1], torch.bincount(idx.flatten(), minlength=N))
        assert bool(((slot_of >= off[idx]) & (slot_of < off[idx + 1])).all())
    # the softmax with a correction and groups, through the fused kernel too
    if N % 4 == 0 and top <= N // 2:
        corr = _rand(g, N).to(DEV)
        a = o.moe_route_plan(z.contiguous(), corr, top, 4, 2, True)
        b = o.moe_route(z.contiguous(), corr, top, 4, 2, True)
        assert torch.equal(a[0], b[0]) and torch.equal(a[1], b[1]) and a[5] is None


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("T,E,top,ff,width", [(5, 4, 2, 16, 24), (40, 3, 1, 40, 64), (90, 2, 2, 33, 30), (130, 2, 1, 64, 96), (600, 2, 1, 72, 128)])
def test_weights_on_the_experts_inputs(T, E, top, ff, width, dtype, tol):
    """A factor per slot on the gate/up product before silu (all tile heights of the mma.sync kernel, the tcgen05 kernel, the
    float32 kernel), and the sum over the choices without weights beside a gated shared row."""
    o = ops()
    g = torch.Generator().manual_seed(T)
    x = _rand(g, T, width, dtype=dtype)
    w = _rand(g, E, 2 * ff, width, dtype=dtype, scale=width ** -0.5)
    idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    wts = torch.rand(T, top, generator=g) * 1.5 + 0.02
    offsets, slot_of, slot_token, slot_wts = o.moe_plan(idx.to(DEV), E, wts.to(DEV))
    got = o.grouped_gemm(x.to(DEV), slot_token, w.to(DEV), offsets, T * top, swiglu_pairs=True, slot_scale=slot_wts).double().cpu()
    flat = o.grouped_gemm(x.to(DEV), slot_token, w.to(DEV), offsets, T * top, slot_scale=slot_wts).double().cpu()
    x64, w64 = x.double(), w.double()
    for t in range(T):
        for k in range(top):
            e, slot = int(idx[t, k]), int(slot_of[t, k])
            both = w64[e] @ (x64[t] * float(wts[t, k]))
            assert (flat[slot] - both).abs().max() < tol * max(1.0, float(both.abs().max()))
            assert (got[slot] - plain.silu(both[0::2]) * both[1::2]).abs().max() < tol * 2
    y, extra, zw = _rand(g, T * top, width, dtype=dtype), _rand(g, T, width, dtype=dtype), _rand(g, T, 4)
    want = y.double()[slot_of.cpu().long()].sum(1) + torch.sigmoid(zw.double()[:, 1:2]) * extra.double()
    out = o.moe_combine(y.to(DEV), x.to(DEV), slot_of, idx.to(DEV), None, E, extra=extra.to(DEV), extra_z=zw.to(DEV)[:, 1:2])
    assert (out.double().cpu() - want).abs().max() < tol * 2
