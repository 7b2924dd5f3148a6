"""A routed mixture of small SwiGLU experts, some of which are the identity, as a feed-forward.

Router logits ``z = W_router h`` over ``experts + identity`` outputs, in float32; scores
``s = softmax(z)``; experts are ranked by ``s + correction``.  Neighbouring outputs form ``groups`` groups of
equal size; a group is ranked by the best ranking value inside it, and outputs outside the ``keep`` best
groups are out of the running whatever their value.  The ``top`` best-ranked outputs are taken, each
weighted by its own ``s`` (the correction only ranks; the weights are left as they are, not rescaled to
sum to one).  The last ``identity`` outputs own no tensors and pass their input through.  A real expert is ``down(silu(gate h) * (up h))``.  The result is the weighted
sum over the chosen.

Options: no correction (``correction`` false: experts are ranked by their scores alone); the chosen outputs'
scores divided by their sum (``normalize``); experts of the capped form (``activation="capped_swish"`` with
``limit`` L: ``g = min(gate h, L), u = clamp(up h, -L, L), down(g sigmoid(1.702 g) (u + 1))``); a shared expert of
the same form (``shared_size``, ``shared_limit``; tensors ``shared.gate`` / ``up`` / ``down``) that every token
takes, added to the weighted sum; scores ``sigmoid(z)`` of each output instead of the softmax (``scoring="sigmoid"``);
the chosen outputs' weights on the experts' *inputs* instead of their outputs (``weight_on="input"``: the sum over the
chosen of ``expert(s h)``); the shared expert's result times ``sigmoid(W_sg h)``, one number per token (``shared_gate``;
tensor ``shared.sg``); a bias per output on the router's logits (``router_bias``; tensor ``router.b``).

On the device: the router's choice and the (token, choice) pairs grouped by expert (a kernel each, one for both in
steps of few tokens), one product per expert over its own rows for gate/up (SwiGLU in its epilogue on the tensor-core
kernel) and for down (a kernel each, walking the per-expert offsets on the device: nothing of the routing
is read on the host), and the weighted sum in the order of the choices, which also norms the result and
adds it to the stream when the block asks.  A weight on an expert's input is a factor on its gate/up product's float32 sums
(the product is linear), in that product's epilogue; the sum over the choices then has no weights, and can be left to the
kernel that adds the layer's results to the stream (``forward(..., defer=True)``).  The shared expert's gate row rides in
the router's product.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import FEED_FORWARDS, BuildContext, FeedForward, TensorSpec
from .feed_forward import SwiGLU


@FEED_FORWARDS.register("routed_experts")
class RoutedExperts(FeedForward):
    graph_safe = True

    def __init__(self, ctx: BuildContext, hidden_size: int, expert_size: int, num_experts: int, num_identity: int,
                 top: int, groups: int = 1, keep: int = 1, correction: bool = True, normalize: bool = False,
                 activation: str = "silu", limit: float = 0.0, shared_size: int | None = None,
                 shared_limit: float | None = None, scoring: str = "softmax", weight_on: str = "output",
                 shared_gate: bool = False, router_bias: bool = False):
        if scoring not in ops.MOE_SCORINGS:
            raise ValueError(f"scoring must be one of {sorted(ops.MOE_SCORINGS)}, got {scoring!r}")
        if weight_on not in ("output", "input") or (weight_on == "input" and (num_identity or num_experts < 1)):
            raise ValueError("weight_on must be 'output' or 'input', the latter without identity experts")
        if shared_gate and not shared_size:
            raise ValueError("shared_gate needs a shared expert")
        self.scoring, self.weight_on, self.shared_gate = scoring, weight_on, bool(shared_gate)
        self.router_bias, self.bias32 = bool(router_bias), None
        self.defers = weight_on == "input"      # ``forward(..., defer=True)`` leaves the sum over the choices undone
        self.defers_weighted = weight_on == "output" and not num_identity and num_experts > 0 and not shared_gate   # ... with its weights
        if activation not in ("silu", "capped_swish"):
            raise ValueError(f"expert activation must be 'silu' or 'capped_swish', got {activation!r}")
        self.correction, self.normalize, self.activation, self.limit = bool(correction), bool(normalize), activation, float(limit)
        self.shared_size, self.shared_limit = shared_size, float(shared_limit if shared_limit is not None else limit)
        # a shared expert is a gated feed-forward like any other
        self.shared_ff = SwiGLU(ctx, hidden_size, shared_size, activation, {"gate": "gate", "up": "up", "down": "down"},
                                limit=self.shared_limit) if shared_size else None
        n = num_experts + num_identity
        if n < 1 or n % groups or not (1 <= keep <= groups) or top > keep * (n // groups):
            raise ValueError(f"{n} router outputs do not split into {groups} groups of which {keep} hold {top} choices")
        self.ctx = ctx
        self.hidden_size, self.ff = hidden_size, expert_size
        self.E, self.I, self.top, self.groups, self.keep = num_experts, num_identity, top, groups, keep
        self.w_router = self.correction32 = self.w_gate_up = self.w_down = None

    def tensor_specs(self):
        n = self.E + self.I
        specs = {"router": TensorSpec((n, self.hidden_size))}
        if self.correction:
            specs["correction"] = TensorSpec((n,), "bias")
        if self.router_bias:
            specs["router.b"] = TensorSpec((n,), "bias")
        if self.shared_gate:
            specs["shared.sg"] = TensorSpec((1, self.hidden_size))
        if self.shared_size:
            specs["shared.gate"] = TensorSpec((self.shared_size, self.hidden_size))
            specs["shared.up"] = TensorSpec((self.shared_size, self.hidden_size))
            specs["shared.down"] = TensorSpec((self.hidden_size, self.shared_size))
        for e in range(self.E):
            specs[f"e{e}.gate"] = TensorSpec((self.ff, self.hidden_size))
            specs[f"e{e}.up"] = TensorSpec((self.ff, self.hidden_size))
            specs[f"e{e}.down"] = TensorSpec((self.hidden_size, self.ff))
        return specs

    def bind(self, tensors):
        t = tensors
        # Under a bfloat16 engine the router's matrix stays as stored: a product of two bfloat16 numbers is
        # exact in float32, so the tensor-core product with float32 accumulation is the float32 computation
        # on the rounded input, up to the order of the sum.
        self.w_router = t["router"].contiguous()
        if self.shared_gate:                       # one more row of the router's product: [router | shared gate]
            sg = t["shared.sg"]
            dtype = sg.dtype if sg.dtype == self.w_router.dtype else torch.float32
            self.w_router = torch.cat([self.w_router.to(dtype), sg.to(dtype)], dim=0).contiguous()
        self.correction32 = t["correction"].to(torch.float32).contiguous() if self.correction else None
        self.bias32 = t["router.b"].to(torch.float32).contiguous() if self.router_bias else None
        if self.shared_ff is not None:
            self.shared_ff.bind({n: t["shared." + n] for n in ("gate", "up", "down")})
        if self.E:
            mats = [t[f"e{e}.{n}"] for e in range(self.E) for n in ("gate", "up", "down")]
            dtype = mats[0].dtype if all(m.dtype == mats[0].dtype for m in mats) else torch.float32
            # gate and up rows in turns (row 2i: gate of output i, row 2i + 1: its up row): a thread of the grouped
            # product's epilogue then holds both and applies SwiGLU itself
            self.w_gate_up = torch.stack([torch.stack([t[f"e{e}.gate"].to(dtype), t[f"e{e}.up"].to(dtype)], dim=1)
                                          .reshape(2 * self.ff, self.hidden_size) for e in range(self.E)]).contiguous()
            self.w_down = torch.stack([t[f"e{e}.down"].to(dtype) for e in range(self.E)]).contiguous()   # [E, width, ff]

    adds_normed_residual = True     # ``forward(..., add_normed=(resid32, norm))`` adds the normed result to the stream itself

    def forward(self, x, inputs, add_normed=None, defer=False):
        T, n = x.shape[0], self.E + self.I
        beside = ops.Branch(lambda: self.shared_ff.forward(x, inputs), inputs) if self.shared_ff is not None else None
        z = ops.linear(x, self.w_router, out_dtype=torch.float32)
        idx, wts, offsets, slot_of, slot_token, slot_wts = ops.moe_route_plan(
            z[:, :n], self.correction32, self.top, self.groups, self.keep, self.normalize, self.scoring,
            by_slot=self.weight_on == "input", bias32=self.bias32)
        if self.weight_on == "input":
            wts = None                       # the weights go in with the rows: the choices are summed as they are
        slots = T * self.top
        if self.E:
            w_gu = self.w_gate_up if self.w_gate_up.dtype == x.dtype else self.w_gate_up.to(x.dtype)
            w_dn = self.w_down if self.w_down.dtype == x.dtype else self.w_down.to(x.dtype)
            hidden = ops.grouped_gemm(x, slot_token, w_gu, offsets, slots, swiglu_pairs=True, activation=self.activation,
                                      limit=self.limit, slot_scale=slot_wts)
            y = ops.grouped_gemm(hidden, None, w_dn, offsets, slots)
        else:
            y = x
        shared = beside.join() if beside is not None else None
        shared_z = z[:, n:n + 1] if self.shared_gate else None
        if defer and (self.defers or self.defers_weighted):
            return ops.ExpertsPending(y, slot_of, shared, shared_z, wts)
        if add_normed is not None:
            resid32, norm = add_normed
            return ops.moe_combine(y, x, slot_of, idx, wts, self.E, resid32=resid32, weight32=norm.weight32, eps=norm.eps,
                                   extra=shared, extra_z=shared_z)
        return ops.moe_combine(y, x, slot_of, idx, wts, self.E, extra=shared, extra_z=shared_z)
