"""minGRU as a mixer: a gated recurrence whose gates read the current token only.

Per token, with ``z = sigmoid(W_z h + b_z)``, ``u = W_x h + b_x`` (``width`` channels each) and the candidate
``c = u + 1/2`` where ``u >= 0``, ``sigmoid(u)`` elsewhere:  ``S <- (1 - z) S + z c``  channel by channel, and the output
``W_o (S silu(W_g h))``.  The state S is float32, starts at zero and lies in the request's state slot.

One product yields ``[z | u | g]``; biases, gates, recurrence and the output gate are one kernel in float32 (two passes
over segments for long rows: ``ops.min_gru``), then the output product.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import MIXERS, BuildContext, CacheNeeds, Mixer, StateNeeds, TensorSpec

_NAMES = {"z": "z", "z_bias": "z.b", "x": "x", "x_bias": "x.b", "g": "g", "o": "o"}


@MIXERS.register("min_gru")
class MinGRU(Mixer):
    # the one host-side value of the step it reads is its longest row, which is 1 in every step that is captured
    graph_safe = True
    adds_residual = True
    state_base = 0              # where this mixer's part of the request's state vector starts

    def __init__(self, ctx: BuildContext, hidden_size: int, width: int, names: dict | None = None):
        """``names``: the tensors' names relative to the part's prefix (keys z, z_bias, x, x_bias, g, o)."""
        if width < 1:
            raise ValueError(f"width must be >= 1, got {width}")
        self.ctx, self.hidden_size, self.width = ctx, hidden_size, width
        self.names = {**_NAMES, **(names or {})}
        self.w_in = self.w_o = self.bias32 = None

    def tensor_specs(self):
        n, C, W = self.names, self.width, self.hidden_size
        return {n["z"]: TensorSpec((C, W)), n["z_bias"]: TensorSpec((C,), "bias"),
                n["x"]: TensorSpec((C, W)), n["x_bias"]: TensorSpec((C,), "bias"),
                n["g"]: TensorSpec((C, W)), n["o"]: TensorSpec((W, C))}

    def bind(self, tensors):
        n = self.names
        mats = [tensors[n[k]] for k in ("z", "x", "g")]
        dtype = mats[0].dtype if all(m.dtype == mats[0].dtype for m in mats) else torch.float32
        self.w_in = torch.cat([m.to(dtype) for m in mats], dim=0).contiguous()
        self.w_o = tensors[n["o"]].contiguous()
        self.bias32 = torch.cat([tensors[n[k]].to(torch.float32) for k in ("z_bias", "x_bias")]).contiguous()

    def cache_needs(self):
        return CacheNeeds(state=StateNeeds((self.width,)))

    def forward(self, x, inputs, cache, residual32=None):
        proj = ops.linear(x, self.w_in, out_dtype=self.ctx.dtype)
        y = ops.min_gru(proj, self.bias32, cache.state, self.state_base, inputs.row_start, inputs.row_slot, inputs.num_rows,
                        longest_row=inputs.plan.max_q_len)
        return ops.linear(y, self.w_o, out_dtype=self.ctx.dtype, residual32=residual32)
