"""The stream that goes on from a layer run as a weighted sum of the results of all runs so far.

``depth_average``: with X_0 the stream as it enters the first layer and X_(i+1) the result of run i (before any such sum),
what goes on is ``sum over j = 0 .. i + 1 of w_i[j] X_j``: a learned vector of i + 2 numbers per run.  The results and
the sums are float32.  What the run still has to add, the sum and the norms through which the next run reads it are one
kernel (``ops.stream_norm``), which reads every earlier result once.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import STREAM_MIXES, BuildContext, StreamMix, TensorSpec


@STREAM_MIXES.register("depth_average")
class DepthAverage(StreamMix):
    graph_safe = True

    def __init__(self, ctx: BuildContext, names: tuple[str, ...]):
        """``names``: the coefficients' tensor of every run, in the order of the runs."""
        self.ctx, self.names = ctx, tuple(names)
        self.coef32: list[torch.Tensor] = []

    def tensor_specs(self):
        return {name: TensorSpec((i + 2,), "depth_average") for i, name in enumerate(self.names)}

    def bind(self, tensors):
        self.coef32 = [tensors[name].to(torch.float32).contiguous() for name in self.names]

    def open(self, num_tokens, width):
        # the last run's result is read by nobody after its own sum: no entry
        return torch.empty((len(self.names), num_tokens, width), dtype=torch.float32, device=self.ctx.device)

    def forward(self, history, run, x32, delta, norms=(), rows=None, x_out=None):
        specs = tuple(n.stream_spec() for n in norms) if norms and all(hasattr(n, "stream_spec") for n in norms) else ()
        if len(specs) > 2 or len({s[1:] for s in specs}) > 1:
            specs = ()
        if not specs:
            rows = None                      # the norms are the caller's: the whole stream goes on
        out = ops.stream_norm(x32, delta, specs, self.ctx.dtype, rows=rows, history=history, coef32=self.coef32[run], x_out=x_out)
        return (x32 if x_out is None else x_out), (out if specs else None)
