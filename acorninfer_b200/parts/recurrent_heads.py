"""Recurrent mixers whose per-request state is a float32 matrix per head, with the same ending: every head's read-out over
its root mean square, times one weight of head size, times silu of a gate, and the output projection.

``head_delta`` (a gated delta rule with one decay per head).  Per token, from the mixer's input h:
  q, k (kv_heads x dim) and v (heads x vdim): projections, a short causal convolution over time per channel (``taps``
  weights, the last for the current token, zeros before a request's start), silu; q and k scaled to unit length per head
  (``x / sqrt(sum x^2 + 1e-6)``), q further by ``dim^-1/2``; head a uses q/k head ``a // (heads / kv_heads)``.
  beta = sigmoid(W_b h) and g = exp(-exp(A_log) softplus(W_a h + dt_bias)), one number per head each.
  Per head:  S = g S;  u = beta (v - S^T k);  S = S + k u^T;  o = S^T q.

``gated_linear_attention``.  q = dim^-1/2 W_q h, k = W_k h (heads x dim), v = W_v h (heads x vdim); a decay per head and key
  channel, ``alpha = sigmoid(W_a2 W_a1 h + bias)^(1 / tau)``.  Per head:  S = diag(alpha) S + k v^T;  o = S^T q.

Everything from the activations (the projections of the second) on is float32, and so is the state: S of every head, and
behind it the convolution's last ``taps - 1`` inputs, in the request's slot (one float32 vector from ``state_base`` on).
All projections of h are one matrix product.  Steps of single tokens run recurrence, norm and gate in one kernel
(``ops.recurrent_step``); steps with rows of ``ops.DELTA_CHUNK_MIN_ROW`` tokens run over chunks of tokens (``ops.delta_chunk``,
``ops.linear_chunk``); others walk their rows' tokens.  The one host-side value of a step that is
read is its longest row, which is 1 in every captured step.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import MIXERS, BuildContext, CacheNeeds, Mixer, StateNeeds, TensorSpec


def _up(n: int, to: int) -> int:
    return -(-n // to) * to


def stack_rows(mats, starts, dtype) -> torch.Tensor:
    """The matrices' rows at the given first rows of one matrix, zero rows between them and up to a multiple of 8."""
    n = _up(max(s + m.shape[0] for m, s in zip(mats, starts)), 8)
    w = torch.zeros((n, mats[0].shape[1]), dtype=dtype, device=mats[0].device)
    for m, s in zip(mats, starts):
        w[s:s + m.shape[0]] = m.to(dtype)
    return w


class _HeadsMixer(Mixer):
    graph_safe = True
    state_base = 0
    w_in = w_o = None

    def cache_needs(self):
        return CacheNeeds(state=StateNeeds((self.state_size(),)))

    def _bind_common(self, tensors, names, starts):
        mats = [tensors[n] for n in names]
        dtype = mats[0].dtype if all(m.dtype == mats[0].dtype for m in mats) else torch.float32
        self.w_in = stack_rows(mats, starts, dtype)
        self.w_o = tensors["o"].contiguous()
        self.norm32 = tensors["norm"].to(torch.float32).contiguous()
        self.norm_heads32 = self.norm32.repeat(self.H).contiguous()           # the same for the kernel that norms rows of heads

    def forward(self, x, inputs, cache):
        return ops.linear(self.inner(x, inputs, cache), self.w_o, out_dtype=self.ctx.dtype)

    def inner(self, x, inputs, cache, out_scale: float = 1.0, out=None, proj=None):
        """The heads' rows before the output projection, times ``out_scale``, into ``out`` if given; ``proj``: the rows of
        ``w_in``'s product where the caller has made it (beside another mixer's)."""
        if proj is None:
            proj = ops.linear(x, self.w_in, out_dtype=self.ctx.dtype)
        if out is None:
            out = torch.empty((proj.shape[0], self.H * self.vdim), dtype=self.ctx.dtype, device=proj.device)
        return self._run(proj, inputs, cache, out_scale, out)

    def _steps(self, inputs, cache, rows) -> bool:
        return inputs.plan.all_decode and ops.recurrent_step_ok(
            self.dim, self.vdim, (cache.state, cache.state.stride(0), self.state_base), rows)


@MIXERS.register("head_delta")
class HeadDelta(_HeadsMixer):
    def __init__(self, ctx: BuildContext, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, norm_eps: float,
                 taps: int | None = None):
        if num_heads % num_kv_heads:
            raise ValueError(f"num_heads ({num_heads}) must be a multiple of num_kv_heads ({num_kv_heads})")
        self.ctx, self.hidden_size, self.eps = ctx, hidden_size, float(norm_eps)
        self.H, self.KH, self.dim, self.vdim, self.taps = num_heads, num_kv_heads, dim, vdim, taps
        self.channels = 2 * num_kv_heads * dim + num_heads * vdim
        self.conv_off = _up(num_heads * dim * vdim, 4)                # the convolution's memory, behind S
        # columns of the projected row: [q | k | v | gate | beta | decay]
        self.gate_col = _up(self.channels, 8)
        self.beta_col = _up(self.gate_col + num_heads * vdim, 8)
        self.decay_col = self.beta_col + num_heads
        self.conv32 = None

    def tensor_specs(self):
        H, KH, d, v, W = self.H, self.KH, self.dim, self.vdim, self.hidden_size
        specs = {"q": TensorSpec((KH * d, W)), "k": TensorSpec((KH * d, W)), "v": TensorSpec((H * v, W)),
                 "b": TensorSpec((H, W)), "a": TensorSpec((H, W)), "g": TensorSpec((H * v, W)),
                 "A_log": TensorSpec((H,), "decay_log"), "dt_bias": TensorSpec((H,), "bias"),
                 "norm": TensorSpec((v,), "norm"), "o": TensorSpec((W, H * v))}
        if self.taps:
            specs.update({n + ".conv": TensorSpec((specs[n].shape[0], self.taps), "conv") for n in ("q", "k", "v")})
        return specs

    def bind(self, tensors):
        f32 = lambda x: x.to(torch.float32).contiguous()
        kd = self.KH * self.dim
        self._bind_common(tensors, ("q", "k", "v", "g", "b", "a"),
                          (0, kd, 2 * kd, self.gate_col, self.beta_col, self.decay_col))
        self.a_log32, self.dt_bias32 = f32(tensors["A_log"]), f32(tensors["dt_bias"])
        if self.taps:
            self.conv32 = f32(torch.cat([tensors[n + ".conv"] for n in ("q", "k", "v")], dim=0))

    def state_size(self) -> int:
        return _up(self.conv_off + (self.taps - 1) * self.channels if self.taps else self.conv_off, 4)

    def _run(self, proj, inputs, cache, out_scale, out):
        conv_off = self.state_base + self.conv_off
        ins = ops.delta_heads_prep(proj, self.beta_col, self.decay_col, self.conv32, cache.state, conv_off, self.a_log32,
                                   self.dt_bias32, inputs.token_row, inputs.row_start, inputs.row_slot, self.H, self.KH, self.dim,
                                   self.vdim, update_single=True)
        if self.taps and self.taps > 1 and inputs.plan.max_q_len > 1:      # rows of one token shifted their memory above
            ops.conv_state_update(proj, cache.state, conv_off, inputs.row_start, inputs.row_slot, inputs.num_rows,
                                  self.channels, self.taps, skip_single=True)
        gate = proj[:, self.gate_col:self.gate_col + self.H * self.vdim]
        if self._steps(inputs, cache, (gate, out)):
            return ops.recurrent_step(cache.state, self.state_base, inputs.row_slot, gate, self.norm32, self.eps, out, self.H,
                                      self.dim, self.vdim, out_scale, delta=ins)
        q, k, v, beta, g, log_g = ins
        o = ops.delta_rule(q, k, v, beta, g, cache.state, inputs.row_start, inputs.row_slot, inputs.num_rows,
                           longest_row=inputs.plan.max_q_len, state_off=self.state_base, log_g=log_g)
        return ops.gated_norm(o.view(o.shape[0], -1), gate, self.norm_heads32, self.eps, self.H, False, out, out_scale, silu=True)


@MIXERS.register("gated_linear_attention")
class GatedLinearAttention(_HeadsMixer):
    def __init__(self, ctx: BuildContext, hidden_size: int, num_heads: int, dim: int, vdim: int, tau: float, norm_eps: float,
                 decay_rank: int | None = None):
        """``decay_rank``: inner size of the decay's low-rank projection; None: taken from the checkpoint's
        tensors (give it when writing a model)."""
        if not tau > 0:
            raise ValueError(f"tau must be > 0, got {tau}")
        self.ctx, self.hidden_size, self.eps, self.tau = ctx, hidden_size, float(norm_eps), float(tau)
        self.H, self.dim, self.vdim, self.decay_rank = num_heads, dim, vdim, decay_rank
        # columns of the projected row: [q | k | v | gate | a1]
        self.gate_col = _up(num_heads * (2 * dim + vdim), 8)
        self.a1_col = _up(self.gate_col + num_heads * vdim, 8)

    def tensor_specs(self):
        H, d, v, W, r = self.H, self.dim, self.vdim, self.hidden_size, self.decay_rank
        return {"q": TensorSpec((H * d, W)), "k": TensorSpec((H * d, W)), "v": TensorSpec((H * v, W)), "g": TensorSpec((H * v, W)),
                "a1": TensorSpec((r, W)), "a2": TensorSpec((H * d, r)), "a2.b": TensorSpec((H * d,), "bias"),
                "norm": TensorSpec((v,), "norm"), "o": TensorSpec((W, H * v))}

    def bind(self, tensors):
        Hd = self.H * self.dim
        self._bind_common(tensors, ("q", "k", "v", "g", "a1"), (0, Hd, 2 * Hd, self.gate_col, self.a1_col))
        self.rank = tensors["a1"].shape[0]
        self.w_a2 = tensors["a2"].contiguous()
        self.a2_bias32 = tensors["a2.b"].to(torch.float32).contiguous()

    def state_size(self) -> int:
        return _up(self.H * self.dim * self.vdim, 4)

    def _run(self, proj, inputs, cache, out_scale, out):
        low = proj[:, self.a1_col:self.a1_col + self.rank]
        z = ops.linear(low if low.dtype == self.w_a2.dtype else low.contiguous(), self.w_a2, out_dtype=torch.float32)
        gate = proj[:, self.gate_col:self.gate_col + self.H * self.vdim]
        if self._steps(inputs, cache, (proj, gate, out)) and (self.H * self.dim) % 2 == 0 and z.stride(0) % 4 == 0:
            return ops.recurrent_step(cache.state, self.state_base, inputs.row_slot, gate, self.norm32, self.eps, out, self.H,
                                      self.dim, self.vdim, out_scale, linear=(proj, z, self.a2_bias32, self.tau))
        longest = inputs.plan.max_q_len
        if ops.linear_chunk_ok(longest, proj, z, cache.state, self.state_base, inputs.num_rows, self.H, self.dim, self.vdim):
            o = ops.linear_chunk(proj, z, self.a2_bias32, self.tau, cache.state, inputs.row_start, inputs.row_slot, inputs.num_rows,
                                 self.H, self.dim, self.vdim, state_off=self.state_base)
        else:
            q, k, v, alpha = ops.linear_heads_prep(proj, z, self.a2_bias32, self.tau, self.H, self.dim, self.vdim)
            o = ops.delta_rule(q, k, v, None, alpha, cache.state, inputs.row_start, inputs.row_slot, inputs.num_rows,
                               longest_row=longest, state_off=self.state_base)
        return ops.gated_norm(o.view(o.shape[0], -1), gate, self.norm_heads32, self.eps, self.H, False, out, out_scale, silu=True)
