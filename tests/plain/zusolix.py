"""Plain implementation of Zusolix: whole sequences, no cache, float64, one function per mechanism.

It shares no code with the package: it takes the ``config.json`` dictionary and the checkpoint's tensors
by name.  Notation: T tokens, W the width; ``m`` is a mixer's part of the configuration and ``w(name)`` the
tensor ``<layer>.mix.<name>`` (``<layer>.mlp.<name>`` in a feed-forward).
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def grouped_norm(x, w, eps, groups):
    """Each of ``groups`` neighbouring parts of a row over its own root mean square, the row times ``w``."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * w


def depth_average(results, weights):
    """``results``: the streams X_0 (token rows), X_1, ... so far, one weight each."""
    assert len(results) == len(weights)
    total = torch.zeros_like(results[0])
    for x, a in zip(results, weights):
        total = total + a * x
    return total


# ------------------------------------------------------------------ mixers


def query_temperature(positions, temp):
    """The factor on a query at each position: 1 + coef ln(whole spans of ``every`` positions behind it + 1)."""
    if not temp:
        return torch.ones(len(positions), dtype=F64)
    return torch.tensor([1.0 + temp["coef"] * math.log((int(p) + 1) // temp["every"] + 1) for p in positions], dtype=F64)


def capped(scores, cap):
    return scores if not cap else cap * torch.tanh(scores / cap)


def attention(h, m, w):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w("q").T + w("q.b")).view(T, H, d)
    k = (h @ w("k").T + w("k.b")).view(T, G, d)
    v = (h @ w("v").T + w("v.b")).view(T, G, dv)
    q = q * query_temperature(range(T), m.get("q_temp"))[:, None, None]
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = torch.empty(T, H, dv, dtype=F64)
    for i in range(H):
        g = i // (H // G)
        s = capped(q[:, i] @ k[:, g].T * m["scale"], m.get("softcap"))
        s = s.masked_fill(~seen, -math.inf)
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, i] = (p / p.sum(-1, keepdim=True)) @ v[:, g]
    return out.reshape(T, H * dv) @ w("o").T


def candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def gated_recurrence(z, c, s0=None):
    """S_t = (1 - z_t) S_(t-1) + z_t c_t for every t (all states returned), token by token."""
    s = torch.zeros(z.shape[1], dtype=F64) if s0 is None else s0
    out = torch.empty_like(z)
    for t in range(z.shape[0]):
        s = (1.0 - z[t]) * s + z[t] * c[t]
        out[t] = s
    return out


def mingru(h, m, w):
    z = sigmoid(h @ w("z").T + w("z.b"))
    u = h @ w("x").T + w("x.b")
    s = gated_recurrence(z, candidate(u))
    return (s * silu(h @ w("g").T)) @ w("o").T


# ------------------------------------------------------------------ feed-forwards


def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def experts_ff(h, f, w, gaps=None):
    """Sigmoid scores, the ``top`` largest chosen, an expert fed with its score times the row; a shared expert
    times one sigmoid number a token."""
    n, top = f["router"]["experts"], f["router"]["top"]
    z = h @ w("router").T
    s = sigmoid(z)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(n), key=lambda e: (-float(z[t, e]), e))
        if gaps is not None:
            gaps.append(float(z[t, order[top - 1]] - z[t, order[top]]) if top < n else math.inf)
        for e in order[:top]:
            out[t] += gated_ff((s[t, e] * h[t])[None], w(f"e{e}.gate"), w(f"e{e}.up"), w(f"e{e}.down"))[0]
    if f.get("shared"):
        out = out + gated_ff(h, w("shared.gate"), w("shared.up"), w("shared.down")) * sigmoid(h @ w("shared.sg").T)
    return out


# ------------------------------------------------------------------ the model


def forward(cfg, weights, tokens, every_layer=None, router_gaps=None):
    """float64 logits [T, vocab].  ``every_layer``: a list that receives the stream after every layer (averaged);
    ``router_gaps``: a list that receives, per routed layer, how far the last chosen expert's router logit lies above the
    first one left out, per token."""
    def tensor(name):
        return weights[name].to(F64)

    eps, groups = cfg["norm"]["eps"], cfg["norm"].get("groups", 1)
    x = tensor("embed")[torch.as_tensor(tokens, dtype=torch.long)] * cfg.get("embedding", {}).get("scale", 1.0)
    results = [x]
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        mix = {"attention": attention, "mingru": mingru}[layer["type"]]
        y = mix(grouped_norm(x, tensor(pre + "norm1"), eps, groups), layer["mixer"], lambda n: tensor(pre + "mix." + n))
        f = layer.get("mlp")
        if f is not None:
            h = grouped_norm(x, tensor(pre + "norm2"), eps, groups)
            w = lambda n: tensor(pre + "mlp." + n)
            if f.get("kind", "dense") == "dense":
                y = y + gated_ff(h, w("gate"), w("up"), w("down"))
            else:
                gaps = None
                if router_gaps is not None:
                    router_gaps.append([])
                    gaps = router_gaps[-1]
                y = y + experts_ff(h, f, w, gaps)
        results.append(x + cfg.get("residual_mult", 1.0) * y)
        x = depth_average(results, tensor(pre + "dwa"))
        if every_layer is not None:
            every_layer.append(x)
    return grouped_norm(x, tensor("final.norm"), eps, groups) @ tensor("head").T
