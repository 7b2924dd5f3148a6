"""Plain implementation of Badepel: whole sequences, no cache, float64, one function per mechanism.

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


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return over_rms(x, eps) * w


def short_conv(u, taps):
    """u [T, C], taps [C, n]: y_t = sum_j taps[:, j] u_(t - n + 1 + j), zeros before the first row."""
    T, n = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            y[back:] += taps[:, j] * u[:T - back]
    return y


# ------------------------------------------------------------------ attention


def rotate_neighbours(x, rot):
    """x [T, heads, d]: pairs (2i, 2i + 1) of the first ``dims`` entries turned by position times base^(-2i / dims)."""
    if not rot or not rot["dims"]:
        return x
    n = rot["dims"]
    freq = torch.tensor([rot["base"] ** (-2.0 * i / n) for i in range(n // 2)], dtype=F64)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * freq
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    y = x.clone()
    a, b = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2] = a * c - b * s
    y[..., 1:n:2] = b * c + a * s
    return y


def visible(T, window):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if window is None else ok & (i - j < window)


def softmax_plus_one(s, ok):
    """exp(s_j) / (1 + sum exp(s)) over the visible keys of each row."""
    s = s.masked_fill(~ok, -math.inf)
    top = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention_rows(h, m, w, eps):
    """The heads' outputs side by side, before the output projection."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    u = {n: h @ w(n).T + w(n + ".b") for n in "qkv"}
    if m.get("conv"):
        u = {n: short_conv(x, w(n + ".conv")) for n, x in u.items()}
    q = rotate_neighbours(rms_norm(u["q"], w("q.norm"), eps).view(T, H, d), m.get("rot"))
    k = rotate_neighbours(rms_norm(u["k"], w("k.norm"), eps).view(T, G, d), m.get("rot"))
    v = u["v"].view(T, G, dv)
    ok = visible(T, (m.get("mask") or {}).get("size"))
    out = torch.empty(T, H, dv, dtype=F64)
    for i in range(H):
        g = i // (H // G)
        s = q[:, i] @ k[:, g].T * m["scale"]
        if m.get("softcap"):
            s = m["softcap"] * torch.tanh(s / m["softcap"])
        out[:, i] = softmax_plus_one(s, ok) @ v[:, g]
    return out.reshape(T, H * dv)


# ------------------------------------------------------------------ recurrences


def gla_recurrence(q, k, v, alpha, s0=None):
    """q, k, alpha [T, H, d], v [T, H, dv]; S <- diag(alpha) S + k v^T; o = S^T q.  Returns o and the last S."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if s0 is None else s0.clone()
    out = torch.empty(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def gla_rows(h, m, w, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w("q").T).view(T, H, d) * d ** -0.5
    k = (h @ w("k").T).view(T, H, d)
    v = (h @ w("v").T).view(T, H, dv)
    z = (h @ w("a1").T) @ w("a2").T + w("a2.b")
    alpha = torch.exp(-softplus(-z) / m["tau"]).view(T, H, d)
    o, _ = gla_recurrence(q, k, v, alpha)
    return rms_norm(o, w("norm"), eps).reshape(T, H * dv) * silu(h @ w("g").T)


def delta_recurrence(q, k, v, beta, g, s0=None):
    """q, k [T, H, d], v [T, H, dv], beta, g [T, H]; S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if s0 is None else s0.clone()
    out = torch.empty(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta(h, m, w, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    u = {}
    for n in "qkv":
        x = h @ w(n).T
        u[n] = silu(short_conv(x, w(n + ".conv"))) if m.get("conv") else silu(x)
    group = torch.arange(H) // (H // G)
    q = (unit(u["q"].view(T, G, d)) * d ** -0.5)[:, group]
    k = unit(u["k"].view(T, G, d))[:, group]
    v = u["v"].view(T, H, dv)
    beta = sigmoid(h @ w("b").T)
    g = torch.exp(-torch.exp(w("A_log")) * softplus(h @ w("a").T + w("dt_bias")))
    o, _ = delta_recurrence(q, k, v, beta, g)
    o = rms_norm(o, w("norm"), eps) * silu(h @ w("g").T).view(T, H, dv)
    return o.reshape(T, H * dv) @ w("o").T


def parallel(h, m, w, eps):
    left, right = (lambda n: w("left." + n)), (lambda n: w("right." + n))
    a = attention_rows(h, m["left"], left, eps) @ left("o").T
    b = gla_rows(h, m["right"], right, eps) @ right("o").T
    return m["left_scale"] * a + m["right_scale"] * b


MIXERS = {"delta": delta, "parallel": parallel}


# ------------------------------------------------------------------ feed-forwards


def gated_ff(h, w):
    return (silu(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


def capped_expert(h, w, prefix, limit):
    g = (h @ w(prefix + "gate").T).clamp(max=limit)
    u = (h @ w(prefix + "up").T).clamp(min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w(prefix + "down").T


def experts_ff(h, f, w, gaps=None):
    """The ``top`` largest router logits (bias and all), weighted by the softmax over those alone, beside a shared expert."""
    n, top = f["router"]["experts"], f["router"]["top"]
    z = h @ w("router").T + w("router.b")
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(n), key=lambda e: (-float(z[t, e]), e))
        if gaps is not None:
            gaps.append(float(z[t, order[top - 1]] - z[t, order[top]]) if top < n else math.inf)
        chosen = order[:top]
        p = torch.exp(z[t, chosen] - z[t, chosen].max())
        p = p / p.sum()
        for share, e in zip(p, chosen):
            out[t] += share * capped_expert(h[t:t + 1], w, f"e{e}.", f["expert"]["limit"])[0]
    if f.get("shared"):
        out = out + capped_expert(h, w, "shared.", f["shared"]["limit"])
    return out


# ------------------------------------------------------------------ the model


def read_streams(xs, coef):
    return sum(c * x for c, x in zip(coef, xs))


def write_streams(xs, mix, out, y):
    """x_t <- sum_s mix[s, t] x_s + out[t] y, all from the old streams."""
    n = len(xs)
    return [sum(mix[s, t] * xs[s] for s in range(n)) + out[t] * y for t in range(n)]


def forward(cfg, weights, tokens, every_layer=None, router_gaps=None):
    """float64 logits [T, vocab].  ``every_layer``: a list that receives the sum of the streams after every layer;
    ``router_gaps``: a list that receives, per routed layer, how far the last chosen expert's router logit lies above the
    first one left out, per token."""
    def tensor(name):
        return weights[name].to(F64)

    eps, m, n = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0), cfg.get("streams")
    x = tensor("embed")[torch.as_tensor(tokens, dtype=torch.long)]
    xs = [x] * (n or 1)

    def sublayer(xs, pre, q, fn):
        if n is None:
            return [xs[0] + m * fn(rms_norm(xs[0], tensor(f"{pre}norm{q}"), eps))]
        hc = lambda name: tensor(f"{pre}hc{q}.{name}")
        y = fn(rms_norm(read_streams(xs, hc("in")), tensor(f"{pre}norm{q}"), eps))
        return write_streams(xs, hc("mix"), m * hc("out"), y)

    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        xs = sublayer(xs, pre, 1, lambda h: MIXERS[layer["type"]](h, layer["mixer"], lambda k: tensor(pre + "mix." + k), eps))
        f = layer.get("mlp")
        if f is not None:
            w = lambda k: tensor(pre + "mlp." + k)
            if f.get("kind", "dense") == "dense":
                xs = sublayer(xs, pre, 2, lambda h: gated_ff(h, w))
            else:
                gaps = None
                if router_gaps is not None:
                    router_gaps.append([])
                    gaps = router_gaps[-1]
                xs = sublayer(xs, pre, 2, lambda h: experts_ff(h, f, w, gaps))
        if every_layer is not None:
            every_layer.append(sum(xs))
    return rms_norm(sum(xs), tensor("final.norm"), eps) @ tensor("head").T
