"""A plain, slow implementation of the Midisun design, one function per mechanism, in torch on the CPU.

It takes a configuration in config.json's form and a dict of tensors by checkpoint name, and shares no code with the library: every
request is computed alone, with full keys and values, one token after the other where the design has a recurrence. ``dtype`` is the
arithmetic's type (float64 by default: the oracle of the tests).

In this file's notation, x the residual stream and N(y) = y / sqrt(mean(y^2) + eps):

* x0 = scale E[token]; a layer: u = G(x; w1), x += mixer(u + conv(u)) * sigmoid(R1 u + b1); u = G(x; w2), x += ff(u) * sigmoid(R2 u + b2)
  (a layer may have no ff), G: N over each of ``groups`` equal parts of the row, then times w; logits = Whead G(x; w_final).
* attention: q = N(Wq h + bq) w_q, k = N(Wk h + bk) w_k over whole rows, v = Wk h + bk; a score is t = scale q.k, then
  cap tanh(t / cap), then - slope_head (i - j); keys 0 <= i - j < size; the softmax's denominator has exp(sink_head) as well; the head's
  output times sigmoid(Wg h)_head; Wo . + bo.
* retention: S <- decay_head S + k v^T, o = S^T q, q and k rotated, k times dim^-1/2; Wo (N(o per head) * silu(Wg h)).
* mlstm: i = cap tanh((Wi h + bi) / cap), f = log sigmoid(cap tanh((Wf h + bf) / cap)), m' = max(f + m, i), S <- e^(f + m - m') S +
  e^(i - m') k v^T, n likewise with k; o = S^T q / (max(|n.q|, e^(-m')) + 1e-6), q times dim^-1/2; Wo (N(o per head) * w * sigmoid(Wg h)).
* routed ff: s = sigmoid(Wr u), c = s + correction; a group's score is the sum of its two largest c; of the members of the best groups
  the ``top`` largest c; weights s / (sum of the chosen s + 1e-20); a unit is Wdown (silu(Wgate u) * Wup u).
"""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------- small pieces
def rms_divide(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, w, groups, eps):
    """The row in ``groups`` equal parts, each divided by its own root mean square, the whole times w."""
    parts = x.view(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms_divide(parts, eps).reshape(x.shape) * w


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(u, c):
    """u [t, channels], c [channels, taps]: y_t = sum_j c[:, j] u_(t - taps + 1 + j), zeros before the start."""
    t, taps = u.shape[0], c.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], 0)
    return sum(c[:, j] * padded[j:j + t] for j in range(taps))


def rotate(x, positions, dims, base):
    """x [t, heads, dim]: the first ``dims`` elements of every head, element i paired with i + dims / 2."""
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = positions.to(torch.float64)[:, None] * f[None, :]
    cos, sin = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


# ---------------------------------------------------------------- mixers
def attention(h, w, p, m, eps):
    t = h.shape[0]
    H, G, D = m["heads"], m.get("kv_heads") or m["heads"], m["dim"]
    q = h @ w[p + "q"].T + w[p + "q.b"]
    k = h @ w[p + "k"].T + w[p + "k.b"]
    v = k.view(t, G, D)                                            # the projection as it is, before the norm
    q = (rms_divide(q, eps) * w[p + "q.norm"]).view(t, H, D)
    k = (rms_divide(k, eps) * w[p + "k.norm"]).view(t, G, D)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    i = torch.arange(t)
    distance = i[:, None] - i[None, :]
    visible = distance >= 0
    size = (m.get("mask") or {}).get("size")
    if size:
        visible &= distance < size
    cap = m.get("softcap")
    out = []
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"]
        if cap:
            s = cap * torch.tanh(s / cap)
        s = (s - slopes(H)[a] * distance).masked_fill(~visible, -math.inf)
        sink = w[p + "sink"][a]
        top = torch.maximum(s.max(-1).values, sink)
        e = torch.exp(s - top[:, None])
        o = (e / (e.sum(-1) + torch.exp(sink - top))[:, None]) @ v[:, g]
        out.append(o * gate[:, a:a + 1])
    return torch.cat(out, -1) @ w[p + "o"].T + w[p + "o.b"]


def retention(h, w, p, m, eps):
    t = h.shape[0]
    H, D, V = m["heads"], m["dim"], m.get("vdim") or m["dim"]
    q, k = (h @ w[p + "q"].T).view(t, H, D), (h @ w[p + "k"].T).view(t, H, D)
    v = (h @ w[p + "v"].T).view(t, H, V)
    rot, pos = m.get("rot"), torch.arange(t)
    if rot:
        q, k = rotate(q, pos, rot["dims"], rot["base"]), rotate(k, pos, rot["dims"], rot["base"])
    k = k * D ** -0.5
    decay = torch.tensor(m["decay"], dtype=h.dtype)[:, None, None]
    S = torch.zeros(H, D, V, dtype=h.dtype)
    o = torch.zeros(t, H, V, dtype=h.dtype)
    for i in range(t):
        S = decay * S + k[i][:, :, None] * v[i][:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", S, q[i])
    return (rms_divide(o, eps).reshape(t, H * V) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mlstm_cell(q, k, v, ig, fg):
    """q, k [t, heads, dim], v [t, heads, vdim], log gates ig, fg [t, heads]; returns o [t, heads, vdim], not yet normed."""
    t, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    n = torch.zeros(H, D, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    o = torch.zeros_like(v)
    for i in range(t):
        m_new = torch.maximum(fg[i] + m, ig[i])
        keep, add = torch.exp(fg[i] + m - m_new), torch.exp(ig[i] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[i][:, :, None] * v[i][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[i]
        m = m_new
        den = torch.maximum((n * q[i]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[i] = torch.einsum("hdv,hd->hv", S, q[i]) / den[:, None]
    return o


def mlstm(h, w, p, m, eps):
    t = h.shape[0]
    H, D, V, cap = m["heads"], m["dim"], m.get("vdim") or m["dim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(t, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(t, H, D)
    v = (h @ w[p + "v"].T).view(t, H, V)
    soft = lambda name: cap * torch.tanh((h @ w[p + name].T + w[p + name + ".b"]) / cap)
    o = mlstm_cell(q, k, v, soft("i"), torch.nn.functional.logsigmoid(soft("f")))
    return (rms_divide(o, eps).reshape(t, H * V) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"attention": attention, "retention": retention, "mlstm": mlstm}


# ---------------------------------------------------------------- feed-forward
def unit(u, w, p):
    return (silu(u @ w[p + "gate"].T) * (u @ w[p + "up"].T)) @ w[p + "down"].T


def choose(z, correction, top, groups=None):
    """(chosen [t, top], margin [t]): the margin is the smallest gap on which the choice of groups and experts rests."""
    t, E = z.shape
    c = torch.sigmoid(z) + correction
    margin = torch.full((t,), math.inf, dtype=z.dtype)
    if groups:
        per = E // groups["count"]
        score = c.view(t, groups["count"], per).sort(-1, descending=True).values[..., :2].sum(-1)
        order = score.sort(-1, descending=True)
        if groups["keep"] < groups["count"]:
            margin = order.values[:, groups["keep"] - 1] - order.values[:, groups["keep"]]
        kept = torch.zeros(t, groups["count"], dtype=torch.bool).scatter_(1, order.indices[:, :groups["keep"]], True)
        c = c.masked_fill(~kept.repeat_interleave(per, 1), -math.inf)
    best = c.sort(-1, descending=True)
    if top < E:
        margin = torch.minimum(margin, best.values[:, top - 1] - best.values[:, top])
    return best.indices[:, :top], margin


def routed(u, w, p, mlp, forced=None):
    """``forced``: {position: experts}, choices to take instead (the weights are still the router's). Returns (out, margins)."""
    r = mlp["router"]
    z = u @ w[p + "router"].T
    chosen, margin = choose(z, w[p + "correction"], r["top"], r.get("groups"))
    if forced is not None:
        chosen = torch.tensor([forced[i] for i in range(u.shape[0])], dtype=torch.long).view(u.shape[0], -1)
    s = torch.sigmoid(z).gather(1, chosen)
    share = s / (s.sum(-1, keepdim=True) + 1e-20)
    out = torch.zeros_like(u)
    for e in range(r["experts"]):
        rows, slot = (chosen == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += share[rows, slot][:, None] * unit(u[rows], w, f"{p}e{e}.")
    return out, margin


# ---------------------------------------------------------------- the model
def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None, margins=None, forced=None):
    """Logits [t, vocab] of one request. ``layers_out``: a list that receives the stream after every layer; ``margins``: a list
    that receives every routed layer's margins [t] ([] for the others); ``forced``: {layer: {position: experts}}."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        u = grouped_norm(x, w[p + "norm1"], groups, eps)
        h = u + causal_conv(u, w[p + "canon1"]) if (cfg.get("canon") or {}).get("taps") else u
        y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        x = x + y * torch.sigmoid(u @ w[p + "rg1"].T + w[p + "rg1.b"])
        mlp = layer.get("mlp")
        margin = []
        if mlp is not None:
            u = grouped_norm(x, w[p + "norm2"], groups, eps)
            if mlp["kind"] == "dense":
                y = unit(u, w, p + "mlp.")
            else:
                y, margin = routed(u, w, p + "mlp.", mlp, None if forced is None else forced.get(i, {}))
                margin = margin.tolist()
            x = x + y * torch.sigmoid(u @ w[p + "rg2"].T + w[p + "rg2.b"])
        if margins is not None:
            margins.append(margin)
        if layers_out is not None:
            layers_out.append(x.clone())
    return grouped_norm(x, w["final.norm"], groups, eps) @ w["head"].T


def generate(cfg, weights, prompt, n, dtype=torch.float64):
    out = list(prompt)
    for _ in range(n):
        out.append(int(forward(cfg, weights, out, dtype)[-1].argmax()))
    return out[len(prompt):]
