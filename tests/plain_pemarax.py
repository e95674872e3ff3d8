"""A plain, slow implementation of the Pemarax design, one function per mechanism, in torch on the CPU.

It takes a configuration in config.json's form and a dict of tensors by checkpoint name, and shares no code with the library: every
request is computed alone, with full keys and values, one token after the other where the design has a recurrence. ``dtype`` is the
arithmetic's type (float64 by default: the oracle of the tests).

In this file's notation, x the residual stream and N(y) = y / sqrt(mean(y^2) + eps):

* x0 = E[token]; a layer: x += m mixer(N(x) (1 + w1)), x += m ff(N(x) (1 + w2)) (a layer may have no ff); logits = Whead N(x) (1 + w).
* attention: u = Wq h, Wk h, Wv h, each through a causal convolution per channel; q and k rotated (neighbouring pairs, YaRN), then
  divided by their root mean square per head; keys with i - j < size or j < keep_first; softmax with a one in the denominator.
* latent_attention: q = Wq h per head [plain, rotated]; [c', r] = Wdkv h, c = N(c') w; a head's key is [Wuk c, r rotated], its value
  Wuv c; half-split rotation; a window.
* parallel: L = attention with q = N(q) w per head (k likewise), no rotation, a window; R = state-space recurrence: per head
  S <- exp(-exp(A) dt) S + dt B x^T, y = S^T C + D x, dt = softplus(dt' + bias), x, B, C through a convolution with bias and silu;
  Wo (N over equal parts (y silu(z)) w). The result is (N(L) w_left + N(R) w_right) / 2.
* routed ff: z = Wr u + b; the ``top`` largest z; weights = softmax over those; a unit is Wdown max(Wup u, 0)^2.
"""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------- small pieces
def rms_divide(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    return rms_divide(x, eps) * (1.0 + w)


def parts_norm(x, w, parts, eps):
    """The row in ``parts`` equal parts, each divided by its own root mean square, the whole times w."""
    y = x.reshape(x.shape[:-1] + (parts, x.shape[-1] // parts))
    return rms_divide(y, eps).reshape(x.shape) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(u, c):
    """u [t, channels], c [channels, taps]: y_t = sum_j c[:, j] u_(t - taps + 1 + j), zeros before the start."""
    t, taps = u.shape[0], c.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], 0)
    return sum(c[:, j] * padded[j:j + t] for j in range(taps))


def frequencies(dims, base, scaling=None):
    """(frequency per pair, multiplier of cos and sin)."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    place = lambda turns: dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(place(scaling["fast"])), 0), min(math.ceil(place(scaling["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / scaling["factor"] * r + v * (1 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot, interleaved):
    """x [t, heads, dim]: the first ``dims`` elements of every head; pairs (2i, 2i + 1), or (i, i + dims / 2)."""
    dims = rot["dims"]
    f, mult = frequencies(dims, rot["base"], rot.get("scaling"))
    a = positions.to(torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
    cos, sin = (torch.cos(a) * mult).to(x.dtype)[:, None, :], (torch.sin(a) * mult).to(x.dtype)[:, None, :]
    out = x.clone()
    if interleaved:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = u * cos - v * sin, v * cos + u * sin
    else:
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        out[..., :dims // 2], out[..., dims // 2:dims] = u * cos - v * sin, v * cos + u * sin
    return out


def visible(t, mask):
    """[query, key]: which keys a query sees."""
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    ok = j <= i
    if mask and mask.get("size"):
        inside = i - j < mask["size"]
        if mask.get("keep_first"):
            inside |= j < mask["keep_first"]
        ok &= inside
    return ok


def attend(q, k, v, scale, ok, one_more=False):
    """q [t, H, d], k [t, G, d], v [t, G, dv] -> [t, H * dv]. ``one_more``: exp(0) joins every denominator."""
    t, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = []
    for a in range(H):
        g = a // (H // G)
        s = ((q[:, a] @ k[:, g].T) * scale).masked_fill(~ok, -math.inf)
        top = s.max(-1, keepdim=True).values
        if one_more:
            top = top.clamp(min=0.0)
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True)
        if one_more:
            den = den + torch.exp(-top)
        out.append((e / den) @ v[:, g])
    return torch.cat(out, -1)


# ---------------------------------------------------------------- mixers
def attention(h, w, p, m, eps):
    t = h.shape[0]
    H, G, D, V = m["heads"], m.get("kv_heads") or m["heads"], m["dim"], m.get("vdim") or m["dim"]
    u = [h @ w[p + n].T for n in ("q", "k", "v")]
    if m.get("conv"):
        u = [causal_conv(y, w[p + n + ".conv"]) for y, n in zip(u, ("q", "k", "v"))]
    q, k, v = u[0].view(t, H, D), u[1].view(t, G, D), u[2].view(t, G, V)
    if m.get("rot"):
        pos = torch.arange(t)
        q, k = rotate(q, pos, m["rot"], True), rotate(k, pos, m["rot"], True)
    q, k = rms_divide(q, eps), rms_divide(k, eps)
    return attend(q, k, v, m["scale"], visible(t, m.get("mask")), one_more=True) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    t = h.shape[0]
    H, D, R, V, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(t, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms_divide(down[:, :rank], eps) * w[p + "dkv.norm"]
    shared = down[:, rank:].view(t, 1, R)
    pos = torch.arange(t)
    q_rot, k_rot = rotate(q[..., D:], pos, m["rot"], False), rotate(shared, pos, m["rot"], False)
    k = torch.cat([(c @ w[p + "uk"].T).view(t, H, D), k_rot.expand(t, H, R)], -1)
    v = (c @ w[p + "uv"].T).view(t, H, V)
    return attend(torch.cat([q[..., :D], q_rot], -1), k, v, m["scale"], visible(t, m.get("mask"))) @ w[p + "o"].T


def normed_attention(h, w, p, m, eps):
    t = h.shape[0]
    H, G, D, V = m["heads"], m.get("kv_heads") or m["heads"], m["dim"], m.get("vdim") or m["dim"]
    q = rms_divide((h @ w[p + "q"].T).view(t, H, D), eps) * w[p + "q.norm"]
    k = rms_divide((h @ w[p + "k"].T).view(t, G, D), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(t, G, V)
    return attend(q, k, v, m["scale"], visible(t, m.get("mask"))) @ w[p + "o"].T


def state_space_cell(x, B, C, dt, log_decay, D):
    """x [t, H, V], B, C [t, G, N], dt [t, H] (after softplus), log_decay [H] (A_log), D [H] -> y [t, H, V]."""
    t, H, V = x.shape
    per = H // B.shape[1]
    S = torch.zeros(H, B.shape[2], V, dtype=x.dtype)
    y = torch.zeros_like(x)
    for i in range(t):
        b, c = B[i].repeat_interleave(per, 0), C[i].repeat_interleave(per, 0)
        keep = torch.exp(-torch.exp(log_decay) * dt[i])
        S = keep[:, None, None] * S + dt[i][:, None, None] * b[:, :, None] * x[i][:, None, :]
        y[i] = torch.einsum("hnv,hn->hv", S, c) + D[:, None] * x[i]
    return y


def state_space(h, w, p, m, eps):
    t = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m.get("groups") or 1
    inner = H * V
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = silu(causal_conv(xbc, w[p + "conv"]) + w[p + "conv.b"])
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    dt = softplus(dt + w[p + "dt_bias"])
    y = state_space_cell(x.view(t, H, V), B.view(t, G, N), C.view(t, G, N), dt, w[p + "A_log"], w[p + "D"]).reshape(t, inner)
    return parts_norm(y * silu(z), w[p + "norm"], m.get("norm_groups") or 1, eps) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    left = normed_attention(h, w, p + "left.", m["left"], eps)
    right = state_space(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms_divide(left, eps) * w[p + "left.out"] + rms_divide(right, eps) * w[p + "right.out"])


MIXERS = {"attention": attention, "latent_attention": latent_attention, "parallel": parallel}


# ---------------------------------------------------------------- feed-forward
def unit(u, w, p):
    return torch.clamp(u @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def choose(z, top):
    """(chosen [t, top], margin [t]): the margin is the gap on which the choice rests."""
    best = z.sort(-1, descending=True)
    margin = torch.full((z.shape[0],), math.inf, dtype=z.dtype)
    if top < z.shape[1]:
        margin = best.values[:, top - 1] - best.values[:, top]
    return best.indices[:, :top], margin


def routed(u, w, p, mlp, forced=None):
    """``forced``: {position: experts}, choices to take instead (the weights are still the router's). Returns (out, margins)."""
    r = mlp["router"]
    z = u @ w[p + "router"].T + w[p + "router.b"]
    chosen, margin = choose(z, r["top"])
    if forced is not None:
        chosen = torch.tensor([forced[i] for i in range(u.shape[0])], dtype=torch.long).view(u.shape[0], -1)
    share = torch.softmax(z.gather(1, chosen), -1)
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
    eps, mult = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mult * MIXERS[layer["type"]](offset_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        margin = []
        if layer.get("mlp") is not None:
            y, margin = routed(offset_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], None if forced is None else forced.get(i, {}))
            x, margin = x + mult * y, margin.tolist()
        if margins is not None:
            margins.append(margin)
        if layers_out is not None:
            layers_out.append(x.clone())
    return offset_norm(x, w["final.norm"], eps) @ w["head"].T


def generate(cfg, weights, prompt, n, dtype=torch.float64):
    out = list(prompt)
    for _ in range(n):
        out.append(int(forward(cfg, weights, out, dtype)[-1].argmax()))
    return out[len(prompt):]
