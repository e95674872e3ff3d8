"""Small Pemarax configurations for the tests, their random model folders and the comparison against the plain implementation
(``plain_pemarax``).

The configurations differ from one another in every size and constant, and none keeps two sizes equal that a kernel could mix up
(query/key size and value size, heads and key/value heads, window and page, kept positions, groups and norm parts, state and value size).
"""
from __future__ import annotations

import os

import numpy as np
import torch

import plain_pemarax as plain
from fasodra_cases import Recorder, compare, load_folder, prompts, tolerance, write_folder          # noqa: F401 (shared by the designs' tests)


def moe(ff, experts, top):
    return {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}


def mask(window, keep=None):
    if window is None:
        return {}
    return {"mask": {"size": window, **({"keep_first": keep} if keep else {})}}


def attention(heads, kv_heads, dim, vdim, scale, mlp, window=None, keep=None, conv=None, rot=None, yarn=None):
    m = {"dim": dim, "heads": heads, "scale": scale, **mask(window, keep)}
    if kv_heads:
        m["kv_heads"] = kv_heads
    if vdim:
        m["vdim"] = vdim
    if conv:
        m["conv"] = conv
    if rot:
        m["rot"] = {"base": rot[1], "dims": rot[0]}
        if yarn:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"mixer": m, "mlp": mlp, "type": "attention"}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, mlp, window=None):
    m = {"dim": dim, "heads": heads, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim}, "rot_dim": rot_dim, "scale": scale, "vdim": vdim,
         **mask(window)}
    return {"mixer": m, "mlp": mlp, "type": "latent_attention"}


def parallel(left, right, mlp):
    """left: (heads, kv_heads, dim, vdim, scale, window); right: (heads, vdim, state, groups, conv, norm_groups)."""
    H, G, D, V, scale, window = left
    l = {"dim": D, "heads": H, "scale": scale, **mask(window)}
    if G:
        l["kv_heads"] = G
    if V:
        l["vdim"] = V
    r = dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right))
    return {"mixer": {"left": l, "right": {k: v for k, v in r.items() if v}}, "mlp": mlp, "type": "parallel"}


def model(vocab, width, eps, mult, layers):
    return {"architecture": "Pemarax", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


# Odd sizes that no fast kernel takes: three query heads per key/value head, windows shorter than a page, part of a head rotated, value and
# state sizes that are no multiple of four, heads in groups, norm parts that cut through heads.
CASE_A = model(131, 60, 1e-5, 0.7, [
    attention(6, 2, 10, 14, 0.6, moe(20, 6, 2), window=9, keep=5, conv=3, rot=(6, 500.0), yarn=(8.0, 64, 8.0, 1.0)),
    parallel((3, 1, 12, 22, 0.3, 33), (6, 7, 10, 3, 4, 2), moe(12, 5, 3)),
    latent(3, 10, 6, 14, 18, 0.25, 300.0, None, window=70),
    parallel((4, 4, 6, 10, 0.5, 7), (4, 9, 18, 2, 2, 6), moe(16, 8, 1)),
    attention(5, 5, 14, 6, 0.4, moe(24, 3, 3), window=66, keep=70, conv=2, rot=(14, 50.0), yarn=(2.0, 32, 4.0, 0.5)),
])
# Sizes the tensor-core kernels take (widths in steps of 8, heads of 64 and 128): windows of exactly a page and across pages, kept positions
# of a few, of exactly a page and beyond one, chunks' products at sizes in steps of 16 and others.
CASE_B = model(320, 128, 1e-6, 0.5, [
    parallel((4, 2, 64, 32, 0.11, 64), (4, 32, 16, 2, 4, 4), moe(64, 8, 2)),
    attention(4, 2, 64, 48, 0.45, moe(32, 16, 4), window=130, keep=3, conv=4, rot=(64, 20000.0), yarn=(4.0, 128, 16.0, 1.0)),
    latent(4, 32, 16, 48, 112, 0.14, 10000.0, moe(64, 8, 3), window=100),
    parallel((2, 1, 128, 64, 0.09, 200), (2, 96, 64, 1, 3, 1), moe(96, 4, 2)),
    attention(3, 1, 128, 128, 0.3, None, window=64, keep=64, conv=1, rot=(32, 100.0)),
    latent(2, 64, 32, 64, 64, 0.1, 1000.0, moe(40, 12, 5), window=65),
    attention(2, 2, 32, 64, 0.8, moe(72, 6, 2), window=70, keep=100, conv=4, rot=(32, 3000.0)),
])
# What may be absent is absent: no windows, no rotation and no convolution, key/value heads, value sizes, groups left out, no residual
# multiplier to speak of, a layer without feed-forward.
CASE_C = model(97, 64, 3e-6, 1.0, [
    attention(2, None, 16, None, 0.8, None),
    parallel((1, None, 32, None, 0.2, None), (2, 16, 16, None, 1, None), moe(24, 2, 1)),
    latent(2, 16, 8, 16, 24, 0.2, 100.0, moe(40, 6, 6)),
])
CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C}


def spread_routers(folder):
    """Rewrites a folder's routers so that choices rest on wider gaps and the biases matter: rows twice as long, biases of the logits' size."""
    from tileinfer_b200.weights.safetensors_io import SafetensorsFile, save_file
    path = os.path.join(folder, "model.safetensors")
    f = SafetensorsFile(path)
    tensors = {n: f.tensor(n).clone() for n in f.entries}
    del f
    for n, t in tensors.items():
        if n.endswith(".mlp.router"):
            tensors[n] = (t.float() * 2.0).to(t.dtype)
        elif n.endswith(".mlp.router.b"):
            tensors[n] = (t.float() * 10.0).to(t.dtype)
    save_file(tensors, path)


class Model:
    """A case's folder, the plain implementation's view of it and cached reference logits."""

    def __init__(self, name: str, seed: int, tmp: str, case: dict = None):
        self.name = name
        self.folder = write_folder(case or CASES[name], seed, os.path.join(tmp, f"pemarax_{name}_{seed}"))
        spread_routers(self.folder)
        self.cfg, self.W = load_folder(self.folder)
        self.vocab = self.cfg["vocab"]
        self._refs = {}

    def reference(self, tokens, forced=None):
        """(logits [n, vocab] in 64-bit arithmetic as numpy, every position's smallest router margin [n]). ``forced``: router
        choices to take instead of the plain implementation's own ({layer: {position: experts}})."""
        if forced is not None:
            return plain.forward(self.cfg, self.W, list(tokens), forced=forced).float().numpy(), np.full(len(tokens), np.inf)
        key = tuple(tokens)
        if key not in self._refs:
            margins = []
            logits = plain.forward(self.cfg, self.W, list(tokens), margins=margins)
            per_layer = [m for m in margins if m]
            smallest = np.min(np.array(per_layer), axis=0) if per_layer else np.full(len(tokens), np.inf)
            self._refs[key] = (logits.float().numpy(), smallest)
        return self._refs[key]

    def layers(self, tokens):
        out = []
        plain.forward(self.cfg, self.W, list(tokens), layers_out=out)
        return [x.float() for x in out]

    def engine(self, dtype: str, **kw):
        from tileinfer_b200.engine import Engine
        args = dict(max_tokens=2048, max_seqs=6, max_context=1024)
        args.update(kw)
        return Engine.load(self.folder, dtype=dtype, **args)
