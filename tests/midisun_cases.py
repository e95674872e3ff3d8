"""Small Midisun configurations for the tests, their random model folders and the comparison against the plain implementation
(``plain_midisun``).

The configurations differ from one another in every size and constant, and none keeps two sizes equal that a kernel could mix up
(query/key size and value size, heads and key/value heads, window and page, groups of the norm and of the router, taps).
"""
from __future__ import annotations

import os

import numpy as np
import torch

import plain_midisun as plain
from fasodra_cases import Recorder, compare, load_folder, prompts, tolerance, write_folder          # noqa: F401 (shared by the designs' tests)


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def moe(ff, experts, top, groups=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"expert": {"ff": ff}, "kind": "moe", "router": r}


def attention(heads, kv_heads, dim, scale, mlp, cap=None, window=None):
    m = {"dim": dim, "heads": heads, "scale": scale}
    if kv_heads:
        m["kv_heads"] = kv_heads
    if cap:
        m["softcap"] = cap
    if window:
        m["mask"] = {"size": window}
    return {"mixer": m, "mlp": mlp, "type": "attention"}


def retention(heads, dim, vdim, decay, mlp, rot=None):
    m = {"decay": decay, "dim": dim, "heads": heads}
    if vdim:
        m["vdim"] = vdim
    if rot:
        m["rot"] = {"base": rot[1], "dims": rot[0]}
    return {"mixer": m, "mlp": mlp, "type": "retention"}


def mlstm(heads, dim, vdim, cap, mlp):
    m = {"dim": dim, "gate_cap": cap, "heads": heads}
    if vdim:
        m["vdim"] = vdim
    return {"mixer": m, "mlp": mlp, "type": "mlstm"}


def model(vocab, width, eps, groups, taps, scale, layers):
    d = {"architecture": "Midisun", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}
    if taps:
        d["canon"] = {"taps": taps}
    return d


# Odd sizes that no fast kernel takes: three query heads per key/value head, a window shorter than a page, value sizes that are no
# multiple of four (their one-token steps run through the scans), part of a head rotated, a layer without feed-forward, three groups.
CASE_A = model(131, 60, 1e-5, 3, 4, 1.7, [
    attention(6, 2, 10, 0.4, moe(20, 6, 2, groups=(3, 2)), cap=7.0, window=9),
    mlstm(3, 10, 14, 5.0, moe(12, 5, 3)),
    retention(3, 12, 22, [0.5, 0.9, 0.995], None, rot=(6, 500.0)),
    attention(5, 5, 14, 0.3, dense(36), cap=3.0, window=70),
    mlstm(2, 18, 8, 9.0, moe(16, 8, 1, groups=(2, 1))),
])
# Sizes the tensor-core kernels take (widths in steps of 8, heads of 64 and 128): a recurrence first, a window of exactly a page
# and one across pages, heads of more than 128 values (no fused one-token kernel), every group kept, two taps.
CASE_B = model(320, 128, 1e-6, 8, 2, 2.5, [
    mlstm(2, 32, 64, 8.0, moe(64, 8, 2, groups=(4, 2))),
    attention(4, 2, 64, 0.13, moe(32, 16, 4, groups=(4, 4)), cap=12.0, window=64),
    retention(2, 64, 192, [0.8, 0.999], dense(256), rot=(64, 10000.0)),
    mlstm(1, 64, 136, 20.0, moe(96, 4, 3)),
    attention(3, 1, 128, 0.07, dense(72), cap=30.0, window=130),
    retention(4, 32, 32, [0.7, 0.97, 0.99, 0.9999], moe(40, 12, 2, groups=(2, 1)), rot=(16, 100.0)),
])
# What may be absent is absent: no window and no cap, key/value heads, value sizes, rotation and the router's groups left out, one
# group in the norm, one tap (no history), a layer without feed-forward.
CASE_C = model(97, 64, 3e-6, 1, 1, 1.0, [
    attention(2, None, 16, 0.25, None),
    retention(1, 16, None, [0.93], moe(24, 3, 2)),
    mlstm(1, 16, None, 4.0, dense(40)),
])
# No router anywhere (nothing that rounding could turn), and no convolution.
CASE_D = model(200, 96, 1e-6, 2, 0, 0.8, [
    retention(3, 48, 80, [0.6, 0.96, 0.998], dense(104), rot=(48, 3000.0)),
    attention(6, 3, 32, 0.18, dense(80), cap=9.0, window=33),
    mlstm(4, 24, 40, 15.0, dense(64)),
])
CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D}


def spread_routers(folder):
    """Rewrites a folder's routers so that choices rest on wider gaps and the corrections matter: rows twice as long, corrections of
    the scores' own size (negative choice scores included)."""
    from tileinfer_b200.weights.safetensors_io import SafetensorsFile, save_file
    path = os.path.join(folder, "model.safetensors")
    f = SafetensorsFile(path)
    tensors = {n: f.tensor(n).clone() for n in f.entries}
    del f
    for n, t in tensors.items():
        if n.endswith(".mlp.router"):
            tensors[n] = (t.float() * 2.0).to(t.dtype)
        elif n.endswith(".mlp.correction"):
            tensors[n] = (t.float() * 25.0 - 0.4).to(t.dtype)
    save_file(tensors, path)


class Model:
    """A case's folder, the plain implementation's view of it and cached reference logits."""

    def __init__(self, name: str, seed: int, tmp: str, case: dict = None):
        self.name = name
        self.folder = write_folder(case or CASES[name], seed, os.path.join(tmp, f"midisun_{name}_{seed}"))
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
