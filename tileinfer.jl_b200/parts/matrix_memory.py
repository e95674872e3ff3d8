"""Mixers with one matrix per head as their only memory, S_t = a_t S_(t-1) + b_t k_t v_t^T, read out by o_t = S_t^T q_t: the weight of the
past and of the new token are one number each per head, fixed or from the token.

``retention``: a fixed decay per head.

    q, k = rotation(W_q h), rotation(W_k h) dim^(-1/2)   [heads, dim]      v = W_v h   [heads, value_dim]
    S_t = decay_head S_(t-1) + k_t v_t^T;   o_t = S_t^T q_t
    out = W_o ( concat_heads(o / rms(o over the head)) * silu(W_g h) )

``mlstm`` (the matrix memory of xLSTM): exponential gates, kept in range by a running maximum m that starts at 0.

    q = W_q h dim^(-1/2), k = W_k h   [heads, dim]      v = W_v h   [heads, value_dim]
    i = c tanh((W_i h + b_i) / c),   f = log sigmoid(c tanh((W_f h + b_f) / c))          one of each per head, c = ``gate_cap``
    m_t = max(f + m_(t-1), i);   S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T;   n_t likewise with k alone
    o = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6)
    out = W_o ( concat_heads(o / rms(o over the head)) * norm * sigmoid(W_g h) )

Each asks the cache for one state of floats per sequence: S, and for mlstm n and m behind it. State, rotation, gates, divisor and norm are
32-bit in every element type; the four projections of a layer are one product (rounded to the model's element type), the gates' logits a
second one whose sums are not rounded. A step of one token per sequence is one kernel from the projections to the output projection's
input (``csrc/matrix_memory.cu``; heads of more than 128 values and sizes it refuses take two to four). Steps that bring a sequence
CHUNKED_FROM tokens or more cut its tokens into chunks that are worked on side by side (``csrc/memory_chunks.cu``), other steps scan their
tokens one by one (``csrc/lightning_scan.cuh``).

Record: ``num_heads``, ``head_dim`` (query/key size) and the options ``value_dim``, ``norm_eps``; retention: ``decay`` (one number per
head) and the position encoding's rotation, if any; mlstm: ``gate_cap``.
"""
from __future__ import annotations

import torch

from ..config.spec import MixerSpec, TensorDecl
from ..kernels import ops
from .base import CacheRequest, Mixer, register_mixer
from .linear import Linear

FUSED_VALUES = 128          # value sizes up to which a block of the one-token and of the chunked kernels holds a whole head
CHUNKED_FROM = 96           # new tokens of a step's longest sequence from which on its tokens are worked on in chunks


class MatrixMemory(Mixer):
    """What the two cells share. A cell sets ``name``, ``vector`` (whether n and m lie behind S) and ``constants`` (the scales of q and k, the
    rotation, the weight and gate of the heads' norm, and retention's decays)."""
    name, vector = "", False

    def __init__(self, spec: MixerSpec, tensors, rt, position):
        self.spec, self.rt = spec, rt
        o, n, p = spec.options, spec.tensor_names, spec.prefix
        self.heads, self.dim, self.vdim = spec.num_heads, spec.head_dim, int(o["value_dim"])
        self.eps = float(o.get("norm_eps", 1e-6))
        get = lambda k: rt.param(tensors[p + n[k]])
        self.proj = Linear(torch.cat([get(k) for k in ("q", "k", "v", "g")], 0).contiguous(), rt, self.name + "_in")
        HD, HV = self.heads * self.dim, self.heads * self.vdim
        self.offs = (0, HD, 2 * HD, 2 * HD + HV)                         # columns of q, k, v and the output gate
        self.o = Linear(get("o"), rt, "o")
        self.o.partials_name = "mixer.partials"

    @classmethod
    def tensors(cls, spec: MixerSpec):
        n, p = spec.tensor_names, spec.prefix
        W, HD, HV = spec.hidden_size, spec.num_heads * spec.head_dim, spec.num_heads * int(spec.options["value_dim"])
        rows = {"q": HD, "k": HD, "v": HV, "g": HV}
        return [TensorDecl(p + n[k], (r, W), ("normal", W ** -0.5)) for k, r in rows.items()] + [TensorDecl(p + n["o"], (W, HV), ("normal", HV ** -0.5))]

    def cache_request(self):
        floats = self.heads * self.dim * self.vdim + (self.heads * (self.dim + 1) if self.vector else 0)
        return CacheRequest("state", shape=(-(-floats // 4) * 4,), dtype=torch.float32)          # whole 16-byte pieces per sequence

    def gate_logits(self, h):
        """The gates' logits [n, 2 heads] in 32-bit, or None."""
        return None

    def forward(self, h, step, cache):
        rt, c = self.rt, self.constants
        n, H, D, V = h.shape[0], self.heads, self.dim, self.vdim
        state, sizes = cache.state, (self.heads, self.dim, self.vdim)
        rows = self.proj.forward(h, rt.buffer(self.name + ".rows", (n, self.proj.out_features)))
        z = self.gate_logits(h)
        y = rt.buffer(self.name + ".normed", (n, H * V))
        fused = V <= FUSED_VALUES
        # Where a block holds a whole head it leaves y; else the raw heads o (with the gated cell's divisor) go through the norm's kernel.
        o = None if fused else rt.buffer(self.name + ".o", (n, H * V), torch.float32)
        nq, em, m_new = (rt.buffer(f"{self.name}.{k}", (n, H), torch.float32) for k in ("nq", "em", "m_new")) if self.vector else (None, None, None)
        where = dict(y=y if fused else None, o=o, q_scale=c["q_scale"], k_scale=c["k_scale"], rotation=c["rotation"], w=c["w"],
                     gate_sigmoid=c["gate_sigmoid"], eps=self.eps, decay=c["decay"])
        moves = None
        if step.is_decode and ops.memory_token(rows, self.offs, state, step, *sizes, outs=(None,) * 3 if fused else (nq, em, m_new), z=z,
                                               bias=c["gate_bias"], cap=c["gate_cap"], **where):
            if self.vector and not fused:
                moves = (m_new, state[:, self.m_off:self.m_off + H], step.seq_slots)
        else:
            coef = None
            if self.vector:
                coef = rt.buffer(self.name + ".coef", (n, H, 2), torch.float32)
                ops.memory_gates(coef, em, z, c["gate_bias"], c["gate_cap"], state, self.m_off, step, H)
            if step.max_q_len >= CHUNKED_FROM:
                chunks, floats = ops.memory_chunk_sizes(step.host_q_lens, *sizes)
                ws, total = rt.buffer("memory.chunks", (floats,), torch.float32), rt.buffer("memory.totals", (chunks, H), torch.float32)
                ops.memory_chunks(rows, self.offs, state, step, *sizes, ws, total, chunks, nq=nq, em=em, coef=coef, **where)
            else:
                fused, o = False, rt.buffer(self.name + ".o", (n, H * V), torch.float32)
                if self.vector:
                    ops.memory_scan(o, nq, rows, *self.offs[:3], state, coef, c["q_scale"], c["k_scale"], step, *sizes)
                else:
                    ops.retention_scan(o, rows, *self.offs[:3], state, c["decay"], c["rotation"], c["q_scale"], c["k_scale"], step, *sizes)
        if not fused:
            ops.heads_norm_gate(y, o, rows[:, self.offs[3]:], c["w"], self.eps, H, V, gate_sigmoid=c["gate_sigmoid"],
                                divisor=(nq, em) if self.vector else None, moves=moves)
        return self.o.forward(y, rt.buffer("mixer.delta", (n, self.spec.hidden_size)), allow_partials=True)


@register_mixer("retention")
class Retention(MatrixMemory):
    name = "retention"

    def __init__(self, spec: MixerSpec, tensors, rt, position):
        super().__init__(spec, tensors, rt, position)
        decay = [float(a) for a in spec.options["decay"]]
        if len(decay) != self.heads:
            raise ValueError(f"retention: {len(decay)} decays for {self.heads} heads")
        self.constants = {"q_scale": 1.0, "k_scale": self.dim ** -0.5, "rotation": position.rotation() if position is not None else None, "w": None,
                          "gate_sigmoid": False, "decay": torch.tensor(decay, dtype=torch.float64).float().to(rt.device), "gate_bias": None, "gate_cap": 0.0}


@register_mixer("mlstm")
class MLstm(MatrixMemory):
    name, vector = "mlstm", True

    def __init__(self, spec: MixerSpec, tensors, rt, position):
        super().__init__(spec, tensors, rt, position)
        n, p = spec.tensor_names, spec.prefix
        self.gates = Linear(torch.cat([rt.param(tensors[p + n[k]]) for k in ("i", "f")], 0).contiguous(), rt, "mlstm_gates")
        bias = [rt.param(tensors[p + n[k] + n["bias_suffix"]], keep_dtype=True).float().flatten() for k in ("i", "f")]
        self.m_off = self.heads * self.dim * (self.vdim + 1)             # where m lies in a sequence's state, behind S and n
        self.constants = {"q_scale": self.dim ** -0.5, "k_scale": 1.0, "rotation": None, "w": rt.param(tensors[p + n["norm"]]), "gate_sigmoid": True,
                          "decay": None, "gate_bias": torch.cat(bias).contiguous(), "gate_cap": float(spec.options["gate_cap"])}

    @classmethod
    def tensors(cls, spec: MixerSpec):
        n, p = spec.tensor_names, spec.prefix
        W, H, V = spec.hidden_size, spec.num_heads, int(spec.options["value_dim"])
        out = super().tensors(spec) + [TensorDecl(p + n["norm"], (H * V,), ("one_plus_normal", 0.1))]
        for k, mean in (("i", -1.0), ("f", 3.0)):
            out += [TensorDecl(p + n[k], (H, W), ("normal", W ** -0.5)),
                    TensorDecl(p + n[k] + n["bias_suffix"], (H,), ("const_plus_normal", mean, 1.0), keep_dtype=True)]
        return out

    def gate_logits(self, h):
        return self.gates.forward_f32(h, self.rt.buffer("mlstm.gates", (h.shape[0], 2 * self.heads), torch.float32))
