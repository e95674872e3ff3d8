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
input (``csrc/matrix_memory.cu``; heads of more than 128 values and sizes it refuses take two to four); other steps scan the step's
tokens (``csrc/lightning_scan.cuh``).

Record: ``num_heads``, ``head_dim`` (query/key size) and the options ``value_dim``, ``norm_eps``; retention: ``decay`` (one number per
head) and the position encoding's rotation, if any; mlstm: ``gate_cap``.
"""
from __future__ import annotations

import torch

from ..config.spec import MixerSpec, TensorDecl
from ..kernels import ops
from .base import CacheRequest, Mixer, register_mixer
from .linear import Linear

FUSED_VALUES = 128          # value sizes up to which a block of the one-token kernel holds a whole head


class MatrixMemory(Mixer):
    """What the two cells share. A cell sets ``q_scale``, ``k_scale``, ``norm_w``, ``gate_sigmoid``, ``vector`` (whether n and m lie behind
    S) and offers ``token`` and ``scan``."""
    name, vector, gate_sigmoid = "", False, False
    norm_w = None
    q_scale = k_scale = 1.0

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

    def forward(self, h, step, cache):
        rt = self.rt
        n, H, V = h.shape[0], self.heads, self.vdim
        rows = rt.buffer(self.name + ".rows", (n, self.proj.out_features))
        self.proj.forward(h, rows)
        y = rt.buffer(self.name + ".normed", (n, H * V))
        if not (step.is_decode and self.token(h, rows, y, step, cache.state)):
            o = rt.buffer(self.name + ".o", (n, H * V), torch.float32)
            divisor, moves = self.scan(h, rows, o, step, cache.state)
            ops.heads_norm_gate(y, o, rows[:, self.offs[3]:], self.norm_w, self.eps, H, V, gate_sigmoid=self.gate_sigmoid, divisor=divisor, moves=moves)
        out = rt.buffer("mixer.delta", (n, self.spec.hidden_size))
        return self.o.forward(y, out, allow_partials=True)


@register_mixer("retention")
class Retention(MatrixMemory):
    name = "retention"

    def __init__(self, spec: MixerSpec, tensors, rt, position):
        super().__init__(spec, tensors, rt, position)
        decay = [float(a) for a in spec.options["decay"]]
        if len(decay) != self.heads:
            raise ValueError(f"retention: {len(decay)} decays for {self.heads} heads")
        self.decay = torch.tensor(decay, dtype=torch.float64).float().to(rt.device)
        self.k_scale = self.dim ** -0.5
        self.rotation = position.rotation() if position is not None else None

    def token(self, h, rows, y, step, state):
        return self.vdim <= FUSED_VALUES and ops.memory_token(rows, self.offs, state, step, self.heads, self.dim, self.vdim, y=y, decay=self.decay,
                                                              rotation=self.rotation, k_scale=self.k_scale, eps=self.eps)

    def scan(self, h, rows, o, step, state):
        done = step.is_decode and ops.memory_token(rows, self.offs, state, step, self.heads, self.dim, self.vdim, o=o, decay=self.decay,
                                                   rotation=self.rotation, k_scale=self.k_scale)
        if not done:
            ops.retention_scan(o, rows, *self.offs[:3], state, self.decay, self.rotation, 1.0, self.k_scale, step, self.heads, self.dim, self.vdim)
        return None, None


@register_mixer("mlstm")
class MLstm(MatrixMemory):
    name, vector, gate_sigmoid = "mlstm", True, True

    def __init__(self, spec: MixerSpec, tensors, rt, position):
        super().__init__(spec, tensors, rt, position)
        n, p = spec.tensor_names, spec.prefix
        self.cap = float(spec.options["gate_cap"])
        self.q_scale = self.dim ** -0.5
        self.norm_w = rt.param(tensors[p + n["norm"]])
        self.gates = Linear(torch.cat([rt.param(tensors[p + n[k]]) for k in ("i", "f")], 0).contiguous(), rt, "mlstm_gates")
        bias = [rt.param(tensors[p + n[k] + n["bias_suffix"]], keep_dtype=True).float().flatten() for k in ("i", "f")]
        self.gate_bias = torch.cat(bias).contiguous()
        self.m_off = self.heads * self.dim * (self.vdim + 1)             # where m lies in a sequence's state, behind S and n

    @classmethod
    def tensors(cls, spec: MixerSpec):
        n, p = spec.tensor_names, spec.prefix
        W, H, V = spec.hidden_size, spec.num_heads, int(spec.options["value_dim"])
        out = super().tensors(spec) + [TensorDecl(p + n["norm"], (H * V,), ("one_plus_normal", 0.1))]
        for k, mean in (("i", -1.0), ("f", 3.0)):
            out += [TensorDecl(p + n[k], (H, W), ("normal", W ** -0.5)),
                    TensorDecl(p + n[k] + n["bias_suffix"], (H,), ("const_plus_normal", mean, 1.0), keep_dtype=True)]
        return out

    def _logits(self, h):
        return self.gates.forward_f32(h, self.rt.buffer("mlstm.gates", (h.shape[0], 2 * self.heads), torch.float32))

    def _token(self, h, rows, step, state, **where):
        return ops.memory_token(rows, self.offs, state, step, self.heads, self.dim, self.vdim, z=self._logits(h), bias=self.gate_bias, cap=self.cap,
                                q_scale=self.q_scale, w=self.norm_w, gate_sigmoid=True, eps=self.eps, **where)

    def token(self, h, rows, y, step, state):
        return self.vdim <= FUSED_VALUES and self._token(h, rows, step, state, y=y)

    def scan(self, h, rows, o, step, state):
        rt, H, n = self.rt, self.heads, h.shape[0]
        nq, em, m_new = (rt.buffer("mlstm." + k, (n, H), torch.float32) for k in ("nq", "em", "m_new"))
        m = state[:, self.m_off:self.m_off + H]
        if step.is_decode and self._token(h, rows, step, state, o=o, outs=(nq, em, m_new)):
            return (nq, em), (m_new, m, step.seq_slots)
        coef = rt.buffer("mlstm.coef", (n, H, 2), torch.float32)
        ops.memory_gates(coef, em, self._logits(h), self.gate_bias, self.cap, state, self.m_off, step, H)
        ops.memory_scan(o, nq, rows, *self.offs[:3], state, coef, self.q_scale, 1.0, step, H, self.dim, self.vdim)
        return (nq, em), None
