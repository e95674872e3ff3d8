"""The state-space mixer of Mamba-2: one matrix per head as the only memory, with one decay and one step size per token and head, behind a
short convolution.

    [z | x | B | C | dt'] = W_in h            z, x [heads, value_dim], B, C [groups, state], dt' [heads]
    x, B, C <- silu(conv(x, B, C) + bias)     per channel, causal over time, ``conv_taps`` taps (the last one the current token's)
    dt = softplus(dt' + dt_bias),  l = -exp(A_log) dt                                         one of each per head, 32-bit
    S_t = e^l S_(t-1) + dt B_t x_t^T  [state, value_dim];   y_t = S_t^T C_t + D x_t           head i reads group i / (heads / groups)
    out = W_o ( norm over ``norm_groups`` equal parts of (y silu(z)) * w )

A sequence keeps the matrices S and the last taps - 1 rows of x | B | C, one block of floats. One-token steps run in ``ssm_token``, others in
chunks of tokens that are worked on side by side (``csrc/ssm_chunks.cu`` on the tensor cores, ``csrc/memory_chunks.cu`` in 32-bit and for the
sizes the other refuses); the recurrence and all that enters it from dt' on is 32-bit in
every element type.

Record: ``num_heads``, ``head_dim`` (the state's size) and the options ``value_dim``, ``groups``, ``conv_taps``, ``norm_groups``, ``norm_eps``.
"""
from __future__ import annotations

import torch

from ..config.spec import MixerSpec, TensorDecl
from ..kernels import ops
from .base import CacheRequest, Mixer, register_mixer
from .linear import Linear


def chunk_step(rt, y, xbc, coef, skip, state, step, heads, groups, dim, vdim):
    """The recurrence over a step of several tokens per sequence, with its work space from the runtime's scratch buffers."""
    chunks, floats = ops.memory_chunk_sizes(step.host_q_lens, heads, dim, vdim)
    ws, total = rt.buffer("memory.chunks", (floats,), torch.float32), rt.buffer("memory.totals", (chunks, heads), torch.float32)
    ops.ssm_chunks(y, xbc, coef, skip, state, step, heads, groups, dim, vdim, ws, total, chunks, tensor_cores=rt.fast)


@register_mixer("state_space")
class StateSpace(Mixer):
    def __init__(self, spec: MixerSpec, tensors, rt, position):
        self.spec, self.rt = spec, rt
        o, n, p = spec.options, spec.tensor_names, spec.prefix
        self.heads, self.dim, self.vdim, self.groups = spec.num_heads, spec.head_dim, int(o["value_dim"]), int(o.get("groups") or 1)
        self.parts, self.eps = int(o.get("norm_groups") or 1), float(o.get("norm_eps", 1e-6))
        self.inner = self.heads * self.vdim
        if self.heads % self.groups or self.inner % self.parts:
            raise ValueError(f"state_space: {self.heads} heads in {self.groups} groups, rows of {self.inner} in {self.parts} parts")
        get = lambda k: rt.param(tensors[p + n[k]])
        exact = lambda k: rt.param(tensors[p + n[k]], keep_dtype=True).float().flatten().contiguous()
        self.channels = self.inner + 2 * self.groups * self.dim
        # Filled up with zero rows so that a token's row of the product is whole 16-byte pieces.
        w = get("in")
        fill = -w.shape[0] % 16
        self.proj = Linear(torch.cat([w, torch.zeros(fill, w.shape[1], dtype=w.dtype, device=w.device)], 0).contiguous() if fill else w, rt, "state_space_in")
        self.conv = get("conv").t().contiguous()                     # [taps, channels]: neighbouring channels' weights of one tap lie together
        self.taps = self.conv.shape[0]
        self.conv_bias = get("conv_bias")
        self.dt_bias, self.a_log, self.skip = exact("dt_bias"), exact("A_log"), exact("D")
        self.norm_w = get("norm")
        self.o = Linear(get("o"), rt, "o")
        self.out_name = "mixer.delta"
        self.o.partials_name = "state_space.partials"
        self.matrices = self.heads * self.dim * self.vdim            # floats of a sequence's state ahead of the convolution's rows
        self.hist_off = -(-self.matrices // 4) * 4

    @classmethod
    def tensors(cls, spec: MixerSpec):
        n, p, o = spec.tensor_names, spec.prefix, spec.options
        W, H, N, V, G, taps = spec.hidden_size, spec.num_heads, spec.head_dim, int(o["value_dim"]), int(o.get("groups") or 1), int(o["conv_taps"])
        C = H * V + 2 * G * N
        return [TensorDecl(p + n["in"], (H * V + C + H, W), ("normal", W ** -0.5)),
                TensorDecl(p + n["conv"], (C, taps), ("const_plus_normal", 1.0 / taps, 0.3)), TensorDecl(p + n["conv_bias"], (C,), ("normal", 0.1)),
                TensorDecl(p + n["dt_bias"], (H,), ("const_plus_normal", -2.0, 1.0), keep_dtype=True),
                TensorDecl(p + n["A_log"], (H,), ("normal", 0.7), keep_dtype=True), TensorDecl(p + n["D"], (H,), ("one_plus_normal", 0.2), keep_dtype=True),
                TensorDecl(p + n["norm"], (H * V,), ("one_plus_normal", 0.1)), TensorDecl(p + n["o"], (W, H * V), ("normal", (H * V) ** -0.5))]

    def cache_request(self):
        floats = self.hist_off + (self.taps - 1) * self.channels
        return CacheRequest("state", shape=(-(-floats // 4) * 4,), dtype=torch.float32)          # whole 16-byte pieces per sequence

    def forward(self, h, step, cache):
        rt, n, state = self.rt, h.shape[0], cache.state
        sizes = (self.heads, self.groups, self.dim, self.vdim)
        rows = self.proj.forward(h, rt.buffer("state_space.rows", (n, self.proj.out_features)))
        xbc = rt.buffer("state_space.inputs", (n, self.channels))
        coef = rt.buffer("state_space.coef", (n, self.heads, 2), torch.float32)
        hist = state[:, self.hist_off:] if self.taps > 1 else None
        ops.ssm_inputs(xbc, coef, rows, self.inner, self.inner + self.channels, self.conv, self.conv_bias, hist, self.dt_bias, self.a_log, step)
        y = rt.buffer("state_space.y", (n, self.inner), torch.float32)
        if step.is_decode:
            ops.ssm_token(y, xbc, coef, self.skip, state, step, *sizes)
        else:
            if self.taps > 1:
                ops.history_update(hist, rows[:, self.inner:], self.taps, step, self.channels)
            chunk_step(rt, y, xbc, coef, self.skip, state, step, *sizes)
        gated = rt.buffer("state_space.normed", (n, self.inner))
        ops.ssm_gate_norm(gated, y, rows[:, :self.inner], self.norm_w, self.eps, self.parts)
        return self.o.forward(gated, rt.buffer(self.out_name, (n, self.spec.hidden_size)), allow_partials=True)
