"""Mamba-2: a recurrence with one decay per head and token (state-space duality).

``W_in x`` is ``[z: inner | x: inner | B: groups * n_state | C: groups * n_state | dt: heads]`` with ``inner = heads *
vdim``.  x, B and C together pass a short causal convolution over time per channel (``conv_taps``; tensor ``conv``
``[channels, taps]`` with bias ``conv.b``; the last ``taps - 1`` projected rows are state) and silu.  Per head, head
``h`` reading group ``h // (heads / groups)``, with ``d = softplus(dt + dt_bias)``:

    S_t = exp(-exp(A_log) d) S_(t-1) + d B_t x_t^T;   y_t = S_t^T C_t + D x_t

``y`` (heads concatenated) times ``silu(z)`` is RMS-normed in ``norm_groups`` equal parts, each by its own root mean
square, multiplied by a weight ``[inner]`` and projected by ``W_o``.  The state ``[heads, n_state, vdim]`` is fp32, starts
at zero and lives in the request's state slot between steps, beside the convolution's.  Projections and the
convolution's activations are kept in the run dtype; steps, decays, the recurrence, gate and norm are fp32.

(Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space
Duality" describes this layer.)
"""
from __future__ import annotations

import torch

from ..registry import MIXERS
from .base import CacheBundle, FixedState, Mixer, WeightSpec


@MIXERS.register("mamba2")
class Mamba2(Mixer):
    writes_fresh = True           # forward(..., fresh=True) stores its result instead of adding it

    def __init__(self, params, rt):
        super().__init__(params, rt)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.vdim = int(params["vdim"])
        self.n_state = int(params["n_state"])
        self.groups = int(params.get("groups", 1))
        self.norm_groups = int(params.get("norm_groups", 1))
        self.taps = int(params["conv_taps"])
        self.eps = float(params["norm_eps"])
        self.inner = self.heads * self.vdim
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.heads} heads of {self.vdim} in {self.groups} groups, normed in {self.norm_groups}")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"mamba2: taps {self.taps} (1 to 16)")
        self.names = {k: params.get(f"{k}_name", k) for k in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}
        self.conv_bias_name = params.get("conv_bias_name", f"{self.names['conv']}.b")
        self.bc = self.groups * self.n_state
        self.conv_cols = self.inner + 2 * self.bc
        # the product's rows as the kernels read them: every part starts on a 32-byte boundary
        self.conv_off = -(-self.inner // 16) * 16
        self.dt_off = self.conv_off + -(-self.conv_cols // 16) * 16
        self.cols = -(-(self.dt_off + self.heads) // 16) * 16
        self.w_in = self.w_o = self.conv_w = self.conv_b = self.norm_w = self.a_log = self.dt_bias = self.d_skip = None

    def weight_specs(self):
        n = self.names
        return [WeightSpec(n["in"], (2 * self.inner + 2 * self.bc + self.heads, self.hidden)),
                WeightSpec(n["conv"], (self.conv_cols, self.taps), std=0.3),
                WeightSpec(self.conv_bias_name, (self.conv_cols,), role="vector", std=0.3),
                WeightSpec(n["dt_bias"], (self.heads,), role="vector", std=0.5),
                WeightSpec(n["A_log"], (self.heads,), role="vector", std=0.5),
                WeightSpec(n["D"], (self.heads,), role="norm", std=0.1),
                WeightSpec(n["norm"], (self.inner,), role="norm", std=0.1),
                WeightSpec(n["o"], (self.hidden, self.inner))]

    def load(self, tensors):
        n = self.names
        src = tensors[n["in"]]
        w = torch.zeros((self.cols, self.hidden), dtype=src.dtype, device=src.device)
        w[:self.inner] = src[:self.inner]
        w[self.conv_off:self.conv_off + self.conv_cols] = src[self.inner:self.inner + self.conv_cols]
        w[self.dt_off:self.dt_off + self.heads] = src[self.inner + self.conv_cols:]
        self.w_in = self.rt.ops.prepare_matrix(w)
        self.w_o = self.rt.ops.prepare_matrix(tensors[n["o"]])
        self.conv_w = tensors[n["conv"]].float().contiguous()
        self.conv_b = tensors[self.conv_bias_name].float().contiguous()
        self.dt_bias, self.a_log, self.d_skip, self.norm_w = \
            (tensors[n[k]].float().contiguous() for k in ("dt_bias", "A_log", "D", "norm"))

    def weight_bytes(self):
        return (self.cols * self.hidden + self.hidden * self.inner) * self.rt.dtype.itemsize

    def scratch_bytes(self, max_tokens):
        chunks = max_tokens // self.chunk_for(max_tokens) + 1
        return max_tokens * ((self.cols + self.conv_cols + self.inner) * self.rt.dtype.itemsize + self.inner * 4) \
            + chunks * self.heads * self.n_state * (self.vdim + 1) * 4

    def load_transient_bytes(self):
        return self.cols * self.hidden * self.rt.dtype.itemsize

    def cache_request(self):
        return CacheBundle({"state": FixedState((self.heads, self.n_state, self.vdim)),
                            "conv": FixedState((self.taps - 1, self.conv_cols)) if self.taps > 1 else None})

    def chunk_for(self, tokens):
        """The longest chunk (a power of two from 64 to 512) that leaves about a block and a half for each of 148 SMs:
        longer chunks move fewer states between the kernels, but an SM without a block does nothing."""
        chunk = 64
        while chunk < 512 and tokens * self.heads * -(-self.vdim // 64) >= 2 * chunk * 200:
            chunk *= 2
        return chunk

    def forward(self, ctx, cache, x, hidden, fresh=False):
        rt, ops = self.rt, self.rt.ops
        n = hidden.shape[0]
        state, conv = cache["state"], cache["conv"]
        proj = rt.buffer("mamba_proj", n, self.cols, rt.dtype)
        ops.linear(x, self.w_in, proj)
        act = rt.buffer("mamba_act", n, self.conv_cols, rt.dtype)
        conv_state = conv.state if conv is not None else None
        raw = proj[:, self.conv_off:self.conv_off + self.conv_cols]
        # a step of one token a sequence: the convolution's kernel moves its state on itself
        fused = conv_state is not None and conv.writes and bool(ctx.decode_only)
        ops.short_conv(ctx, raw, self.conv_w, conv_state, act, activation="silu", update_state=fused, bias=self.conv_b)
        if conv_state is not None and conv.writes and not fused:
            ops.short_conv_state(ctx, raw, conv_state)
        # long portions run chunk-parallel
        chunk = 0 if ctx.decode_only else self.chunk_for(n)
        if ctx.max_q_len <= chunk:
            chunk = 0
        y = rt.buffer("mamba_y", n, self.inner, torch.float32)
        ops.ssd(ctx, act, proj, y, state.state, self.a_log, self.dt_bias, self.d_skip, self.heads, self.groups, self.n_state,
                self.vdim, x_off=0, b_off=self.inner, c_off=self.inner + self.bc, dt_off=self.dt_off, chunk=chunk)
        gated = rt.buffer("mamba_gated", n, self.inner, rt.dtype)
        ops.grouped_gate_norm(y, proj[:, :self.inner], self.norm_w, gated, self.eps, self.norm_groups)
        ops.linear(gated, self.w_o, hidden, residual=None if fresh else hidden)
