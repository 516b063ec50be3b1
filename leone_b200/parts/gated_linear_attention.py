"""Gated linear attention: a state per head whose rows decay each at its own, token-dependent rate.

``q = W_q x * q_scale`` and ``k = W_k x`` (heads x dim), ``v = W_v x`` (heads x vdim); a decay per key channel
``alpha = sigmoid(z)^(1/tau)`` with ``z = W_a2 (W_a1 x) + b`` (heads x dim; ``W_a1`` has ``decay_rank`` rows).
Per head ``S_t = diag(alpha_t) S_(t-1) + k_t v_t^T`` and ``o_t = S_t^T q_t``; every head's ``o`` is divided by
its root mean square over ``vdim`` and multiplied by a weight ``[vdim]`` shared by the heads and by
``silu(W_g x)``, then ``W_o``.  The state ``[heads, dim, vdim]`` is fp32, starts at zero and lives in the request's
state slot between steps.  The input projections are one product with fp32 results; the decay, the
recurrence, the norm and the gate are fp32.

(Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training" describes this recurrence.)
"""
from __future__ import annotations

import torch

from ..registry import MIXERS
from .base import FixedState, Mixer, WeightSpec


@MIXERS.register("gated_linear_attention")
class GatedLinearAttention(Mixer):
    writes_fresh = True           # forward(..., fresh=True) stores its result instead of adding it

    def __init__(self, params, rt):
        super().__init__(params, rt)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.dim = int(params["dim"])
        self.vdim = int(params["vdim"])
        self.rank = int(params["decay_rank"])
        self.tau = float(params["tau"])
        self.eps = float(params["norm_eps"])
        self.q_scale = float(params.get("q_scale", self.dim ** -0.5))
        self.names = {k: params.get(f"{k}_name", k) for k in ("q", "k", "v", "g", "a1", "a2", "o", "norm")}
        self.names["a2_bias"] = params.get("a2_bias_name", f"{self.names['a2']}.b")
        # tokens per chunk of a long prompt portion (the chunks run side by side); None: from the step's size
        self.fixed_chunk = int(params["chunk"]) if params.get("chunk") else None
        self.qk = self.heads * self.dim
        self.hv = self.heads * self.vdim
        # rows of the one input product: q, k, v, the gate, the decay's low-rank part
        self.v_off = 2 * self.qk
        self.g_off = self.v_off + self.hv
        self.u_off = self.g_off + self.hv
        self.cols = -(-(self.u_off + self.rank) // 16) * 16
        self.w_in = self.w_o = self.norm_w = self.w2 = self.w2_bias = None

    def weight_specs(self):
        n = self.names
        return [WeightSpec(n["q"], (self.qk, self.hidden)), WeightSpec(n["k"], (self.qk, self.hidden)),
                WeightSpec(n["v"], (self.hv, self.hidden)), WeightSpec(n["g"], (self.hv, self.hidden)),
                WeightSpec(n["o"], (self.hidden, self.hv)), WeightSpec(n["norm"], (self.vdim,), role="norm", std=0.1),
                WeightSpec(n["a1"], (self.rank, self.hidden)), WeightSpec(n["a2"], (self.qk, self.rank)),
                WeightSpec(n["a2_bias"], (self.qk,), role="vector", std=0.5)]

    def load(self, tensors):
        n = self.names
        rows = [tensors[n[k]] for k in ("q", "k", "v", "g", "a1")]
        used = sum(r.shape[0] for r in rows)
        if used < self.cols:
            rows.append(torch.zeros((self.cols - used, self.hidden), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = self.rt.ops.prepare_matrix(torch.cat(rows, dim=0).contiguous())
        self.w_o = self.rt.ops.prepare_matrix(tensors[n["o"]])
        self.norm_w = tensors[n["norm"]].float().contiguous()
        self.w2 = tensors[n["a2"]].float().t().contiguous()
        self.w2_bias = tensors[n["a2_bias"]].float().contiguous()

    def weight_bytes(self):
        return (self.cols * self.hidden + self.hidden * self.hv) * self.rt.dtype.itemsize + self.rank * self.qk * 4

    def scratch_bytes(self, max_tokens):
        chunks = max_tokens // self.chunk_for(max_tokens) + 1
        return max_tokens * ((self.cols + self.qk) * 4 + self.hv * (4 + self.rt.dtype.itemsize)) \
            + chunks * self.heads * self.dim * (self.vdim + 1) * 4

    def load_transient_bytes(self):
        return self.cols * self.hidden * self.rt.dtype.itemsize

    def cache_request(self):
        return FixedState((self.heads, self.dim, self.vdim))

    def chunk_for(self, tokens):
        """The longest chunk (a power of two from 32 to 256) that leaves about a block and a half for each of
        148 SMs: longer chunks move fewer states between the kernels, but an SM without a block does nothing."""
        chunk = self.fixed_chunk or 32
        while self.fixed_chunk is None and chunk < 256 and tokens * self.heads >= 2 * chunk * 200:
            chunk *= 2
        return chunk

    def forward(self, ctx, cache, x, hidden, fresh=False):
        rt, ops = self.rt, self.rt.ops
        n = hidden.shape[0]
        proj = rt.buffer("gla_proj", n, self.cols, torch.float32)
        ops.linear(x, self.w_in, proj)
        # a captured step has one token per sequence; otherwise long portions run chunk-parallel
        chunk = 0 if ctx.decode_only else self.chunk_for(n)
        if ctx.max_q_len <= 2 * chunk:
            chunk = 0
        gated = rt.buffer("gla_gated", n, self.hv, rt.dtype)
        ops.gated_linear_attention(ctx, proj, gated, cache.state, self.w2, self.w2_bias, self.norm_w, self.heads, self.dim,
                                   self.vdim, self.rank, self.tau, self.q_scale, self.eps, q_off=0, k_off=self.qk,
                                   v_off=self.v_off, u_off=self.u_off, gate_off=self.g_off, chunk=chunk)
        ops.linear(gated, self.w_o, hidden, residual=None if fresh else hidden)
