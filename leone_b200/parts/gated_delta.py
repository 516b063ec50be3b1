"""The gated delta rule: a recurrence whose state is corrected towards each new value.

``q = W_q x`` and ``k = W_k x`` (``kv_heads x dim``), ``v = W_v x`` (``heads x vdim``); each passes a short
causal convolution over time per channel (``conv_taps``; tensors ``<name>.conv`` ``[channels, taps]``, the
last ``taps - 1`` projected rows are state) and silu; q and k become unit vectors per head (``x /
sqrt(sum x^2 + 1e-6)``), q times ``dim^(-1/2)``; head ``h`` reads q/k head ``h // (heads / kv_heads)``.
Per head, with ``beta = sigmoid(W_b x)`` and ``g = exp(-exp(A_log) softplus(W_a x + dt_bias))``:

    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

so the read-out sees the token's own write.  Every head's ``o`` is divided by its root mean square over
``vdim``, multiplied by a weight ``[vdim]`` shared by the heads and by ``silu(W_g x)``, then ``W_o``.
The state ``[heads, dim, vdim]`` is fp32, starts at zero and lives in the request's state slot between
steps, beside the convolution's.  The convolution's sums, its activation, the unit norms, the gates, the decay
and the recurrence are fp32.

``decay = "channel"``: one decay per head and key channel instead, ``g = exp(-exp(A_log_h) softplus(W_a2 (W_a1 x) +
dt_bias))`` (``W_a1``: ``decay_rank`` rows; ``dt_bias``: ``[heads * dim]``), acting on the rows of ``S``.
``gate = "low_rank"``: the output gate's logits are ``W_g2 (W_g1 x)`` (``gate_rank`` inner rows).  ``gate_act``: ``"silu"`` or
``"sigmoid"``.  With both low ranks the two second products are one product of a block-diagonal matrix.
With ``projections = "run"`` the input product's rows are kept in the run dtype; by default they are fp32.

(Yang et al., "Gated Delta Networks: Improving Mamba2 with Delta Rule" describes this recurrence.)
"""
from __future__ import annotations

import torch

from ..registry import MIXERS
from .base import CacheBundle, FixedState, Mixer, WeightSpec


@MIXERS.register("gated_delta_rule")
class GatedDeltaRule(Mixer):
    writes_fresh = True           # forward(..., fresh=True) stores its result instead of adding it

    def __init__(self, params, rt):
        super().__init__(params, rt)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.kv_heads = int(params.get("kv_heads") or self.heads)
        if self.heads % self.kv_heads:
            raise ValueError(f"gated_delta_rule: heads {self.heads} is not a multiple of kv_heads {self.kv_heads}")
        self.dim = int(params["dim"])
        self.vdim = int(params["vdim"])
        self.taps = int(params.get("conv_taps") or 0)
        self.eps = float(params["norm_eps"])
        self.q_scale = float(params.get("q_scale", self.dim ** -0.5))
        self.channel = params.get("decay", "head") == "channel"
        self.low_rank_gate = params.get("gate", "full") == "low_rank"
        if params.get("decay", "head") not in ("head", "channel") or params.get("gate", "full") not in ("full", "low_rank"):
            raise ValueError(f"gated_delta_rule: decay '{params.get('decay')}' / gate '{params.get('gate')}'")
        self.gate_act = params.get("gate_act", "silu")
        if self.gate_act not in ("silu", "sigmoid"):
            raise ValueError(f"gated_delta_rule: gate_act '{self.gate_act}'")
        self.proj_dtype = rt.dtype if params.get("projections") == "run" else torch.float32
        if self.proj_dtype != rt.dtype and (self.channel or self.low_rank_gate):
            raise ValueError("gated_delta_rule: low-rank inner rows feed a second product, so the projections are in the run dtype")
        if self.proj_dtype != torch.float32 and not self.low_rank_gate:
            raise ValueError("gated_delta_rule: a full gate's logits are fp32 rows of the input product")
        self.decay_rank = int(params["decay_rank"]) if self.channel else 0
        self.gate_rank = int(params["gate_rank"]) if self.low_rank_gate else 0
        self.names = {k: params.get(f"{k}_name", k) for k in ("q", "k", "v", "g", "a", "b", "o", "norm", "A_log", "dt_bias",
                                                              "a1", "a2", "g1", "g2")}
        self.conv_names = {k: params.get(f"{k}_conv_name", f"{self.names[k]}.conv") for k in ("q", "k", "v")}
        self.qk = self.kv_heads * self.dim
        self.hv = self.heads * self.vdim
        self.conv_cols = 2 * self.qk + self.hv
        # rows of the one input product: q, k, v (the convolution's channels), then either the gate or its inner rows,
        # a (or the decay's inner rows) and b; padded so that what another product reads starts on a 16-byte boundary
        def up(x, m):
            return -(-x // m) * m
        self.inner = bool(self.channel or self.low_rank_gate)
        self.a_rows, self.g_rows = up(self.decay_rank, 8), up(self.gate_rank, 8)      # inner rows with padding
        if self.inner:
            self.u_off = up(self.conv_cols, 16)
            self.g_off = self.u_off + self.a_rows + self.g_rows
        else:
            self.u_off = self.g_off = self.conv_cols
        self.a_off = self.g_off + (0 if self.low_rank_gate else self.hv)
        self.b_off = self.a_off + (0 if self.channel else self.heads)
        self.cols = up(self.b_off + self.heads, 16)
        # columns of the second product: the decay's logits, then the gate's
        self.z_gate = up(self.heads * self.dim, 16) if self.channel else 0
        self.z_cols = up(self.z_gate + (self.hv if self.low_rank_gate else 0), 16)
        self.w_in = self.w_z = self.w_o = self.conv_w = self.norm_w = self.a_log = self.dt_bias = None

    def weight_specs(self):
        n = self.names
        rows = {"q": self.qk, "k": self.qk, "v": self.hv}
        specs = []
        for k in ("q", "k", "v"):
            specs.append(WeightSpec(n[k], (rows[k], self.hidden)))
            if self.taps:
                specs.append(WeightSpec(self.conv_names[k], (rows[k], self.taps), std=0.3))
        specs += [WeightSpec(n["b"], (self.heads, self.hidden)), WeightSpec(n["A_log"], (self.heads,), role="vector", std=0.5),
                  WeightSpec(n["norm"], (self.vdim,), role="norm", std=0.1), WeightSpec(n["o"], (self.hidden, self.hv))]
        if self.channel:
            specs += [WeightSpec(n["a1"], (self.decay_rank, self.hidden)),
                      WeightSpec(n["a2"], (self.heads * self.dim, self.decay_rank)),
                      WeightSpec(n["dt_bias"], (self.heads * self.dim,), role="vector", std=0.5)]
        else:
            specs += [WeightSpec(n["a"], (self.heads, self.hidden)), WeightSpec(n["dt_bias"], (self.heads,), role="vector", std=0.5)]
        if self.low_rank_gate:
            specs += [WeightSpec(n["g1"], (self.gate_rank, self.hidden)), WeightSpec(n["g2"], (self.hv, self.gate_rank))]
        else:
            specs.append(WeightSpec(n["g"], (self.hv, self.hidden)))
        return specs

    def load(self, tensors):
        n = self.names
        some = tensors[n["q"]]
        w = torch.zeros((self.cols, self.hidden), dtype=some.dtype, device=some.device)
        places = [("q", 0), ("k", self.qk), ("v", 2 * self.qk), ("b", self.b_off)]
        places += [("a1", self.u_off)] if self.channel else [("a", self.a_off)]
        places += [("g1", self.u_off + self.a_rows)] if self.low_rank_gate else [("g", self.g_off)]
        for k, at in places:
            w[at:at + tensors[n[k]].shape[0]] = tensors[n[k]]
        self.w_in = self.rt.ops.prepare_matrix(w)
        if self.inner:
            z = torch.zeros((self.z_cols, self.a_rows + self.g_rows), dtype=some.dtype, device=some.device)
            bias = torch.zeros(self.z_cols, dtype=torch.float32, device=some.device)
            if self.channel:
                z[:self.heads * self.dim, :self.decay_rank] = tensors[n["a2"]]
                bias[:self.heads * self.dim] = tensors[n["dt_bias"]].float()
            if self.low_rank_gate:
                z[self.z_gate:self.z_gate + self.hv, self.a_rows:self.a_rows + self.gate_rank] = tensors[n["g2"]]
            self.w_z = self.rt.ops.prepare_matrix(z, bias)
        self.w_o = self.rt.ops.prepare_matrix(tensors[n["o"]])
        if self.taps:
            self.conv_w = torch.cat([tensors[self.conv_names[k]].float() for k in ("q", "k", "v")], dim=0).contiguous()
        else:       # no convolution: one tap of weight one, so that the same kernel applies the activation
            self.conv_w = torch.ones((self.conv_cols, 1), dtype=torch.float32, device=some.device)
        self.norm_w = tensors[n["norm"]]
        self.a_log = tensors[n["A_log"]].float().contiguous()
        self.dt_bias = tensors[n["dt_bias"]].float().contiguous()

    def weight_bytes(self):
        return (self.cols * self.hidden + self.hidden * self.hv + self.z_cols * (self.a_rows + self.g_rows)) * self.rt.dtype.itemsize

    def scratch_bytes(self, max_tokens):
        rows = max_tokens * ((self.cols + self.conv_cols + self.z_cols + self.hv) * 4 + self.hv * self.rt.dtype.itemsize)
        if self.rt.dtype == torch.float32 or self.dim > 128:
            return rows
        # prompt portions on tensor cores: what 16 tokens of a head bring, as bfloat16 terms (csrc/gated_delta_mma.cu)
        padded = 64 if self.dim <= 64 else 128
        return rows + min(max_tokens, max_tokens // 16 + 256) * self.heads * (192 * (padded + 8) + 3072 + 4 * padded)

    def load_transient_bytes(self):
        return self.cols * self.hidden * self.rt.dtype.itemsize

    def cache_request(self):
        return CacheBundle({"state": FixedState((self.heads, self.dim, self.vdim)),
                            "conv": FixedState((self.taps - 1, self.conv_cols)) if self.taps > 1 else None})

    def forward(self, ctx, cache, x, hidden, fresh=False):
        rt, ops = self.rt, self.rt.ops
        n = hidden.shape[0]
        state, conv = cache["state"], cache["conv"]
        proj = rt.buffer("delta_proj", n, self.cols, self.proj_dtype)
        ops.linear(x, self.w_in, proj)
        act = rt.buffer("delta_act", n, self.conv_cols, torch.float32)
        conv_state = conv.state if conv is not None else None
        raw = proj[:, :self.conv_cols]
        # a step of one token a sequence: the convolution's kernel moves its state on itself
        fused = conv_state is not None and conv.writes and bool(ctx.decode_only)
        ops.short_conv(ctx, raw, self.conv_w, conv_state, act, activation="silu", update_state=fused)
        if conv_state is not None and conv.writes and not fused:
            ops.short_conv_state(ctx, raw, conv_state)
        z = None
        if self.inner:
            u = proj[:, self.u_off:self.u_off + self.a_rows + self.g_rows]
            z = rt.buffer("delta_z", n, self.z_cols, torch.float32)
            ops.linear(u, self.w_z, z)
        o = rt.buffer("delta_o", n, self.hv, torch.float32)
        kw = {"channel_logits": z[:, :self.heads * self.dim]} if self.channel else {}
        ops.gated_delta(ctx, act, proj, o, state.state, self.a_log, self.dt_bias, self.heads, self.kv_heads, self.dim,
                        self.vdim, q_off=0, k_off=self.qk, v_off=2 * self.qk, a_off=self.a_off, b_off=self.b_off,
                        q_scale=self.q_scale, **kw)
        gated = rt.buffer("delta_gated", n, self.hv, rt.dtype)
        gate = z[:, self.z_gate:self.z_gate + self.hv] if self.low_rank_gate else proj[:, self.g_off:self.g_off + self.hv]
        ops.group_gate_norm(o, self.norm_w, gate, gated, self.eps, self.heads, self.vdim, act=self.gate_act)
        ops.linear(gated, self.w_o, hidden, residual=None if fresh else hidden)
