"""Dense SwiGLU feed-forward: ``hidden += W_down (silu(W_gate x) * W_up x)``.

``silu(g) = g / (1 + exp(-g))`` in fp32 (crates/leone/src/cpu.rs:903-905);
order of operations crates/leone/src/runtime.rs:9298-9317.  Gate and up
matrices are stacked row-wise at load time so one product feeds both
(the reference pairs them in one launch too, ie_cuda.cu:1896-1931).

The gate's shape is this part's own parameters, for gated layers of the same family:
``y = g' * sigmoid(gate_slope * g' * (1 + gate_cubic * g'^2)) * (u' + up_shift)`` with ``g' = min(g, limit)``
and ``u' = clamp(u, -limit, limit)``.  The defaults (``gate_slope = 1``, no ``limit``, ``up_shift`` and
``gate_cubic`` 0) are SwiGLU.  ``activation = "gelu_tanh"`` sets the slope and the cubic term to gelu's tanh form
(GeGLU): ``z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))) = z sigmoid(2 sqrt(2/pi) z (1 + 0.044715 z^2))``.
``bias = True``: all three projections have biases (tensors ``<name>.b`` by default), added to their sums in the products.
"""
from __future__ import annotations

import math

from ..registry import FEED_FORWARDS
from .base import DeferredNorm, FeedForward, WeightSpec


@FEED_FORWARDS.register("swiglu")
class SwiGLU(FeedForward):
    accepts_deferred_norm = True
    fuses_following_norm = True
    writes_fresh = True           # forward(..., fresh=True) stores its result instead of adding it

    def __init__(self, params, rt):
        super().__init__(params, rt)
        self.hidden = int(params["hidden_size"])
        self.inter = int(params["intermediate_size"])
        self.gate_name = params.get("gate_name", "gate_proj.weight")
        self.up_name = params.get("up_name", "up_proj.weight")
        self.down_name = params.get("down_name", "down_proj.weight")
        self.bias = bool(params.get("bias", False))
        self.bias_names = {k: params.get(f"{k}_bias_name", f"{n}.b") for k, n in
                           (("gate", self.gate_name), ("up", self.up_name), ("down", self.down_name))}
        self.w_gate_up = None
        self.w_down = None
        activation = params.get("activation", "silu")
        if activation not in ("silu", "gelu_tanh"):
            raise ValueError(f"a gated layer's activation is silu or gelu_tanh, not '{activation}'")
        if activation == "gelu_tanh" and ("gate_slope" in params or "gate_cubic" in params):
            raise ValueError("a gated layer's activation gelu_tanh sets the gate's slope and cubic term itself")
        slope, cubic = (2.0 * math.sqrt(2.0 / math.pi), 0.044715) if activation == "gelu_tanh" else \
            (float(params.get("gate_slope", 1.0)), float(params.get("gate_cubic", 0.0)))
        limit, shift = params.get("limit"), float(params.get("up_shift", 0.0))
        if limit is not None and not float(limit) > 0.0:
            raise ValueError(f"a gated layer's limit must be positive, got {limit}")
        # None: plain SwiGLU (the kernels' default); else (slope, limit, shift, cubic) with limit = inf for none
        self.gate_shape = None if (slope == 1.0 and limit is None and shift == 0.0 and cubic == 0.0) else \
            (slope, float("inf") if limit is None else float(limit), shift, cubic)

    def weight_specs(self):
        specs = [WeightSpec(self.gate_name, (self.inter, self.hidden)),
                 WeightSpec(self.up_name, (self.inter, self.hidden)),
                 WeightSpec(self.down_name, (self.hidden, self.inter))]
        if self.bias:
            b = self.bias_names
            specs += [WeightSpec(b["gate"], (self.inter,), role="vector", std=0.5),
                      WeightSpec(b["up"], (self.inter,), role="vector", std=0.5),
                      WeightSpec(b["down"], (self.hidden,), role="vector", std=0.5)]
        return specs

    def load(self, tensors):
        if self.bias:
            gate_b, up_b, down_b = (tensors[self.bias_names[k]].float().contiguous() for k in ("gate", "up", "down"))
            self.w_gate_up = self.rt.ops.prepare_gate_up(tensors[self.gate_name], tensors[self.up_name], gate_b, up_b)
            self.w_down = self.rt.ops.prepare_matrix(tensors[self.down_name], down_b)
            return
        self.w_gate_up = self.rt.ops.prepare_gate_up(tensors[self.gate_name], tensors[self.up_name])
        self.w_down = self.rt.ops.prepare_matrix(tensors[self.down_name])

    def weight_bytes(self):
        return (2 * self.inter * self.hidden + self.hidden * self.inter) * self.rt.dtype.itemsize

    def scratch_bytes(self, max_tokens):
        # the activation; a path without the fused epilogue also holds gate and up side by side
        return max_tokens * 3 * self.inter * self.rt.dtype.itemsize

    def load_transient_bytes(self):
        return 2 * self.inter * self.hidden * self.rt.dtype.itemsize       # gate and up beside their interleaved copy

    def forward(self, ctx, x, hidden, then=None, fresh=False):
        n = hidden.shape[0]
        ops = self.rt.ops
        act = self.rt.buffer("ffn_act", n, self.inter, self.rt.dtype)
        kw = {} if self.gate_shape is None else {"gate_shape": self.gate_shape}
        if isinstance(x, DeferredNorm):
            if x.ready and ops.linear_fuses_norm(n, self.w_gate_up):
                ops.linear_swiglu(x.xn, self.w_gate_up, act, norm_in=x, **kw)      # the norm's factor in the epilogue
            else:
                ops.linear_swiglu(x.materialize(), self.w_gate_up, act, **kw)
        else:
            ops.linear_swiglu(x, self.w_gate_up, act, **kw)
        if then is not None and hasattr(ops, "linear_fuses_norm") and ops.linear_fuses_norm(n, self.w_down):
            then.prepare(self.rt, ops.norm_parts(n, self.hidden))
            ops.linear(act, self.w_down, hidden, residual=hidden, norm_out=then)
            then.ready = True
        else:
            ops.linear(act, self.w_down, hidden, residual=None if fresh else hidden)
