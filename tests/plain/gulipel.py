"""A plain, slow implementation of the Gulipel decoder for the tests.

Whole sequences, no cache, no batching, one function per mechanism, float64 by default.  It shares
no code with ``leone_b200``: it takes the raw ``config.json`` mapping and a dict of tensors under the
checkpoint's names.  Notation: ``h`` is a sublayer's input ``[T, width]``; ``W["foo"]`` is the tensor
``<layer>.mix.foo`` or ``<layer>.mlp.foo``.

The design: a token's row (scaled) plus a row chosen by the pair of the previous token and this one plus a
row for the position; layers ``x <- x + ls1 * norm1b(mixer(norm1(x)))``, ``x <- x + ls2 * norm2b(ff(norm2(x)))``
with RMS norms on both sides of every sublayer and an elementwise scale, then a gated term made from the
layer's slice of a second token table; mixers: a Mamba-2 recurrence (one decay per head), or softmax
attention (biases, q/k norm, a temperature that grows with the position, an output gate, no rotation) beside a
delta-rule recurrence whose state rows decay each at its own rate, their normed outputs averaged; a gated
feed-forward with biases; an output matrix of its own and soft-capped logits.
"""
from __future__ import annotations

import math

import torch

DT = torch.float64


def linear(x, w, b=None):
    y = x @ w.t()
    return y if b is None else y + b


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(x, w, b=None):
    """Causal, per channel: ``y_t = sum_j w[:, j] x_(t - taps + 1 + j)`` with zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * x[:T - back]
    return y if b is None else y + b


# -- the stream before the first layer ----------------------------------------------------------------
def bigram_rows(tokens, bigram):
    """Which row of the pair table every token reads; a sequence's first token reads the last row."""
    buckets, a, b = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    return [buckets if i == 0 else (int(tokens[i - 1]) * a + int(t) * b) % buckets for i, t in enumerate(tokens)]


def embed(tokens, W, cfg):
    emb = cfg.get("embedding", {})
    x = W["embed"][torch.as_tensor(list(tokens))] * float(emb.get("scale", 1.0))
    if emb.get("bigram"):
        x = x + W["bigram"][torch.tensor(bigram_rows(tokens, emb["bigram"]))]
    return x + W["pos"][:len(tokens)]


# -- attention ----------------------------------------------------------------------------------------
def query_temperature(T, q_temp, dtype):
    every, coef = int(q_temp["every"]), float(q_temp["coef"])
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in range(T)], dtype=dtype)


def causal_softmax(scores):
    """``scores``: [H, T, T]; softmax over j <= i."""
    i = torch.arange(scores.shape[-1])
    return torch.softmax(scores.masked_fill(~(i[None, :] <= i[:, None])[None], float("-inf")), dim=-1)


def attention(h, W, cfg, eps, cache_round=None):
    T = h.shape[0]
    H, G, d, dv = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"]), int(cfg["vdim"])
    q = linear(h, W["q"], W["q.b"]).reshape(T, H, d)
    k = linear(h, W["k"], W["k.b"]).reshape(T, G, d)
    v = linear(h, W["v"], W["v.b"]).reshape(T, G, dv)
    q, k = rms(q, eps) * W["q.norm"], rms(k, eps) * W["k.norm"]
    if cfg.get("q_temp"):
        q = q * query_temperature(T, cfg["q_temp"], q.dtype)[:, None, None]
    if cache_round is not None:
        k, v = cache_round(k), cache_round(v)
    kh = k.repeat_interleave(H // G, dim=1)          # query head h uses key/value head h // (H/G)
    vh = v.repeat_interleave(H // G, dim=1)
    w = causal_softmax(torch.einsum("ihd,jhd->hij", q, kh) * float(cfg["scale"]))
    o = torch.einsum("hij,jhv->ihv", w, vh).reshape(T, H * dv)
    return linear(o * torch.sigmoid(linear(h, W["g"])), W["o"])


# -- the delta rule with a decay per key channel --------------------------------------------------------
def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def channel_decay(h, W, heads, dim):
    """``[T, heads, dim]``: what every state row keeps of itself."""
    z = linear(linear(h, W["a1"]), W["a2"]) + W["dt_bias"]
    return torch.exp(-torch.exp(W["A_log"])[None, :, None] * softplus(z).reshape(-1, heads, dim))


def delta_recurrence(q, k, v, g, beta, state=None):
    """q, k, g: [T, H, d]; v: [T, H, dv]; beta: [T, H].  Returns o [T, H, dv] and the last state [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def delta_rule(h, W, cfg, eps, act_round=None):
    T = h.shape[0]
    H, G, d, dv = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"]), int(cfg["vdim"])
    acts = []
    for name in ("q", "k", "v"):
        x = linear(h, W[name])
        if act_round is not None:
            x = act_round(x)
        if f"{name}.conv" in W:
            x = short_conv(x, W[f"{name}.conv"])
        x = silu(x)
        acts.append(x if act_round is None else act_round(x))
    q = (unit(acts[0].reshape(T, G, d)) * d ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(acts[1].reshape(T, G, d)).repeat_interleave(H // G, dim=1)
    v = acts[2].reshape(T, H, dv)
    o, _ = delta_recurrence(q, k, v, channel_decay(h, W, H, d), torch.sigmoid(linear(h, W["b"])))
    o = (rms(o, eps) * W["norm"]).reshape(T, H * dv)
    return linear(o * torch.sigmoid(linear(linear(h, W["g1"]), W["g2"])), W["o"])


def parallel(h, W, cfg, eps, cache_round=None, act_round=None):
    def side(name):
        return {k[len(name) + 1:]: v for k, v in W.items() if k.startswith(name + ".")}
    left = attention(h, side("left"), cfg["left"], eps, cache_round)
    right = delta_rule(h, side("right"), cfg["right"], eps, act_round)
    return 0.5 * (rms(left, eps) * W["left.out"] + rms(right, eps) * W["right.out"])


# -- Mamba-2 --------------------------------------------------------------------------------------------
def ssd_recurrence(x, B, C, dt, rate, state=None):
    """x: [T, H, dv]; B, C: [T, H, N]; dt: [T, H]; rate: [H].  Returns y [T, H, dv] (without the D x term)
    and the last state [H, N, dv]."""
    T, H, dv = x.shape
    S = torch.zeros(H, B.shape[2], dv, dtype=x.dtype) if state is None else state
    out = []
    for t in range(T):
        a = torch.exp(-rate * dt[t])
        S = a[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", S, C[t]))
    return torch.stack(out), S


def grouped_rms(x, groups, eps):
    T, n = x.shape
    return rms(x.reshape(T, groups, n // groups), eps).reshape(T, n)


def mamba2(h, W, cfg, eps, act_round=None):
    T = h.shape[0]
    H, dv, N, G = int(cfg["heads"]), int(cfg["vdim"]), int(cfg["state"]), int(cfg["groups"])
    inner = H * dv
    p = linear(h, W["in"])
    if act_round is not None:
        p = act_round(p)
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, W["conv"], W["conv.b"]) if "conv" in W else xbc)
    if act_round is not None:
        xbc = act_round(xbc)
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N).repeat_interleave(H // G, dim=1)
    C = xbc[:, inner + G * N:].reshape(T, G, N).repeat_interleave(H // G, dim=1)
    y, _ = ssd_recurrence(x, B, C, softplus(dt + W["dt_bias"]), torch.exp(W["A_log"]))
    y = (y + W["D"][None, :, None] * x).reshape(T, inner)
    return linear(grouped_rms(y * silu(z), int(cfg["norm_groups"]), eps) * W["norm"], W["o"])


# -- the rest of a layer ----------------------------------------------------------------------------------
def feed_forward(h, W):
    return linear(silu(linear(h, W["gate"], W["gate.b"])) * linear(h, W["up"], W["up.b"]), W["down"], W["down.b"])


def token_side(x, e, W, eps):
    y = linear(gelu_tanh(linear(x, W["gate"])) * e, W["proj"])
    return rms(y, eps) * W["norm"]


class PlainGulipel:
    """``cache_round`` rounds what the attention layers' cache holds, ``read_round`` what the sublayers read of
    the norms, ``act_round`` a recurrence's projections and activations (all for comparison with a bfloat16 run)."""

    def __init__(self, config, tensors, dtype=DT, cache_round=None, read_round=None, act_round=None):
        self.config = config
        self.eps = float(config["norm"]["eps"])
        self.W = {k: v.to(dtype) for k, v in tensors.items()}
        self.cache_round, self.read_round, self.act_round = cache_round, read_round, act_round
        self._seen = {}

    def _part(self, prefix):
        return {k[len(prefix):]: v for k, v in self.W.items() if k.startswith(prefix)}

    def _norm(self, x, name):
        y = rms(x, self.eps) * self.W[name]
        return y if self.read_round is None else self.read_round(y)

    def mixer(self, h, i):
        entry, W = self.config["layers"][i], self._part(f"l{i}.mix.")
        if entry["type"].startswith("parallel"):
            return parallel(h, W, entry["mixer"], self.eps, self.cache_round, self.act_round)
        return mamba2(h, W, entry["mixer"], self.eps, self.act_round)

    def layer(self, x, i, tokens):
        entry, p, W = self.config["layers"][i], f"l{i}.", self.W
        x = x + rms(self.mixer(self._norm(x, p + "norm1"), i), self.eps) * W[p + "norm1b"] * W[p + "ls1"]
        if entry.get("mlp"):
            y = feed_forward(self._norm(x, p + "norm2"), self._part(p + "mlp."))
            x = x + rms(y, self.eps) * W[p + "norm2b"] * W[p + "ls2"]
        if self.config.get("token_side"):
            dim = int(self.config["token_side"]["dim"])
            e = W["side.embed"][torch.as_tensor(list(tokens))][:, i * dim:(i + 1) * dim]
            r = x if self.read_round is None else self.read_round(x)
            x = x + token_side(r, e, self._part(p + "side."), self.eps)
        return x

    def residuals(self, tokens):
        """The residual stream after every layer."""
        x, out = embed(tokens, self.W, self.config), []
        for i in range(len(self.config["layers"])):
            x = self.layer(x, i, tokens)
            out.append(x)
        return out

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self._seen:
            z = linear(self._norm(self.residuals(tokens)[-1], "final.norm"), self.W["head"])
            cap = self.config.get("logit_softcap")
            self._seen[key] = z if not cap else float(cap) * torch.tanh(z / float(cap))
        return self._seen[key]
