"""A plain, slow implementation of the Kakirax decoder for the tests.

Whole sequences, no cache, no batching, one function per mechanism, float64 by default.  It shares
no code with ``leone_b200``: it takes the raw ``config.json`` mapping and a dict of tensors under the
checkpoint's names.  Notation: ``h`` is a sublayer's input ``[T, width]``; ``W["foo"]`` is the tensor
``<layer>.mix.foo`` or ``<layer>.mlp.foo``.

The design: scaled embeddings; pre-norm layers ``x <- x + mixer(norm1(x))``, ``x <- x + ff(norm2(x))``
(the second half only where a layer has a feed-forward) whose norms are layer norms with weight and
bias; two mixers, grouped softmax attention (per-head RMS norm of q and k, half-split rotation with
frequencies scaled by wavelength, an elementwise output gate) and gated linear attention (a state per
head that every key channel decays at its own, token-dependent rate); a gated feed-forward with
gelu; a layer may run another layer's tensors; the head is the embedding table, its logits soft-capped.
"""
from __future__ import annotations

import math

import torch

DT = torch.float64


def linear(x, w):
    return x @ w.t()


def layer_norm(x, w, b, eps):
    mean = x.mean(dim=-1, keepdim=True)
    var = ((x - mean) ** 2).mean(dim=-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * w + b


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
    """Per pair the angle per position.  With ``scaling`` a pair's frequency is judged by its wavelength:
    short ones stay, long ones are divided by ``factor``, those between are blended."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate(x, positions, rot, angle_dtype=torch.float32):
    """``x``: [T, heads, dim]; element i of the first ``dims`` turns with element i + dims/2."""
    dims = int(rot["dims"])
    half = dims // 2
    f = torch.tensor(frequencies(rot), dtype=torch.float64).to(angle_dtype)
    ang = torch.as_tensor(positions).to(angle_dtype)[:, None] * f[None, :]
    cos, sin = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * cos - v * sin
    out[..., half:dims] = v * cos + u * sin
    return out


def causal_softmax(scores):
    """``scores``: [H, T, T]; softmax over j <= i."""
    T = scores.shape[-1]
    i = torch.arange(T)
    return torch.softmax(scores.masked_fill(~(i[None, :] <= i[:, None])[None], float("-inf")), dim=-1)


def attention(h, W, cfg, eps, cache_round=None):
    T = h.shape[0]
    H, G, d, dv = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"]), int(cfg["vdim"])
    q = linear(h, W["q"]).reshape(T, H, d)
    k = linear(h, W["k"]).reshape(T, G, d)
    v = linear(h, W["v"]).reshape(T, G, dv)
    q, k = rms(q, eps) * W["q.norm"], rms(k, eps) * W["k.norm"]
    if cfg.get("rot"):
        q, k = rotate(q, list(range(T)), cfg["rot"]), rotate(k, list(range(T)), cfg["rot"])
    if cache_round is not None:
        k, v = cache_round(k), cache_round(v)
    kh = k.repeat_interleave(H // G, dim=1)          # query head h uses key/value head h // (H/G)
    vh = v.repeat_interleave(H // G, dim=1)
    w = causal_softmax(torch.einsum("ihd,jhd->hij", q, kh) * float(cfg["scale"]))
    o = torch.einsum("hij,jhv->ihv", w, vh).reshape(T, H * dv)
    return linear(o * torch.sigmoid(linear(h, W["g"])), W["o"])


def channel_decay(h, W, tau):
    """``[T, heads * dim]``: what a state row keeps, ``sigmoid(z)^(1/tau)``."""
    z = linear(linear(h, W["a1"]), W["a2"]) + W["a2.b"]
    return torch.sigmoid(z) ** (1.0 / tau)


def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha: [T, H, d]; v: [T, H, dv].  Returns o [T, H, dv] and the last state [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gated_linear_attention(h, W, cfg, eps):
    T = h.shape[0]
    H, d, dv = int(cfg["heads"]), int(cfg["dim"]), int(cfg["vdim"])
    q = linear(h, W["q"]).reshape(T, H, d) * d ** -0.5
    k = linear(h, W["k"]).reshape(T, H, d)
    v = linear(h, W["v"]).reshape(T, H, dv)
    alpha = channel_decay(h, W, float(cfg["tau"])).reshape(T, H, d)
    o, _ = gla_recurrence(q, k, v, alpha)
    o = (rms(o, eps) * W["norm"]).reshape(T, H * dv)
    return linear(o * silu(linear(h, W["g"])), W["o"])


def feed_forward(h, W):
    return linear(gelu_tanh(linear(h, W["gate"])) * linear(h, W["up"]), W["down"])


class PlainKakirax:
    """``cache_round`` rounds what the attention layers' cache holds, ``read_round`` what the sublayers
    read of the norms (both for comparison with a bfloat16 run)."""

    def __init__(self, config, tensors, dtype=DT, cache_round=None, read_round=None):
        self.config = config
        self.W = {k: v.to(dtype) for k, v in tensors.items()}
        self.cache_round, self.read_round = cache_round, read_round
        self._seen = {}

    def source(self, i):
        """The layer whose tensors layer ``i`` runs."""
        j = self.config["layers"][i].get("weights_of")
        return i if j is None else self.source(int(j))

    def _part(self, prefix):
        return {k[len(prefix):]: v for k, v in self.W.items() if k.startswith(prefix)}

    def _norm(self, x, name):
        y = layer_norm(x, self.W[name], self.W[name + ".b"], float(self.config["norm"]["eps"]))
        return y if self.read_round is None else self.read_round(y)

    def layer(self, x, i):
        entry, p = self.config["layers"][i], f"l{self.source(i)}."
        eps = float(self.config["norm"]["eps"])
        h, W = self._norm(x, p + "norm1"), self._part(p + "mix.")
        if entry["type"] == "attention":
            x = x + attention(h, W, entry["mixer"], eps, self.cache_round)
        else:
            x = x + gated_linear_attention(h, W, entry["mixer"], eps)
        if entry.get("mlp"):
            x = x + feed_forward(self._norm(x, p + "norm2"), self._part(p + "mlp."))
        return x

    def residuals(self, tokens):
        """The residual stream after every layer."""
        scale = float(self.config.get("embedding", {}).get("scale", 1.0))
        x = self.W["embed"][torch.as_tensor(list(tokens))] * scale
        out = []
        for i in range(len(self.config["layers"])):
            x = self.layer(x, i)
            out.append(x)
        return out

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self._seen:
            x = self._norm(self.residuals(tokens)[-1], "final.norm")
            z = linear(x, self.W["embed"])
            cap = self.config.get("logit_softcap")
            self._seen[key] = z if not cap else float(cap) * torch.tanh(z / float(cap))
        return self._seen[key]
