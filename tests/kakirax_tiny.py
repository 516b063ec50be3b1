"""Tiny Kakirax configurations for the tests, and random weights for them.

They differ from one another in every size and option, and avoid coincidences: key and value widths
differ, query heads share key/value heads in different ratios (also one to one, also all on one), rotated
dimensions are all, some or none of a head, with and without scaled frequencies (some pairs kept, some
divided, some blended), decays have inner widths from 3 to 24 and tau from 1 to 20, recurrent heads have 4 to
300 rows and 7 to 200 columns, layers with and without a feed-forward come in every order, layers run other
layers' tensors (also one that runs a layer that runs another, also right after it), embeddings are scaled
or not, logits capped or not."""
import torch

from leone_b200.engine.model import weight_specs_for_config
from leone_b200.registry import config_from_dict
from leone_b200.weights.random_init import random_tensors


def attn(heads, kv_heads, dim, vdim, scale, ff=None, rot_dims=None, base=10000.0, scaling=None, of=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot_dims != 0:
        m["rot"] = {"base": base, "dims": dim if rot_dims is None else rot_dims}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), (float(s) for s in scaling)))
    return _entry("attention", m, ff, of)


def gla(heads, dim, vdim, tau, rank, ff=None, of=None):
    return _entry("gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}, ff, of)


def _entry(kind, mixer, ff, of):
    out = {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if of is not None:
        out["weights_of"] = of
    return out


def model(vocab, width, eps, layers, scale=None, cap=None):
    raw = {"architecture": "Kakirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale:
        raw["embedding"] = {"scale": scale}
    if cap:
        raw["logit_softcap"] = cap
    return raw


_A0 = dict(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.3, rot_dims=8, base=500.0, scaling=(4, 1, 4, 32), ff=40)
_C0 = dict(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.125, base=30000.0, scaling=(8, 1, 4, 128), ff=192)
TINY = {
    # every kind of layer, two of them run again; a partial rotation; pages of 4
    "A": model(97, 64, 1e-5, scale=2.5, cap=9.0, layers=[
        attn(**_A0), gla(3, 12, 20, 4.0, 8, ff=56), attn(**_A0, of=0), gla(2, 20, 36, 2.0, 5), gla(3, 12, 20, 4.0, 8, ff=56, of=1)]),
    # sizes that no vector load fits, tau 1, no rotation, no cap, no scale; a recurrent layer first; pages of 8
    "B": model(101, 50, 3e-6, layers=[
        gla(1, 5, 7, 1.0, 3), attn(3, 1, 6, 7, 0.5, rot_dims=0, ff=13), gla(3, 10, 14, 1.0, 7, ff=22),
        attn(4, 4, 10, 6, 0.4, rot_dims=4, base=50.0)]),
    # head sizes of real models, a layer run twice in a row, one that runs a layer that runs another; pages of 16
    "C": model(256, 128, 1e-6, scale=0.7, cap=20.0, layers=[
        attn(**_C0), gla(2, 64, 128, 16.0, 16, ff=96), gla(2, 64, 128, 16.0, 16, ff=96, of=1), gla(4, 128, 32, 8.0, 24),
        attn(**_C0, of=0), attn(2, 2, 128, 32, 0.09, base=1000.0), gla(2, 64, 128, 16.0, 16, ff=96, of=2)]),
    # wide recurrent heads (the kernel's forms for up to 256 and 512 rows, heads wider than a block), 18 query
    # heads; pages of 32
    "D": model(200, 96, 2e-6, scale=11.0, cap=50.0, layers=[
        gla(1, 144, 40, 12.0, 16), attn(18, 6, 16, 48, 0.2, rot_dims=12, base=200000.0, scaling=(32, 2, 8, 40), ff=64),
        gla(1, 300, 24, 20.0, 4), gla(2, 32, 200, 6.0, 12, ff=72)]),
}
PAGE_TOKENS = {"A": 4, "B": 8, "C": 16, "D": 32}


def tiny_config(which):
    return config_from_dict(TINY[which])


def tiny_tensors(which, seed=5, gain=4.0, raw=None):
    """fp32 random tensors; matrices are scaled up so that scores, decays and gates are far from uniform and
    every mechanism matters to the logits."""
    specs = weight_specs_for_config(config_from_dict(raw) if raw is not None else tiny_config(which))
    tensors = random_tensors(specs, seed)
    for name, t in tensors.items():
        if name == "embed":
            tensors[name] = t * 30.0
        elif name.endswith(".a2"):
            tensors[name] = t * 40.0
        elif name.endswith(".norm1.b") or name.endswith(".norm2.b") or name == "final.norm.b":
            tensors[name] = t * 3.0
        elif t.dim() == 2:
            tensors[name] = t * gain
    return tensors


def as_bf16(tensors):
    return {k: v.to(torch.bfloat16).float() for k, v in tensors.items()}
