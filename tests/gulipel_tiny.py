"""Tiny Gulipel configurations for the tests, and random weights for them.

They differ from one another in every size and option, and avoid coincidences: key and value widths differ,
query heads share key/value heads in different ratios (also one to one, also all on one), on the delta rule's side
too; Mamba-2 heads share one group, several, or have one each, and are normed in parts that do and do not follow the
heads; states have 4 to 160 rows, convolutions 1 to 5 taps (the delta rule also without), inner widths of decay and gate
differ; layers with and without a feed-forward come in every order; embeddings with and without a scale and a pair
table, with a prime and a round number of rows; logits capped or not; token inputs of different widths or none; a query
temperature that steps every few tokens, or none."""
import torch

from leone_b200.config.gulipel import GulipelConfig
from leone_b200.engine.model import weight_specs_for_config
from leone_b200.registry import config_from_dict
from leone_b200.weights.random_init import random_tensors


def left(heads, kv_heads, dim, vdim, scale, temp=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        out["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return out


def right(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
           "gate_rank": gate_rank}
    if not conv:
        out.pop("conv")
    return out


def parallel(lf, rg, ff=None, name="parallel"):
    return _entry(name, {"left": lf, "right": rg}, ff)


def mamba(heads, vdim, state, groups, norm_groups, conv, ff=None, name="mamba2"):
    return _entry(name, {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                         "conv": conv}, ff)


def _entry(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(vocab, width, eps, layers, positions=512, scale=None, bigram=None, side=None, cap=None):
    raw = {"architecture": "Gulipel", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
           "layers": layers}
    emb = {}
    if scale:
        emb["scale"] = scale
    if bigram:
        emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if emb:
        raw["embedding"] = emb
    if side:
        raw["token_side"] = {"dim": side}
    if cap:
        raw["logit_softcap"] = cap
    return raw


TINY = {
    # every kind of layer, a second set of Mamba-2 sizes; pages of 4
    "A": model(97, 64, 1e-5, scale=2.5, bigram=(53, 31, 5), side=8, cap=9.0, layers=[
        mamba(4, 16, 12, 2, 2, 4, ff=40),
        parallel(left(6, 2, 16, 24, 0.3, (0.4, 7)), right(4, 2, 12, 20, 3, 5, 7), ff=56),
        mamba(6, 8, 20, 3, 4, 2, ff=24, name="mamba2_2"), mamba(4, 16, 12, 2, 2, 4)]),
    # sizes that no vector load fits, no scale, no cap, no pairs, one tap, no convolution beside the attention; pages of 8
    "B": model(101, 50, 3e-6, side=3, layers=[
        parallel(left(3, 1, 6, 7, 0.5, (1.5, 3)), right(3, 3, 5, 9, 0, 3, 2)),
        mamba(3, 7, 5, 1, 3, 1, ff=13), mamba(5, 6, 9, 5, 1, 5),
        parallel(left(4, 4, 10, 6, 0.4), right(6, 2, 7, 4, 2, 9, 1), ff=22, name="parallel_2")]),
    # head sizes of real models; the state in the kernels' chunked forms; pages of 16
    "C": model(256, 128, 1e-6, scale=0.7, bigram=(64, 127, 7), side=16, cap=20.0, layers=[
        mamba(4, 64, 128, 2, 2, 4, ff=192), mamba(8, 32, 64, 1, 8, 3, ff=96, name="mamba2_3"),
        parallel(left(8, 2, 64, 64, 0.125, (0.1, 64)), right(2, 1, 64, 128, 4, 16, 24), ff=192),
        mamba(4, 64, 128, 2, 2, 4), parallel(left(2, 2, 128, 32, 0.09, (2.0, 50)), right(4, 4, 32, 32, 3, 8, 8))]),
    # wide recurrent heads, heads that share every group, 18 query heads, no token inputs; pages of 32
    "D": model(200, 96, 2e-6, scale=11.0, bigram=(1, 3, 2), cap=50.0, layers=[
        parallel(left(18, 6, 16, 48, 0.2, (0.7, 33)), right(1, 1, 144, 40, 4, 12, 20)),
        mamba(2, 40, 160, 1, 1, 4, ff=64), mamba(12, 20, 24, 4, 6, 3, ff=72, name="mamba2_2")]),
}
PAGE_TOKENS = {"A": 4, "B": 8, "C": 16, "D": 32}


def tiny_config(which) -> GulipelConfig:
    return config_from_dict(TINY[which])


def tiny_tensors(which, seed=None, gain=4.0, raw=None):
    """fp32 random tensors; tables and matrices are scaled up so that scores, decays, gates and both tables' rows matter
    to the logits.  (B's narrow heads nearly cancel at some positions, which magnifies rounding; with its seed
    rounding alone moves no logit of the tests' requests by more than a few per cent.)"""
    seed = {"B": 6}.get(which, 5) if seed is None else seed
    specs = weight_specs_for_config(config_from_dict(raw) if raw is not None else tiny_config(which))
    tensors = random_tensors(specs, seed)
    for name, t in tensors.items():
        if name in ("embed", "bigram", "pos"):
            tensors[name] = t * 30.0
        elif name == "side.embed":
            tensors[name] = t * 60.0
        elif name.endswith((".a1", ".a2", ".g1", ".g2")):
            tensors[name] = t * 12.0
        elif t.dim() == 2 and not name.endswith(".conv"):
            tensors[name] = t * gain
    return tensors


def as_bf16(tensors):
    return {k: v.to(torch.bfloat16).float() for k, v in tensors.items()}
