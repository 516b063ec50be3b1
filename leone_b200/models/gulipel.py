"""The Gulipel decoder as a :class:`ModelSpec`.

The stream starts as ``token_embedding`` with a scale, a row chosen by the pair (previous token, token) and a learned
position row.  Every layer is the ``sandwich_norm`` arrangement: RMS norms ``norm1`` / ``norm2`` before the sublayers,
``norm1b`` / ``norm2b`` (with the layer scales ``ls1`` / ``ls2`` in their gains) on what they give back, and after the
feed-forward the layer's ``token_gate``, which gates its slice of the token's row of a second table.

Mixer type ``parallel`` is ``side_by_side`` with the normed mean: ``attention`` (biases, per-head q/k norm, a query
temperature that grows with the position, an elementwise output gate, no rotation) and ``gated_delta_rule`` with a decay
per key channel and a low-rank sigmoid gate.  Mixer type ``mamba2`` is the part of that name.  The feed-forward is
``swiglu`` with biases; the head has a matrix of its own and soft-caps its logits.

Tensor names: ``embed``, ``bigram``, ``pos``, ``side.embed``, ``l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2``,
``l<i>.mix.left.q|k|v|q.b|k.b|v.b|q.norm|k.norm|g|o|out``, ``l<i>.mix.right.q|k|v|q.conv|k.conv|v.conv|b|A_log|norm|a1|a2|
dt_bias|g1|g2|o|out``, ``l<i>.mix.in|conv|conv.b|dt_bias|A_log|D|norm|o``, ``l<i>.mlp.gate|up|down`` and ``.b`` of each,
``l<i>.side.gate|proj|norm``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.gulipel import DEFAULT_RANK, GulipelConfig, ParallelMixer
from ..parts.spec import LayerSpec, ModelSpec, PartSpec
from ..registry import ARCHITECTURES

SIDE_TABLE = "side.embed"


def build_spec(cfg: GulipelConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.norm_eps

    def norm(name, **more):
        return PartSpec("rms_norm", {"size": width, "eps": eps, "name": name, **more})

    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if isinstance(m, ParallelMixer):
            lf, rg = m.left, m.right
            left = {"hidden_size": width, "num_heads": lf.heads, "num_kv_heads": lf.kv_heads, "head_dim": lf.dim,
                    "value_head_dim": lf.vdim, "scale": lf.scale, "qk_norm": True, "qk_norm_eps": eps, "bias": True,
                    "query_temp": None if lf.q_temp is None else lf.q_temp.to_json(), "gate_name": "mix.left.g",
                    **{f"{k}_name": f"mix.left.{k}" for k in ("q", "k", "v", "o")},
                    "q_norm_name": "mix.left.q.norm", "k_norm_name": "mix.left.k.norm"}
            right = {"hidden_size": width, "heads": rg.heads, "kv_heads": rg.kv_heads, "dim": rg.dim, "vdim": rg.vdim,
                     "conv_taps": rg.conv, "norm_eps": eps, "decay": "channel", "gate": "low_rank", "gate_act": "sigmoid",
                     "projections": "run", "decay_rank": rg.decay_rank or DEFAULT_RANK, "gate_rank": rg.gate_rank or DEFAULT_RANK,
                     **{f"{k}_name": f"mix.right.{k}" for k in ("q", "k", "v", "b", "o", "norm", "A_log", "dt_bias", "a1", "a2",
                                                               "g1", "g2")}}
            mixer = PartSpec("side_by_side", {"combine": "normed_mean", "hidden_size": width, "norm_eps": eps, "branches": [
                {"name": "left", "kind": "attention", "params": left, "norm_name": "mix.left.out"},
                {"name": "right", "kind": "gated_delta_rule", "params": right, "norm_name": "mix.right.out"}]})
        else:
            mixer = PartSpec("mamba2", {
                "hidden_size": width, "heads": m.heads, "vdim": m.vdim, "n_state": m.state, "groups": m.groups,
                "norm_groups": m.norm_groups, "conv_taps": m.conv, "norm_eps": eps,
                **{f"{k}_name": f"mix.{k}" for k in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}})
        extra = {"mixer_out_norm": ("norm", norm("norm1b", scale_name="ls1"))}
        ffn = None
        if layer.mlp is not None:
            ffn = PartSpec("swiglu", {"hidden_size": width, "intermediate_size": layer.mlp.ff, "bias": True,
                                      "gate_name": "mlp.gate", "up_name": "mlp.up", "down_name": "mlp.down"})
            extra["ffn_out_norm"] = ("norm", norm("norm2b", scale_name="ls2"))
        if cfg.side_dim:
            extra["after"] = ("feed_forward", PartSpec("token_gate", {
                "hidden_size": width, "dim": cfg.side_dim, "offset": i * cfg.side_dim, "table": SIDE_TABLE,
                "norm_eps": eps, "gate_name": "side.gate", "proj_name": "side.proj", "norm_name": "side.norm"}))
        layers.append(LayerSpec(prefix=f"l{i}", block="sandwich_norm", mixer=mixer, feed_forward=ffn, mixer_norm=norm("norm1"),
                                ffn_norm=None if ffn is None else norm("norm2"), extra=extra))
    embedding = {"name": "embed", "scale": cfg.embedding_scale, "places": {"name": "pos", "positions": cfg.max_positions}}
    if cfg.bigram is not None:
        embedding["pairs"] = {"name": "bigram", **cfg.bigram.to_json()}
    if cfg.side_dim:
        embedding["side_tables"] = [{"name": SIDE_TABLE, "width": cfg.side_dim * len(cfg.layers)}]
    spec = ModelSpec(
        architecture=cfg.architecture, hidden_size=width, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding_name="embed", layers=tuple(layers), run_order=tuple(range(len(layers))), final_norm=norm("final.norm"),
        final_norm_name="final.norm", lm_head_name="head", embedding=PartSpec("token_embedding", embedding),
        head=PartSpec("linear_head", {"name": "head", "soft_cap": cfg.logit_softcap or None}))
    spec.validate()
    return spec


ARCHITECTURES.add(GulipelConfig.ARCHITECTURE, GulipelConfig, build_spec)
