"""The Kakirax decoder as a :class:`ModelSpec`.

Every layer is the ``pre_norm`` arrangement with ``layer_norm`` (weight and bias); a layer without a
feed-forward is its first half only.  Mixer type ``attention`` is the part of that name with per-head q/k
norm, a half-split rotation whose frequencies are scaled by wavelength and an elementwise output gate;
mixer type ``gla`` is ``gated_linear_attention``.  The feed-forward is ``swiglu`` with gelu's tanh form.  A
layer that names another layer's tensors is a further run of that layer (``run_order``), with a cache or
state of its own.  The embedding is scaled; the head is tied (without the scale) and soft-capped.

Tensor names: ``embed``, ``l<i>.norm1|norm2`` and ``l<i>.norm1.b|norm2.b``, attention ``l<i>.mix.q|k|v|q.norm|
k.norm|g|o``, gla ``l<i>.mix.q|k|v|g|a1|a2|a2.b|norm|o``, ``l<i>.mlp.gate|up|down``, ``final.norm``,
``final.norm.b``.
"""
from __future__ import annotations

from ..config.kakirax import DEFAULT_DECAY_RANK, KakiraxConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec
from ..registry import ARCHITECTURES


def build_spec(cfg: KakiraxConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.norm_eps
    encodings = {}

    def norm(name):
        return PartSpec("layer_norm", {"size": width, "eps": eps, "name": name, "bias_name": f"{name}.b"})

    def encoding_for(m):
        if not m.rot_dims:
            return None
        params = {"rotary_dim": m.rot_dims, "base": m.rot_base, "pairing": "half_split",
                  "scaling": None if m.rot_scaling is None else {"kind": "wavelength", **m.rot_scaling.to_json()}}
        for name, ps in encodings.items():
            if ps.params == params:
                return name
        name = f"rot{len(encodings)}"
        encodings[name] = PartSpec("rotary_computed", params)
        return name

    layers, index = [], {}
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        m = layer.mixer
        if layer.type == "attention":
            mixer = PartSpec("attention", {
                "hidden_size": width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                "value_head_dim": m.vdim, "scale": m.scale, "qk_norm": True, "qk_norm_eps": eps,
                "position_encoding": encoding_for(m), "gate_name": "mix.g",
                **{f"{k}_name": f"mix.{k}" for k in ("q", "k", "v", "o")},
                "q_norm_name": "mix.q.norm", "k_norm_name": "mix.k.norm"})
        else:
            mixer = PartSpec("gated_linear_attention", {
                "hidden_size": width, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau,
                "decay_rank": m.decay_rank or DEFAULT_DECAY_RANK, "norm_eps": eps,
                **{f"{k}_name": f"mix.{k}" for k in ("q", "k", "v", "g", "a1", "a2", "o", "norm")}, "a2_bias_name": "mix.a2.b"})
        ffn = None if layer.mlp is None else PartSpec("swiglu", {
            "hidden_size": width, "intermediate_size": layer.mlp.ff, "activation": "gelu_tanh",
            "gate_name": "mlp.gate", "up_name": "mlp.up", "down_name": "mlp.down"})
        index[i] = len(layers)
        layers.append(LayerSpec(prefix=f"l{i}", block="pre_norm", mixer=mixer, feed_forward=ffn, mixer_norm=norm("norm1"),
                                ffn_norm=None if ffn is None else norm("norm2")))
    spec = ModelSpec(
        architecture=cfg.architecture, hidden_size=width, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding_name="embed", layers=tuple(layers),
        run_order=tuple(index[cfg.source_layer(i)] for i in range(len(cfg.layers))), final_norm=norm("final.norm"),
        final_norm_name="final.norm", lm_head_name=None, position_encodings=encodings,
        embedding=PartSpec("token_embedding", {"name": "embed", "scale": cfg.embedding_scale}),
        head=PartSpec("linear_head", {"name": None, "soft_cap": cfg.logit_softcap or None}))
    spec.validate()
    return spec


ARCHITECTURES.add(KakiraxConfig.ARCHITECTURE, KakiraxConfig, build_spec)
