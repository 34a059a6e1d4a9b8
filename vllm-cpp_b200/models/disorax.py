"""Disorax: from its typed configuration to a model description.

A decoder whose layers are listed one by one in config.json; in each the mixer and the feed-forward run side by side,
both on the stream as the layer found it but each behind a norm of its own, and their results' sum enters the stream
times a constant.  Three mixer types: "attention" -- grouped-query softmax attention under a sliding window that keeps a
request's first tokens, part of every q and k head turned in halves, the values mixed with those that the first such
layer made of the same token, a gate per output lane; "latent_attention" -- keys and values expanded from one normed
latent per token, no positions, a gate per head; "latent_attention_2" -- the same under a sliding window, with a learned
score per head of a silent key in the softmax.  The feed-forward is routed SiLU-gated experts whose weights are the
softmax over the chosen logits, beside a shared expert that every token runs behind a gate of its own.  Final norm,
untied head.

Tensor names: ``embed``, ``head``, ``final.norm``; layer i under ``l<i>.``: ``norm1``, ``norm2``; attention
``mix.{q,k,v,g,o}`` and, where values are mixed, ``mix.vmix``; latent attention ``mix.{q,dkv,dkv.norm,uk,uv,g,o}`` and, of
the second type, ``mix.sink``; experts ``mlp.router``, ``mlp.router.b``, ``mlp.e<j>.{gate,up,down}``,
``mlp.shared.{gate,up,down,sg}``.
This file only writes data.
"""
from __future__ import annotations

from ..config.base import ConfigError
from ..config.disorax import DisoraxConfig
from ..registry import LayerRun, LayerSpec, ModelSpec, PartSpec, register_architecture


def _attention(cfg: DisoraxConfig, m, first: bool) -> PartSpec:
    return PartSpec("rotary_window_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
        "scale": m.scale, "window": m.window, "keep_first": m.keep_first, "rope_base": m.rope_base, "rotary_dim": m.rope_dims,
        "pairing": "half", "eps": cfg.norm_eps, "lane_gate": True, "pad_heads": True,
        "value_mix": ("first" if first else "mixed") if m.v_mix else ""})


def _latent(cfg: DisoraxConfig, m, sink: bool) -> PartSpec:
    return PartSpec("latent_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": 0, "v_head_dim": m.vdim, "q_rank": 0,
        "kv_rank": m.kv_rank, "scale": m.scale, "window": m.window, "eps": cfg.norm_eps, "head_gate": True, "sink": sink})


# layer type -> its mixer's description (from the configuration, the mixer's numbers, and whether it is the first layer
# whose values are mixed into later ones)
MIXERS = {"attention": _attention,
          "latent_attention": lambda cfg, m, first: _latent(cfg, m, False),
          "latent_attention_2": lambda cfg, m, first: _latent(cfg, m, True)}


def describe_disorax(cfg: DisoraxConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "name": ""})
    block = PartSpec("parallel", {"result_scale": cfg.residual_mult})
    first_mixing = next((i for i, l in enumerate(cfg.layers) if getattr(l.mixer, "v_mix", False)), -1)
    layers = []
    for i, layer in enumerate(cfg.layers):
        if layer.type not in MIXERS:
            raise ConfigError(f"layer {i}: no mixer of type '{layer.type}' (known: {sorted(MIXERS)})")
        parts = {"norm1": (norm, "norm1"), "mixer": (MIXERS[layer.type](cfg, layer.mixer, i == first_mixing), "mix.")}
        mlp = layer.mlp
        if mlp is None:      # its checkpoint may hold a second norm all the same: nothing reads it
            parts["norm2"] = (PartSpec("rmsnorm", {**norm.params, "unused": True}), "norm2")
        else:
            parts["norm2"] = (norm, "norm2")
            parts["feed_forward"] = (PartSpec("routed_experts", {
                "hidden_size": cfg.width, "num_experts": mlp.experts, "top": mlp.top, "expert_size": mlp.ff,
                "shared_size": mlp.shared_ff, "activation": "silu", "gated": True, "shared_gated": True, "shared_gate": True,
                "router_weights": "softmax", "router_bias": True, "weight_on": "output"}), "mlp.")
        layers.append(LayerSpec(prefix=f"l{i}.", block=block, parts=parts))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_positions, embed_tensor="embed",
        layers=tuple(layers), order=tuple(LayerRun(layer=i, cache=i) for i in range(len(layers))), final_norm=norm,
        final_norm_prefix="final.norm", lm_head_tensor="head")


register_architecture("Disorax", DisoraxConfig, describe_disorax)
