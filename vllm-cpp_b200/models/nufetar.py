"""Nufetar: from its typed configuration to a model description.

A pre-norm decoder whose layers are listed one by one in config.json, with three mixer types.  "attention":
grouped-query softmax attention within chunks of positions that stand still, biases on all four projections, part of
every q and k head turned in halves, values divided by their own root mean square, the heads' scores mixed by a learned
matrix before the softmax and every head's sum weighted by a gate of the input.  "latent_attention": keys and values
expanded from one normed latent per token beside a turned key part that all heads share, queries straight from the
input, neighbouring lanes turned, under a sliding window.  "wkv": a recurrence on a matrix per head with a decay per key
channel from a low-rank projection and a bonus for the current token, every projection reading its own mix of the
token's and the previous token's input, a norm per head and an output gate.  The feed-forward is one hidden layer with
an xIELU; the head is the embedding table.

Tensor names: ``embed``, ``final.norm``; layer i under ``l<i>.``: ``norm1``, ``norm2``; attention ``mix.{q,k,v,o}`` each
with ``.b``, ``mix.{talk,g}``; latent_attention ``mix.{q,dkv,dkv.norm,uk,uv,o}``; wkv ``mix.{r,k,v,g,o,w1,w2,w0,u,norm}``,
``mix.mu.{r,k,v,g,w}``; feed-forward ``mlp.{up,down,act}``.
This file only writes data.
"""
from __future__ import annotations

from ..config.base import ConfigError
from ..config.nufetar import NufetarConfig
from ..registry import LayerRun, LayerSpec, ModelSpec, PartSpec, register_architecture


def _attention(cfg: NufetarConfig, m) -> PartSpec:
    return PartSpec("rotary_window_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
        "scale": m.scale, "window": m.chunk, "chunked": True, "rope_base": m.rot.base, "rotary_dim": m.rot.dims,
        "pairing": "half", "eps": cfg.norm_eps, "bias": True, "unit_values": True, "talk": True, "head_gate": True})


def _latent_attention(cfg: NufetarConfig, m) -> PartSpec:
    return PartSpec("latent_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim,
        "q_rank": 0, "kv_rank": m.kv_rank, "scale": m.scale, "window": m.window, "rope_base": m.rot.base,
        "pairing": "interleaved", "eps": cfg.norm_eps})


def _wkv(cfg: NufetarConfig, m) -> PartSpec:
    return PartSpec("wkv", {"hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.dim,
                            "rank": m.rank, "eps": cfg.norm_eps})


MIXERS = {"attention": _attention, "latent_attention": _latent_attention, "wkv": _wkv}
# mixers that compute on their input in 32-bit before a product reads it: their norm hands it on so
READS_32BIT = ("wkv",)


def describe_nufetar(cfg: NufetarConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "name": ""})
    norm32 = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "name": "", "keep_32bit": True})
    layers = []
    for i, layer in enumerate(cfg.layers):
        if layer.type not in MIXERS:
            raise ConfigError(f"layer {i}: no mixer of type '{layer.type}' (known: {sorted(MIXERS)})")
        parts = {"norm1": (norm32 if layer.type in READS_32BIT else norm, "norm1"),
                 "mixer": (MIXERS[layer.type](cfg, layer.mixer), "mix.")}
        if layer.mlp is not None:
            parts["norm2"] = (norm, "norm2")
            parts["feed_forward"] = (PartSpec("dense", {
                "hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "activation": "xielu", "up_tensor": "up",
                "down_tensor": "down", "act_tensor": "act"}), "mlp.")
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("prenorm", {}), parts=parts))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_positions, embed_tensor="embed",
        layers=tuple(layers), order=tuple(LayerRun(layer=i, cache=i) for i in range(len(layers))), final_norm=norm,
        final_norm_prefix="final.norm", lm_head_tensor=None)


register_architecture("Nufetar", NufetarConfig, describe_nufetar)
