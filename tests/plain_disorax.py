"""A plain, slow implementation of the Disorax design: float64, whole sequences, one function per mechanism.

It shares no code with the package: its own reading of config.json's keys, its own loops.  A model is a dict of the
configuration (as config.json holds it) and a dict name -> float64 tensor.  ``forward`` returns the logits of every
position and, if asked, the residual stream after every layer.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

from plain_qwen3 import read_safetensors

F64 = torch.float64


def read_model(model_dir):
    model_dir = Path(model_dir)
    return json.loads((model_dir / "config.json").read_text()), read_safetensors(model_dir / "model.safetensors")


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def turn_halves(x, positions, base, dims):
    """x [T, heads, n]: lanes (i, i + dims/2) of every head turn by position * base^(-2i/dims), i < dims/2."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i] = u * c - v * s
        out[..., i + dims // 2] = v * c + u * s
    return out


def window_mask(T, size, keep_first=0):
    """[T, T] bool: query i (row) sees key j <= i if i - j < size or j < keep_first (size 0: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & ((i - j < size) | (j < keep_first)) if size else seen


def masked_softmax(s, mask, sink=None):
    """s [H, T, T]; sink [H]: a term exp(sink_h) in head h's denominator that belongs to no key."""
    s = s.masked_fill(~mask, float("-inf"))
    if sink is None:
        return torch.softmax(s, -1)
    top = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def mixed_values(v, lam, first):
    """(1 - lam) v + lam first: a share of the values that an earlier layer made of the same token."""
    return (1.0 - lam) * v + lam * first


def mask_of(m):
    mask = m.get("mask") or {}
    return int(mask.get("size") or 0), int(mask.get("keep_first") or 0)


def attention(h, w, m, positions, first_values=None):
    """Grouped-query attention, rotation in halves, window with kept first keys, values mixed with an earlier layer's,
    a gate per output lane.  -> (result, this layer's values before mixing)."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    q = turn_halves((h @ w["q"].T).view(T, H, d), positions, base, dims)
    k = turn_halves((h @ w["k"].T).view(T, G, d), positions, base, dims)
    own = (h @ w["v"].T).view(T, G, dv)
    v = own if first_values is None else mixed_values(own, w["vmix"].reshape(()), first_values)
    of = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * float(m["scale"])
    o = torch.einsum("hij,jhe->ihe", masked_softmax(s, window_mask(T, *mask_of(m))), v[:, of]).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T, own


def latent_attention(h, w, m, eps, sink=None):
    """Keys and values expanded from one normed latent per token, no positions, a gate per head."""
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w["q"].T).view(T, H, d)
    c = rms(h @ w["dkv"].T, eps) * w["dkv.norm"]
    k = (c @ w["uk"].T).view(T, H, d)
    v = (c @ w["uv"].T).view(T, H, dv)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    o = torch.einsum("hij,jhe->ihe", masked_softmax(s, window_mask(T, *mask_of(m)), sink), v)
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T


def expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z, top):
    """Router logits [T, E] -> (chosen experts [T, top], their weights: the softmax over the chosen logits only)."""
    best, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(best, -1)


def feed_forward(h, w, mlp):
    z = h @ w["router"].T + w["router.b"]
    idx, weight = route(z, int(mlp["router"]["top"]))
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        share = (weight * (idx == e)).sum(-1, keepdim=True)
        out = out + share * expert(h, sub(w, f"e{e}."))
    if mlp.get("shared") is not None:
        s = sub(w, "shared.")
        out = out + torch.sigmoid(h @ s["sg"].T) * expert(h, s)
    return out


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, want_layers=False):
    eps, m_res = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(ids))
    x = tensors["embed"][ids].clone()
    first_values = None
    after = []
    for i, layer in enumerate(cfg["layers"]):
        w = sub(tensors, f"l{i}.")
        h = rms(x, eps) * w["norm1"]
        mw, m = sub(w, "mix."), layer["mixer"]
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, mw, m, positions, first_values if mixes else None)
            if mixes and first_values is None:
                first_values = own
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, mw, m, eps)
        elif layer["type"] == "latent_attention_2":
            y = latent_attention(h, mw, m, eps, mw["sink"])
        else:
            raise ValueError(f"layer type {layer['type']}")
        if layer.get("mlp") is not None:
            y = y + feed_forward(rms(x, eps) * w["norm2"], sub(w, "mlp."), layer["mlp"])
        x = x + m_res * y
        after.append(x.clone())
    logits = (rms(x, eps) * tensors["final.norm"]) @ tensors["head"].T
    return (logits, torch.stack(after)) if want_layers else logits


def greedy(cfg, tensors, prompt, n_new):
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(forward(cfg, tensors, seq)[-1].argmax()))
    return seq[len(prompt):]
