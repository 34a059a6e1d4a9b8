"""A plain, slow implementation of the Nufetar design: float64, whole sequences, one function per mechanism.

It shares no code with the package: its own reading of config.json's keys, its own loops.  A model is a dict of the
configuration (as config.json holds it) and a dict name -> float64 tensor.  ``forward`` returns the logits of every
position and, if asked, the residual stream after every layer.
"""
from __future__ import annotations

import json
import math
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


def softplus(z: float) -> float:
    return math.log1p(math.exp(-abs(z))) + max(z, 0.0)


def xielu(z, p: float, q: float):
    """Two branches that share the slope 1/2 at zero: a parabola above it, an exponential below."""
    above = softplus(p) * z * z + 0.5 * z
    low = torch.clamp(z, max=0.0)
    below = (0.5 + softplus(q)) * (torch.expm1(low) - low) + 0.5 * low
    return torch.where(z > 0, above, below)


def turn(x, positions, base, dims, neighbours):
    """x [T, heads, n]: the first ``dims`` lanes of every head turn by position * base^(-2i/dims); pairs are lanes
    (2i, 2i + 1) with ``neighbours``, else (i, i + dims/2)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        lu, lv = (2 * i, 2 * i + 1) if neighbours else (i, i + dims // 2)
        u, v = x[..., lu], x[..., lv]
        out[..., lu] = u * c - v * s
        out[..., lv] = v * c + u * s
    return out


def window_mask(T, size):
    """[T, T] bool: query i (row) sees key j: 0 <= i - j < size (size 0: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i - j < size) if size else seen


def chunk_mask(T, size):
    """[T, T] bool: query i sees key j <= i of its own chunk; chunks of ``size`` positions, counted from position 0
    (size 0: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i // size == j // size) if size else seen


def masked_softmax(s, mask):
    return torch.softmax(s.masked_fill(~mask, float("-inf")), -1)


def mixed_scores(scores, talk):
    """scores [H, T, T] before the softmax: head h reads sum_g talk[h, g] scores[g]."""
    return torch.einsum("hg,gij->hij", talk, scores)


def unit_values(v, eps):
    """v [T, G, dv]: every head's value divided by its root mean square (no gain)."""
    return rms(v, eps)


def attention(h, w, m, eps, positions):
    """Grouped-query attention within chunks: biases on every projection, rotation in halves, unit values, scores mixed
    across the heads, one output gate per head."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    q = turn((h @ w["q"].T + w["q.b"]).view(T, H, d), positions, base, dims, False)
    k = turn((h @ w["k"].T + w["k.b"]).view(T, G, d), positions, base, dims, False)
    v = unit_values((h @ w["v"].T + w["v.b"]).view(T, G, dv), eps)
    of = torch.arange(H) // (H // G)
    raw = torch.einsum("ihd,jhd->hij", q, k[:, of]) * float(m["scale"])
    weights = masked_softmax(mixed_scores(raw, w["talk"]), chunk_mask(T, int((m.get("mask") or {}).get("size") or 0)))
    o = torch.einsum("hij,jhe->ihe", weights, v[:, of])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T + w["o.b"]


def latent_attention(h, w, m, eps, positions):
    """Keys and values expanded from one normed latent per token, beside one rotated key part that all heads share."""
    T = h.shape[0]
    H, d, r, dv, kr = (int(m[n]) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    base = float(m["rot"]["base"])
    q = (h @ w["q"].T).view(T, H, d + r)
    down = h @ w["dkv"].T
    c = rms(down[:, :kr], eps) * w["dkv.norm"]
    k_rot = turn(down[:, None, kr:], positions, base, r, True)
    q_rot = turn(q[..., d:], positions, base, r, True)
    k = (c @ w["uk"].T).view(T, H, d)
    v = (c @ w["uv"].T).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot[:, 0])) * float(m["scale"])
    weights = masked_softmax(s, window_mask(T, int((m.get("mask") or {}).get("size") or 0)))
    return torch.einsum("hij,jhe->ihe", weights, v).reshape(T, H * dv) @ w["o"].T


def wkv_scan(r, k, v, decay, u, state=None):
    """One head: r, k, decay [T, d], v [T, dv], u [d].  o_t reads the state as it was plus u-weighted k_t v_t^T."""
    T, d = r.shape
    S = torch.zeros(d, v.shape[1], dtype=F64) if state is None else state.clone()
    out = torch.zeros(T, v.shape[1], dtype=F64)
    for t in range(T):
        kv = torch.outer(k[t], v[t])
        out[t] = (S + u[:, None] * kv).T @ r[t]
        S = decay[t][:, None] * S + kv
    return out, S


def shifted(h, mu, before=None):
    """h + (h' - h) mu, h' the row before (``before``, or zeros, for the first)."""
    prev = torch.cat([torch.zeros_like(h[:1]) if before is None else before[None], h[:-1]])
    return h + (prev - h) * mu


def wkv(h, w, m, eps):
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    x = {n: shifted(h, w["mu." + n]) for n in "rkvgw"}
    r, k, v = ((x[n] @ w[n].T).view(T, H, d) for n in "rkv")
    decay = torch.exp(-torch.exp(torch.tanh(x["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).view(T, H, d)
    u = w["u"].view(H, d)
    o = torch.stack([wkv_scan(r[:, i], k[:, i], v[:, i], decay[:, i], u[i])[0] for i in range(H)], 1)
    return (rms(o, eps).reshape(T, H * d) * w["norm"] * silu(x["g"] @ w["g"].T)) @ w["o"].T


def feed_forward(h, w):
    p, q = (float(a) for a in w["act"])
    return xielu(h @ w["up"].T, p, q) @ w["down"].T


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, want_layers=False):
    eps = float(cfg["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(ids))
    x = tensors["embed"][ids].clone()
    after = []
    for i, layer in enumerate(cfg["layers"]):
        w = sub(tensors, f"l{i}.")
        h = rms(x, eps) * w["norm1"]
        mw, m = sub(w, "mix."), layer["mixer"]
        if layer["type"] == "attention":
            x = x + attention(h, mw, m, eps, positions)
        elif layer["type"] == "latent_attention":
            x = x + latent_attention(h, mw, m, eps, positions)
        elif layer["type"] == "wkv":
            x = x + wkv(h, mw, m, eps)
        else:
            raise ValueError(f"layer type {layer['type']}")
        if layer.get("mlp") is not None:
            x = x + feed_forward(rms(x, eps) * w["norm2"], sub(w, "mlp."))
        after.append(x.clone())
    logits = (rms(x, eps) * tensors["final.norm"]) @ tensors["embed"].T
    return (logits, torch.stack(after)) if want_layers else logits


def greedy(cfg, tensors, prompt, n_new):
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(forward(cfg, tensors, seq)[-1].argmax()))
    return seq[len(prompt):]
