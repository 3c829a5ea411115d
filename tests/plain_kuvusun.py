"""A plain, slow implementation of the Kuvusun design: whole sequences, no cache, float64 by default.

One function per mechanism, written from the design's equations in this file's own notation and
sharing no code with the package.  ``forward(config, tensors, tokens)`` runs one sequence and
returns the logits of every position (and, on request, the residual stream after every layer).
``tensors`` maps checkpoint names to torch tensors.

Notation: ``T`` tokens at positions ``0 .. T-1``; linear weights are stored ``[out, in]``.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

DT = torch.float64


def _w(tensors, name):
    return tensors[name].to(DT)


def _map(tensors, name, x):
    return x @ _w(tensors, name).T


# -- small pieces ---------------------------------------------------------------------------


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def part_norm(x, weight, parts, eps):
    """Each of ``parts`` equal consecutive pieces of a row by its own root mean square, then the weight."""
    width = x.shape[-1]
    pieces = [unit_rms(x[..., i * (width // parts) : (i + 1) * (width // parts)], eps) for i in range(parts)]
    return torch.cat(pieces, dim=-1) * weight


def silu(z):
    return z * torch.sigmoid(z)


def turn_halves(x, base, dims):
    """``x`` [T, heads, size >= dims]: dimensions ``i`` and ``i + dims/2`` of position ``p`` turn together
    by ``p * base^(-2i/dims)``; dimensions from ``dims`` on stay."""
    half = dims // 2
    freqs = float(base) ** (-2.0 * torch.arange(half, dtype=DT) / dims)
    ang = torch.arange(x.shape[0], dtype=DT)[:, None, None] * freqs
    c, s = torch.cos(ang), torch.sin(ang)
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def causal_softmax_attention(q, k, v, scale):
    """``q``, ``k`` [T, H, d], ``v`` [T, H, e] -> [T, H, e]; position i sees positions 0 .. i."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    later = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    s = s.masked_fill(later[None], -math.inf)
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, dim=-1), v)


# -- mixers -----------------------------------------------------------------------------------


def latent_entries(h, tensors, prefix, m, eps, turned):
    """What a layer keeps per token: the normed latent [T, R] and, where the mixer turns a part of its
    keys, the turned key part [T, r] that all heads share (``None`` otherwise)."""
    R = m["kv_rank"]
    down = _map(tensors, prefix + "dkv", h)
    c = unit_rms(down[:, :R], eps) * _w(tensors, prefix + "dkv.norm")
    if not turned:
        return c, None
    return c, turn_halves(down[:, None, R:], m["rot"]["base"], m["rot"]["dims"])[:, 0]


def latent_attention(h, tensors, prefix, m, eps, entries):
    """Latent attention without positions, queries through a normed latent of their own."""
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    c, _ = entries
    cq = unit_rms(_map(tensors, prefix + "dq", h), eps) * _w(tensors, prefix + "dq.norm")
    q = _map(tensors, prefix + "uq", cq).view(T, H, d)
    k = _map(tensors, prefix + "uk", c).view(T, H, d)
    v = _map(tensors, prefix + "uv", c).view(T, H, e)
    o = causal_softmax_attention(q, k, v, float(m["scale"]))
    return _map(tensors, prefix + "o", o.reshape(T, H * e))


def turned_latent_attention(h, tensors, prefix, m, eps, entries):
    """Latent attention whose queries and keys have a turned part, with a gate on every output number."""
    T = h.shape[0]
    H, d, r, e = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kt = entries
    q = _map(tensors, prefix + "q", h).view(T, H, d + r)
    qt = turn_halves(q[..., d:], m["rot"]["base"], m["rot"]["dims"])
    k = _map(tensors, prefix + "uk", c).view(T, H, d)
    v = _map(tensors, prefix + "uv", c).view(T, H, e)
    kk = torch.cat([k, kt[:, None, :].expand(T, H, r)], dim=-1)
    o = causal_softmax_attention(torch.cat([q[..., :d], qt], dim=-1), kk, v, float(m["scale"]))
    o = o.reshape(T, H * e) * torch.sigmoid(_map(tensors, prefix + "g", h))
    return _map(tensors, prefix + "o", o)


# -- feed-forwards ------------------------------------------------------------------------------


def squared_relu_mlp(h, tensors, prefix):
    return _map(tensors, prefix + "down", torch.clamp(_map(tensors, prefix + "up", h), min=0) ** 2)


def silu_mlp(h, tensors, prefix):
    return _map(tensors, prefix + "down", silu(_map(tensors, prefix + "gate", h)) * _map(tensors, prefix + "up", h))


def chosen_experts(h, tensors, prefix, router):
    """[T, experts] weights: the softmax over a token's ``top`` largest logits, zero elsewhere."""
    z = _map(tensors, prefix + "router", h) + _w(tensors, prefix + "router.b")
    out = torch.zeros_like(z)
    for t in range(h.shape[0]):
        best = sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[: router["top"]]
        ex = torch.exp(z[t, best] - z[t, best].max())
        out[t, best] = ex / ex.sum()
    return out


def shared_expert(h, tensors, prefix):
    return torch.sigmoid(_map(tensors, prefix + "shared.sg", h)) * silu_mlp(h, tensors, prefix + "shared.")


def experts_mlp(h, tensors, prefix, mlp):
    weights = chosen_experts(h, tensors, prefix, mlp["router"])
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        y = y + weights[:, e : e + 1] * silu_mlp(h, tensors, f"{prefix}e{e}.")
    if mlp.get("shared"):
        y = y + shared_expert(h, tensors, prefix)
    return y


# -- the model ------------------------------------------------------------------------------


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens, layer_outputs: Optional[List] = None):
    eps, parts = float(config["norm"]["eps"]), int(config["norm"].get("groups", 1))
    norm = lambda x, name: part_norm(x, _w(tensors, name), parts, eps)
    table = _w(tensors, "embed")
    x = norm(table[torch.as_tensor(tokens, dtype=torch.long)], "embed.norm")
    kept = {}
    for i, layer in enumerate(config["layers"]):
        m, p, turned = layer["mixer"], f"l{i}.", layer["type"] == "latent_attention_2"
        src = m.get("kv_from")
        if src is None:
            src = i
            kept[i] = latent_entries(x, tensors, p + "mix.", m, eps, turned)
        mixer = turned_latent_attention if turned else latent_attention
        x = x + norm(mixer(x, tensors, p + "mix.", m, eps, kept[src]), p + "norm1")
        mlp = layer.get("mlp")
        if mlp is not None:
            if mlp["kind"] == "dense":
                y = squared_relu_mlp(x, tensors, p + "mlp.")
            else:
                y = experts_mlp(x, tensors, p + "mlp.", mlp)
            x = x + norm(y, p + "norm2")
        if layer_outputs is not None:
            layer_outputs.append(x)
    return norm(x, "final.norm") @ table.T


def greedy(config, tensors, prompt, n_new: int):
    seq, out = list(prompt), []
    for _ in range(n_new):
        tok = int(forward(config, tensors, seq)[-1].argmax())
        out.append(tok)
        seq.append(tok)
    return out


def read_model(model_dir, dtype=DT):
    """``(config, tensors)`` of a model folder."""
    import json
    from pathlib import Path

    from safetensors.torch import load_file

    with open(Path(model_dir) / "config.json") as f:
        config = json.load(f)
    tensors = {k: v.to(dtype) for k, v in load_file(str(Path(model_dir) / "model.safetensors")).items()}
    return config, tensors
