"""A plain, slow implementation of the Pegurax design: whole sequences, no cache, float64 by default.

One function per mechanism, written from the design's equations in this file's own notation
and sharing no code with the package.  ``forward(config, tensors, tokens)`` runs one sequence
and returns the logits of every position (and, on request, the residual stream after every
layer).  ``tensors`` maps checkpoint names to torch tensors.

Notation: ``T`` tokens, positions ``0 .. T-1``; linear weights are stored ``[out, in]``.
"""

from __future__ import annotations

import math
from typing import Dict, Optional

import torch

DT = torch.float64


def _w(tensors, name):
    return tensors[name].to(DT)


# -- small pieces ---------------------------------------------------------------------------


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """Mean off, divided by the root of the mean squared deviation (plus ``eps``), times ``w``."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def yarn(base: float, dims: int, scaling: Optional[dict]):
    """``(frequencies of the dims/2 pairs, factor of cosine and sine)``.  Pairs that turn more than
    ``fast`` times over ``original`` positions keep their frequency, those that turn less than ``slow``
    times are slowed down by ``factor``, a straight ramp over the pair's index in between."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=DT)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    out = f.clone()
    for i in range(dims // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / factor * r + f[i] * (1 - r)
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, freqs, magnitude: float):
    """``x`` [T, heads, size]: among a head's first ``2P`` dimensions, dimension ``i`` and dimension
    ``i + P`` of position ``p`` turn together by ``p * freqs[i]`` and grow by ``magnitude``; the others
    stay as they are."""
    half = freqs.numel()
    ang = positions.to(DT)[:, None, None] * freqs
    c, s = torch.cos(ang) * magnitude, torch.sin(ang) * magnitude
    a, b = x[..., :half], x[..., half : 2 * half]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., 2 * half :]], dim=-1)


def causal_conv(x, taps, bias=None):
    """``x`` [T, C], ``taps`` [C, K]: ``y[t] = bias + sum_j taps[:, K-1-j] x[t-j]``, zeros before the start."""
    t, k = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, x.shape[1], dtype=x.dtype), x], dim=0)
    y = torch.zeros_like(x)
    for j in range(k):
        y = y + padded[j : j + t] * taps[:, j]
    return y if bias is None else y + bias


# -- mixers -----------------------------------------------------------------------------------


def chunked_attention(h, m, tensors, prefix, eps):
    """Grouped-query attention inside chunks of ``mask.size`` positions (counted from the sequence's
    start); queries and keys are RMS-normed over the whole projection before they turn; the softmax's
    denominator has one more summand, 1 (a score of zero without a value)."""
    t = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(h @ _w(tensors, prefix + "q").T, eps) * _w(tensors, prefix + "q.norm")
    k = unit_rms(h @ _w(tensors, prefix + "k").T, eps) * _w(tensors, prefix + "k.norm")
    v = (h @ _w(tensors, prefix + "v").T).reshape(t, G, dv)
    q, k = q.reshape(t, H, d), k.reshape(t, G, d)
    rot = m.get("rot")
    if rot:
        f, magnitude = yarn(float(rot["base"]), int(rot["dims"]), rot.get("scaling"))
        pos = torch.arange(t)
        q, k = rotate_halves(q, pos, f, magnitude), rotate_halves(k, pos, f, magnitude)
    i = torch.arange(t)
    seen = i[None, :] <= i[:, None]
    if m.get("mask"):
        c = int(m["mask"]["size"])
        seen = seen & (i[None, :] // c == i[:, None] // c)
    outs = []
    for head in range(H):
        g = head // (H // G)
        s = ((q[:, head] @ k[:, g].T) * float(m["scale"])).masked_fill(~seen, float("-inf"))
        top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
        e = torch.exp(s - top)
        outs.append(e @ v[:, g] / (torch.exp(-top) + e.sum(-1, keepdim=True)))
    return torch.cat(outs, dim=-1) @ _w(tensors, prefix + "o").T


def delta_recurrence(q, k, v, g, beta):
    """One head: ``q``, ``k`` [T, d], ``v`` [T, dv], ``g``, ``beta`` [T].  ``S <- g S;
    u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q``."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for n in range(q.shape[0]):
        S = g[n] * S
        u = beta[n] * (v[n] - S.T @ k[n])
        S = S + torch.outer(k[n], u)
        out.append(S.T @ q[n])
    return torch.stack(out)


def gated_delta_rule(h, m, tensors, prefix, eps):
    t = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda n: silu(causal_conv(h @ _w(tensors, prefix + n).T, _w(tensors, prefix + n + ".conv")))
    q, k, v = conv("q").reshape(t, G, d), conv("k").reshape(t, G, d), conv("v").reshape(t, H, dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * d ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(h @ _w(tensors, prefix + "b").T)  # [T, H]
    step = softplus(h @ _w(tensors, prefix + "a").T + _w(tensors, prefix + "dt_bias"))
    g = torch.exp(-torch.exp(_w(tensors, prefix + "A_log")) * step)  # one decay per head
    out = torch.stack([delta_recurrence(q[:, n // (H // G)], k[:, n // (H // G)], v[:, n], g[:, n], beta[:, n])
                       for n in range(H)], dim=1)
    out = unit_rms(out, eps) * _w(tensors, prefix + "norm") * silu(h @ _w(tensors, prefix + "g").T).reshape(t, H, dv)
    return out.reshape(t, H * dv) @ _w(tensors, prefix + "o").T


def two_mixers(h, m, tensors, prefix, eps):
    left = chunked_attention(h, m["left"], tensors, prefix + "left.", eps)
    right = gated_delta_rule(h, m["right"], tensors, prefix + "right.", eps)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


def selective_recurrence(x, dt, A, B, C, D):
    """``x``, ``dt`` [T, inner], ``A`` [inner, N], ``B``, ``C`` [T, N], ``D`` [inner]:
    ``S <- exp(dt A) S + dt x B;  y = S C + D x``, a row of ``S`` per channel."""
    S = torch.zeros_like(A)
    out = []
    for n in range(x.shape[0]):
        S = torch.exp(dt[n][:, None] * A) * S + (dt[n] * x[n])[:, None] * B[n][None, :]
        out.append(S @ C[n] + D * x[n])
    return torch.stack(out)


def mamba(h, m, tensors, prefix):
    inner, N, rank = m["inner"], m["state"], m["dt_rank"]
    proj = h @ _w(tensors, prefix + "in").T
    x, z = proj[:, :inner], proj[:, inner:]
    x = silu(causal_conv(x, _w(tensors, prefix + "conv"), _w(tensors, prefix + "conv.b")))
    low = x @ _w(tensors, prefix + "x").T
    dt = softplus(low[:, :rank] @ _w(tensors, prefix + "dt").T + _w(tensors, prefix + "dt.b"))
    y = selective_recurrence(x, dt, -torch.exp(_w(tensors, prefix + "A_log")), low[:, rank : rank + N], low[:, rank + N :],
                             _w(tensors, prefix + "D"))
    return (y * silu(z)) @ _w(tensors, prefix + "o").T


# -- feed-forwards ----------------------------------------------------------------------------


def gated_mlp(h, tensors, prefix, act):
    return (act(h @ _w(tensors, prefix + "gate").T) * (h @ _w(tensors, prefix + "up").T)) @ _w(tensors, prefix + "down").T


def routed_experts(h, mlp, tensors, prefix):
    """Every token goes through the ``top`` experts with the largest ``sigmoid(router)``; an expert reads
    the input times its score, and the experts' outputs are added as they are."""
    n, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
    s = torch.sigmoid(h @ _w(tensors, prefix + "router").T)
    picked = torch.topk(s, top, dim=-1).indices  # [T, top]
    out = torch.zeros_like(h)
    for e in range(n):
        chosen = (picked == e).any(-1)
        if chosen.any():
            out[chosen] = out[chosen] + gated_mlp(s[chosen, e : e + 1] * h[chosen], tensors, f"{prefix}e{e}.", silu)
    return out


# -- the model --------------------------------------------------------------------------------


def forward(config, tensors: Dict[str, torch.Tensor], tokens, return_layers: bool = False):
    eps = float(config["norm"]["eps"])
    table = _w(tensors, "embed")
    x = table[torch.as_tensor(tokens, dtype=torch.long)] * float((config.get("embedding") or {}).get("scale", 1.0))
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        norm = lambda y, n: centred_norm(y, _w(tensors, p + n), eps)
        h = norm(x, "norm1")
        if layer["type"] == "parallel":
            mixed = two_mixers(h, layer["mixer"], tensors, p + "mix.", eps)
        elif layer["type"] == "mamba1":
            mixed = mamba(h, layer["mixer"], tensors, p + "mix.")
        else:
            raise ValueError(layer["type"])
        x = x + norm(mixed, "norm1b") * _w(tensors, p + "ls1")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm(x, "norm2")
            if mlp["kind"] == "dense":
                ff = gated_mlp(h, tensors, p + "mlp.", torch.relu)
            else:
                ff = routed_experts(h, mlp, tensors, p + "mlp.")
            x = x + norm(ff, "norm2b") * _w(tensors, p + "ls2")
        after.append(x.clone())
    logits = centred_norm(x, _w(tensors, "final.norm"), eps) @ table.T
    if return_layers:
        return logits, torch.stack(after)
    return logits


def read_model(model_dir, dtype=DT):
    """``(config, tensors)`` of a model folder."""
    import json
    from pathlib import Path

    from safetensors.torch import load_file

    with open(Path(model_dir) / "config.json") as f:
        config = json.load(f)
    tensors = {k: v.to(dtype) for k, v in load_file(str(Path(model_dir) / "model.safetensors")).items()}
    return config, tensors


def greedy(config, tensors, prompt, n_new: int):
    seq, out = list(prompt), []
    for _ in range(n_new):
        tok = int(forward(config, tensors, seq)[-1].argmax())
        out.append(tok)
        seq.append(tok)
    return out
