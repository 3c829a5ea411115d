"""Attention whose keys and values are linear maps of a cached latent."""

from __future__ import annotations

from typing import List, Optional

import torch

from .base import CacheSpec, Mixer, WeightSpec, make_position, register_mixer
from .params import LatentAttentionParams


class LatentAttention(Mixer):
    """Causal softmax attention over a compressed cache.

    Per token ``c = rmsnorm(w_dkv[:R] x) * dkv_norm`` (``R = kv_rank``) and ``k_t = turn(w_dkv[R:] x)``
    (``rot_dim`` numbers, shared by all heads) are all that is cached: one pool, one entry a token.
    Queries: ``q = w_uq (rmsnorm(w_dq x) * dq_norm)``, or ``q = w_q x`` in a model without a query latent,
    per head ``[head_dim plain | rot_dim turned]``.  Head ``h`` has keys ``[w_uk,h c | k_t]`` and values
    ``w_uv,h c``; its output is multiplied before ``wo`` by ``sigmoid(w_g x)_h``, a number per head (in the
    attention kernel's last step) or one per value dimension (on the mapped values), where the model
    has the gate.  ``rot_dim = 0``: no turned part.

    Computed with the key map folded into the query: ``qa_h = w_uk,h^T q_plain,h`` makes the score
    ``(qa_h . c + q_turned,h . k_t) * scale``, the attention kernel sums latents instead of values
    and ``w_uv,h`` maps a head's summed latent to its output afterwards.  Nothing per head is ever
    made for a cached token, in prompts or in decoding.  The projections of ``x`` (``w_dq`` or ``w_q``,
    ``w_g``, ``w_dkv``) run as one product.

    A layer with ``own_cache`` false has no ``w_dkv``: its run of the schedule reads the entries of
    the run it names (``ScheduleEntry.kv_from``), with its own ``w_uk`` and ``w_uv``.
    """

    params: LatentAttentionParams
    graph_safe = True

    def __init__(self, spec) -> None:
        super().__init__(spec)
        p = self.params
        self.position = make_position(p.position)
        self.gate_size = {None: 0, "head": p.n_heads, "value": p.n_heads * p.v_head_dim}[p.gate]
        self.qk = p.head_dim + p.rot_dim
        # entries are padded to 16 bytes in both compute types
        self.entry = -(-(p.kv_rank + p.rot_dim) // 8) * 8

    def weight_specs(self) -> List[WeightSpec]:
        p, n = self.params, self.names
        if p.q_rank is None:
            specs = [WeightSpec(n["w_q"], (p.n_heads * self.qk, p.dim))]
        else:
            specs = [
                WeightSpec(n["w_dq"], (p.q_rank, p.dim)),
                WeightSpec(n["dq_norm"], (p.q_rank,), ("ones",)),
                WeightSpec(n["w_uq"], (p.n_heads * self.qk, p.q_rank)),
            ]
        if p.own_cache:
            specs += [
                WeightSpec(n["w_dkv"], (p.kv_rank + p.rot_dim, p.dim)),
                WeightSpec(n["dkv_norm"], (p.kv_rank,), ("ones",)),
            ]
        specs += [
            WeightSpec(n["w_uk"], (p.n_heads * p.head_dim, p.kv_rank)),
            WeightSpec(n["w_uv"], (p.n_heads * p.v_head_dim, p.kv_rank)),
        ]
        if p.gate:
            specs.append(WeightSpec(n["w_g"], (self.gate_size, p.dim)))
        specs.append(WeightSpec(n["wo"], (p.dim, p.n_heads * p.v_head_dim)))
        return specs

    def cache_spec(self) -> Optional[CacheSpec]:
        return CacheSpec(1, self.entry, None, n_pools=1)

    def bind(self, tensors, ops) -> None:
        p = self.params
        self.ops = ops
        dt = ops.act_dtype
        # one projection of x: [w_dq or w_q; w_g; w_dkv] (each part's rows padded to a multiple of 8 so
        # that the next one starts on 16 bytes)
        pad = lambda w: torch.cat([w, w.new_zeros((-w.shape[0] % 8, p.dim))], dim=0)
        parts = [pad(self._turn_rows(tensors["w_q"], p.n_heads) if p.q_rank is None else tensors["w_dq"])]
        self.gate_offset = parts[0].shape[0]
        if p.gate:
            parts.append(pad(tensors["w_g"]))
        self.entry_offset = sum(w.shape[0] for w in parts)
        if p.own_cache:
            parts.append(self._turn_rows(tensors["w_dkv"], 1))
        self.w_down = torch.cat(parts, dim=0).to(dt).contiguous()
        self.dkv_norm = tensors["dkv_norm"].float().contiguous() if p.own_cache else None
        if p.q_rank is not None:
            self.dq_norm = tensors["dq_norm"].float().contiguous()
            self.w_uq = self._turn_rows(tensors["w_uq"], p.n_heads).to(dt).contiguous()
        self.w_uk = tensors["w_uk"].to(dt).reshape(p.n_heads, p.head_dim, p.kv_rank).contiguous()
        self.w_uv = tensors["w_uv"].to(dt).reshape(p.n_heads, p.v_head_dim, p.kv_rank).contiguous()
        # the float32 product takes [out, in] operands: the key map transposed per head
        self.w_uk_t = self.w_uk.transpose(1, 2).contiguous() if dt == torch.float32 else None
        self.w_uv_t = self.w_uv.transpose(1, 2).contiguous() if dt == torch.bfloat16 else None
        self.wo = tensors["wo"].to(dt).contiguous()
        self.freqs = self.position.table(ops.device)
        if self.freqs is None:
            self.freqs = torch.zeros(max(1, p.rot_dim // 2), dtype=torch.float32, device=ops.device)
        self.magnitude = float(getattr(self.position, "magnitude", lambda: 1.0)())

    def _turn_rows(self, w, heads: int):
        """The rows of a projection with ``heads`` heads whose last ``rot_dim`` rows turn, reordered from the
        checkpoint's pairs (``i`` with ``i + rot_dim / 2``) to the kernels' adjacent ones."""
        r = self.params.rot_dim
        if self.params.rot_layout != "half_split" or r == 0:
            return w
        w = w.view(heads, -1, w.shape[-1])
        turned = w[:, -r:].view(heads, 2, r // 2, w.shape[-1]).transpose(1, 2).reshape(heads, r, w.shape[-1])
        return torch.cat([w[:, :-r], turned], dim=1).reshape(-1, w.shape[-1])

    def forward(self, x, ctx, memory):
        p, ops = self.params, self.ops
        t, H, R = x.shape[0], p.n_heads, p.kv_rank
        down = ops.linear(x, self.w_down)
        gate = down[:, self.gate_offset : self.gate_offset + self.gate_size] if p.gate else None
        turn = (ctx, self.freqs, self.magnitude, H, self.qk, p.head_dim, p.rot_dim)
        q = down[:, : p.q_rank if p.q_rank is not None else H * self.qk]
        if memory.writes and (p.q_rank is not None or p.rot_dim):
            # the cache entries and what the queries need first, in one launch
            q = ops.latent_prepare(down[:, self.entry_offset : self.entry_offset + R + p.rot_dim], self.dkv_norm, p.eps,
                                   self.freqs, self.magnitude, memory, ctx, R, p.rot_dim, q,
                                   q_norm=self.dq_norm if p.q_rank is not None else None, n_heads=H, head_size=self.qk)
        else:
            if memory.writes:
                ops.latent_entry_write(down[:, self.entry_offset : self.entry_offset + R + p.rot_dim], self.dkv_norm,
                                       p.eps, self.freqs, self.magnitude, memory, ctx, R, p.rot_dim)
            if p.q_rank is not None:
                q = ops.rms_rows(q, self.dq_norm, p.eps)
            elif p.rot_dim:
                ops.rotate_part(q, *turn)
        if p.q_rank is not None:
            q = ops.linear(q, self.w_uq)
            if p.rot_dim:
                ops.rotate_part(q, *turn)
        q = q.view(t, H, self.qk)
        # the key map folded into the queries: qa[h] = q_plain[h] @ w_uk[h]
        qa = ops.head_products(q[:, :, : p.head_dim], self.w_uk, self.w_uk_t)  # [H, T, R]
        lat = torch.empty((H, t, R), dtype=x.dtype, device=x.device)
        ops.latent_attention(qa, q[:, :, p.head_dim :], lat, gate if p.gate == "head" else None, memory, ctx, H, R,
                             p.rot_dim, p.softmax_scale)
        # a head's summed latent through its value map, heads side by side for wo
        o = torch.empty((t, H, p.v_head_dim), dtype=x.dtype, device=x.device)
        ops.head_products_out(lat, self.w_uv, self.w_uv_t, o)
        o = o.view(t, H * p.v_head_dim)
        if p.gate == "value":
            ops.head_gate(o, gate, ctx.req, self.gate_size, 1)
        return ops.linear(o, self.wo)


register_mixer("latent_attention", LatentAttention)
