"""``Kuvusun``: config.json keys -> model description.

A decoder whose layers are listed one by one under ``layers``.  Norms sit on the sub-layers' outputs only:
``x <- x + norm1(mixer(x)); x <- x + norm2(ff(x))``; the token embedding passes a norm of its own and the
output projection is the embedding table.  Every norm of the model is an RMS norm in ``norm.groups`` equal
parts of the row (``parts/norm.py``).

Keys read: ``architecture``, ``vocab``, ``width``, ``norm{eps, groups}`` and per layer ``type``, ``mixer`` and
``mlp`` (or null):

* ``latent_attention``: ``heads, dim, vdim, q_rank, kv_rank, scale``: causal attention over a cached latent
  (``parts/latent_attention.py``), no positions, queries through a normed latent;
* ``latent_attention_2``: ``heads, dim, rot_dim, vdim, kv_rank, scale, rot{dims, base}``: queries straight from
  the input, a part of queries and keys that turns (dimension ``i`` with ``i + dims/2``), a sigmoid gate on
  every number of the heads' outputs.  With ``kv_from: j`` the layer reads layer ``j``'s cache;
* ``mlp{kind: dense, ff}``: ``down(relu(up x)^2)``;
* ``mlp{kind: moe, expert{ff}, router{experts, top}, shared{ff}}``: gated experts chosen by their logits (with
  a bias), weighted by the softmax over the chosen logits, and a gated shared expert (optional) whose
  output is multiplied by the sigmoid of one number per token.

Tensors: ``embed``, ``embed.norm``, ``l<i>.norm1|norm2``, ``l<i>.mix.q|dq|dq.norm|uq|dkv|dkv.norm|uk|uv|g|o``,
``l<i>.mlp.up|down`` or ``l<i>.mlp.router|router.b|e<j>.gate|up|down|shared.gate|up|down|sg``, ``final.norm``.
"""

from __future__ import annotations

from typing import Any, Mapping

from ..parts.params import (
    DenseMLPParams,
    LatentAttentionParams,
    NoPositionParams,
    PartRMSNormParams,
    RopeParams,
    RoutedExpertsParams,
    SwiGLUParams,
    TableEmbeddingParams,
)
from .model_args import ConfigError, LayerSpec, ModelArgs, PartSpec, ScheduleEntry, positive_int, require
from .registry import register_architecture

#: the design sets no limit on positions; the engine's own limits (cache size) apply
MAX_POSITIONS = 1 << 30

#: the activation the design fixes for its dense feed-forwards
DENSE_ACT = "relu2"


def _latent_attention(dim: int, eps: float, m: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(m, ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale"), where)
    params = LatentAttentionParams(
        dim=dim,
        n_heads=positive_int(m, "heads"),
        head_dim=positive_int(m, "dim"),
        rot_dim=0,
        v_head_dim=positive_int(m, "vdim"),
        q_rank=positive_int(m, "q_rank"),
        kv_rank=positive_int(m, "kv_rank"),
        softmax_scale=float(m["scale"]),
        eps=eps,
        position=PartSpec("none", NoPositionParams()),
        gate=None,
    )
    names = {"w_dq": "dq", "dq_norm": "dq.norm", "w_uq": "uq", "w_dkv": "dkv", "dkv_norm": "dkv.norm", "w_uk": "uk",
             "w_uv": "uv", "wo": "o"}
    return PartSpec("latent_attention", params, {k: prefix + v for k, v in names.items()})


def _turned_latent_attention(dim: int, eps: float, m: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"), where)
    require(m["rot"], ("dims", "base"), f"{where}.rot")
    rot_dim = positive_int(m, "rot_dim")
    if positive_int(m["rot"], "dims") != rot_dim:
        raise ConfigError(f"{where}: rot.dims must equal rot_dim")
    own = m.get("kv_from") is None
    params = LatentAttentionParams(
        dim=dim,
        n_heads=positive_int(m, "heads"),
        head_dim=positive_int(m, "dim"),
        rot_dim=rot_dim,
        v_head_dim=positive_int(m, "vdim"),
        q_rank=None,
        kv_rank=positive_int(m, "kv_rank"),
        softmax_scale=float(m["scale"]),
        eps=eps,
        position=PartSpec("rope", RopeParams(head_dim=rot_dim, theta=float(m["rot"]["base"]), rot_dims=rot_dim)),
        own_cache=own,
        gate="value",
        rot_layout="half_split",
    )
    names = {"w_q": "q", "w_uk": "uk", "w_uv": "uv", "w_g": "g", "wo": "o"}
    if own:
        names.update({"w_dkv": "dkv", "dkv_norm": "dkv.norm"})
    return PartSpec("latent_attention", params, {k: prefix + v for k, v in names.items()})


_MIXERS = {"latent_attention": _latent_attention, "latent_attention_2": _turned_latent_attention}


def _feed_forward(dim: int, mlp: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(mlp, ("kind",), where)
    if mlp["kind"] == "dense":
        require(mlp, ("ff",), where)
        return PartSpec("dense_mlp", DenseMLPParams(dim, positive_int(mlp, "ff"), act=DENSE_ACT),
                        {"up": prefix + "up", "down": prefix + "down"})
    if mlp["kind"] != "moe":
        raise ConfigError(f"{where}: unknown kind {mlp['kind']!r}; known: dense, moe")
    require(mlp, ("expert", "router"), where)
    require(mlp["expert"], ("ff",), f"{where}.expert")
    router = mlp["router"]
    require(router, ("experts", "top"), f"{where}.router")
    names = {"router": "router", "router_bias": "router.b", "w1": "e{}.gate", "w3": "e{}.up", "w2": "e{}.down"}
    shared = mlp.get("shared")
    if shared:
        require(shared, ("ff",), f"{where}.shared")
        shared = PartSpec("swiglu", SwiGLUParams(dim, positive_int(shared, "ff")),
                          {"w1": prefix + "shared.gate", "w3": prefix + "shared.up", "w2": prefix + "shared.down"})
        names["shared_gate"] = "shared.sg"
    # the softmax over the chosen logits is the softmax over all of them divided by the chosen ones' sum
    params = RoutedExpertsParams(
        dim, positive_int(mlp["expert"], "ff"), positive_int(router, "experts"), positive_int(router, "top"),
        correction=False, renormalize=True, router_bias=True, shared=shared or None, shared_gate=bool(shared))
    return PartSpec("routed_experts", params, {k: prefix + v for k, v in names.items()})


def kuvusun_model_args(config: Mapping[str, Any]) -> ModelArgs:
    require(config, ("vocab", "width", "layers", "norm"), "Kuvusun config.json")
    require(config["norm"], ("eps",), "Kuvusun config.json: norm")
    dim = positive_int(config, "width")
    vocab = positive_int(config, "vocab")
    eps = float(config["norm"]["eps"])
    groups = positive_int(config["norm"], "groups") if config["norm"].get("groups") is not None else 1
    if dim % groups:
        raise ConfigError(f"Kuvusun config.json: a width of {dim} cannot be normed in {groups} equal groups")
    if not isinstance(config["layers"], (list, tuple)) or not config["layers"]:
        raise ConfigError("Kuvusun config.json: 'layers' must be a non-empty list")

    def norm(name: str) -> PartSpec:
        return PartSpec("part_rmsnorm", PartRMSNormParams(dim, eps, groups), {"weight": name})

    layers, schedule, optional = [], [], []
    for i, layer in enumerate(config["layers"]):
        where = f"layers[{i}]"
        require(layer, ("type", "mixer"), where)
        kind = layer["type"]
        if kind not in _MIXERS:
            raise ConfigError(f"{where}: unknown mixer type {kind!r}; known: {', '.join(sorted(_MIXERS))}")
        p = f"l{i}."
        mlp = layer.get("mlp")
        try:
            mixer = _MIXERS[kind](dim, eps, layer["mixer"], p + "mix.", f"{where}.mixer")
            ffn = _feed_forward(dim, mlp, p + "mlp.", f"{where}.mlp") if mlp is not None else None
        except ValueError as e:
            raise ConfigError(f"{where}: {e}") from None
        kv_from = layer["mixer"].get("kv_from")
        if kv_from is not None:
            src = config["layers"][kv_from] if isinstance(kv_from, int) and 0 <= kv_from < i else None
            if kind != "latent_attention_2" or src is None or src["type"] != kind or src["mixer"].get("kv_from") is not None:
                raise ConfigError(f"{where}: kv_from joins two latent_attention_2 layers, of which the earlier one has "
                                  "a cache of its own")
            for key in ("kv_rank", "rot_dim", "rot"):
                if src["mixer"].get(key) != layer["mixer"].get(key):
                    raise ConfigError(f"{where}: {key} differs from that of layer {kv_from}, whose cache it reads")
        if ffn is None:
            optional.append(p + "norm2")  # a layer without a feed-forward has no use for it
        layers.append(LayerSpec(block="postnorm", mixer=mixer, mixer_norm=norm(p + "norm1"), ffn=ffn,
                                ffn_norm=norm(p + "norm2") if ffn is not None else None))
        schedule.append(ScheduleEntry(i, kv_from))

    return ModelArgs(
        architecture="Kuvusun",
        dim=dim,
        vocab_size=vocab,
        max_positions=MAX_POSITIONS,
        tie_embeddings=True,
        embedding_name="embed",
        output_name=None,
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm"),
        embedder=PartSpec("table", TableEmbeddingParams(vocab, dim), {"table": "embed"}),
        embed_norm=norm("embed.norm"),
        optional_tensors=tuple(optional),
    )


register_architecture("Kuvusun", kuvusun_model_args)
