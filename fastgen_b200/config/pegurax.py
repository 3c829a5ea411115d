"""``Pegurax``: config.json keys -> model description.

A decoder whose layers are listed one by one under ``layers``.  Every layer norms its sub-layers on both
sides (layer norms with a weight and no bias) and scales what they add, element by element:
``x <- x + ls1 * norm1b(mixer(norm1(x))); x <- x + ls2 * norm2b(ff(norm2(x)))``.  The logits are the token
table itself (without the embedding's scale) times the normed stream.

Keys read: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (optional) and per layer
``type``, ``mixer`` and ``mlp`` (or null):

* ``parallel``: two mixers that read the same input, ``left_scale * left + right_scale * right``.
  ``left{heads, kv_heads, dim, vdim, scale, rot{dims, base, scaling{factor, original, fast, slow}}, mask.size}``:
  grouped-query softmax attention inside chunks of ``mask.size`` positions, an RMS norm of queries and keys
  over their whole projection, a rotation of a head's first ``rot.dims`` dimensions (dimension ``i`` with
  ``i + dims/2``, YaRN frequencies and magnitude), a sink of score zero in every head's softmax;
  ``right{heads, kv_heads, dim, vdim, conv}``: the gated delta rule with one decay per head and a full
  SiLU gate (``parts/gated_delta.py``);
* ``mamba1``: ``inner, state, dt_rank, conv``: the selective scan (``parts/selective_scan.py``);
* ``mlp{kind: dense, ff}``: ``down(relu(gate x) * up x)``; ``mlp{kind: moe, expert{ff}, router{experts, top}}``:
  SwiGLU experts chosen by sigmoid scores, whose scores multiply their inputs.

Tensors: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2``, ``l<i>.mix.*`` (``.left.*`` / ``.right.*``),
``l<i>.mlp.gate|up|down`` or ``l<i>.mlp.router|e<j>.gate|up|down``, ``final.norm``.
"""

from __future__ import annotations

from typing import Any, Mapping, Optional

from ..parts.params import (
    AttentionParams,
    GatedDeltaParams,
    LayerNormParams,
    NoPositionParams,
    RopeParams,
    RoutedExpertsParams,
    SelectiveScanParams,
    SideBySideParams,
    SwiGLUParams,
    TableEmbeddingParams,
    YarnScaling,
)
from .model_args import ConfigError, LayerSpec, ModelArgs, PartSpec, ScheduleEntry, positive_int, require
from .registry import register_architecture

#: the design sets no limit on positions; the engine's own limits (cache size) apply
MAX_POSITIONS = 1 << 30

#: constants the design fixes
SINK_SCORE = 0.0
DENSE_ACT = "relu"


def _norm(dim: int, eps: float, name: str, scale: Optional[str] = None) -> PartSpec:
    names = {"weight": name}
    if scale is not None:
        names["scale"] = scale
    return PartSpec("layernorm", LayerNormParams(dim, eps, bias=False, scale=scale is not None), names)


def _rope(rot: Optional[Mapping[str, Any]], head_dim: int, where: str) -> PartSpec:
    if not rot:
        return PartSpec("none", NoPositionParams())
    require(rot, ("dims", "base"), f"{where}.rot")
    sc = rot.get("scaling")
    scaling = None
    if sc:
        require(sc, ("factor", "original", "fast", "slow"), f"{where}.rot.scaling")
        scaling = YarnScaling(float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
    return PartSpec("rope", RopeParams(head_dim=head_dim, theta=float(rot["base"]), scaling=scaling,
                                       rot_dims=positive_int(rot, "dims")))


def _chunked_attention(dim: int, eps: float, m: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
    head_dim = positive_int(m, "dim")
    mask = m.get("mask")
    if mask:
        require(mask, ("size",), f"{where}.mask")
    params = AttentionParams(
        dim=dim,
        n_heads=positive_int(m, "heads"),
        n_kv_heads=positive_int(m, "kv_heads"),
        head_dim=head_dim,
        v_head_dim=positive_int(m, "vdim"),
        position=_rope(m.get("rot"), head_dim, where),
        chunk=positive_int(mask, "size") if mask else None,
        softmax_scale=float(m["scale"]),
        qk_layout="half_split",
        qk_norm="projection",
        qk_norm_eps=eps,
        sink_score=SINK_SCORE,
    )
    names = {"wq": "q", "wk": "k", "wv": "v", "wo": "o", "q_norm": "q.norm", "k_norm": "k.norm"}
    return PartSpec("gqa_attention", params, {k: prefix + v for k, v in names.items()})


def _gated_delta(dim: int, eps: float, m: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(m, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
    params = GatedDeltaParams(
        dim=dim,
        n_heads=positive_int(m, "heads"),
        n_kv_heads=positive_int(m, "kv_heads"),
        head_dim=positive_int(m, "dim"),
        v_head_dim=positive_int(m, "vdim"),
        conv=positive_int(m, "conv"),
        eps=eps,
        head_decay=True,
        full_gate=True,
        gate_act="silu",
    )
    names = {"wq": "q", "wk": "k", "wv": "v", "conv_q": "q.conv", "conv_k": "k.conv", "conv_v": "v.conv", "wb": "b",
             "a_log": "A_log", "norm": "norm", "wa": "a", "dt_bias": "dt_bias", "wg": "g", "wo": "o"}
    return PartSpec("gated_delta", params, {k: prefix + v for k, v in names.items()})


def _pair(dim: int, eps: float, m: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(m, ("left", "right"), where)
    params = SideBySideParams(
        left=_chunked_attention(dim, eps, m["left"], prefix + "left.", f"{where}.left"),
        right=_gated_delta(dim, eps, m["right"], prefix + "right.", f"{where}.right"),
        left_scale=float(m.get("left_scale", 1.0)),
        right_scale=float(m.get("right_scale", 1.0)),
    )
    return PartSpec("side_by_side", params, {})


def _selective_scan(dim: int, eps: float, m: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(m, ("inner", "state", "dt_rank", "conv"), where)
    params = SelectiveScanParams(dim=dim, inner=positive_int(m, "inner"), state=positive_int(m, "state"),
                                 dt_rank=positive_int(m, "dt_rank"), conv=positive_int(m, "conv"))
    names = {"w_in": "in", "conv": "conv", "conv_bias": "conv.b", "w_x": "x", "w_dt": "dt", "dt_bias": "dt.b",
             "a_log": "A_log", "d": "D", "wo": "o"}
    return PartSpec("selective_scan", params, {k: prefix + v for k, v in names.items()})


_MIXERS = {"parallel": _pair, "mamba1": _selective_scan}


def _feed_forward(dim: int, mlp: Mapping[str, Any], prefix: str, where: str) -> PartSpec:
    require(mlp, ("kind",), where)
    kind = mlp["kind"]
    if kind == "dense":
        require(mlp, ("ff",), where)
        return PartSpec("swiglu", SwiGLUParams(dim, positive_int(mlp, "ff"), act=DENSE_ACT),
                        {"w1": prefix + "gate", "w3": prefix + "up", "w2": prefix + "down"})
    if kind == "moe":
        require(mlp, ("expert", "router"), where)
        require(mlp["expert"], ("ff",), f"{where}.expert")
        require(mlp["router"], ("experts", "top"), f"{where}.router")
        params = RoutedExpertsParams(dim, positive_int(mlp["expert"], "ff"), positive_int(mlp["router"], "experts"),
                                     positive_int(mlp["router"], "top"), correction=False, renormalize=False,
                                     score="sigmoid", weigh_input=True)
        return PartSpec("routed_experts", params,
                        {"router": prefix + "router", "w1": prefix + "e{}.gate", "w3": prefix + "e{}.up",
                         "w2": prefix + "e{}.down"})
    raise ConfigError(f"{where}: unknown kind {kind!r}; known: dense, moe")


def pegurax_model_args(config: Mapping[str, Any]) -> ModelArgs:
    require(config, ("vocab", "width", "layers", "norm"), "Pegurax config.json")
    require(config["norm"], ("eps",), "Pegurax config.json: norm")
    dim = positive_int(config, "width")
    vocab = positive_int(config, "vocab")
    eps = float(config["norm"]["eps"])
    if not isinstance(config["layers"], (list, tuple)) or not config["layers"]:
        raise ConfigError("Pegurax config.json: 'layers' must be a non-empty list")

    layers = []
    optional = []
    for i, layer in enumerate(config["layers"]):
        where = f"layers[{i}]"
        require(layer, ("type", "mixer"), where)
        kind = layer["type"]
        if kind not in _MIXERS:
            raise ConfigError(f"{where}: unknown mixer type {kind!r}; known: {', '.join(sorted(_MIXERS))}")
        p = f"l{i}."
        try:
            mixer = _MIXERS[kind](dim, eps, layer["mixer"], p + "mix.", f"{where}.mixer")
            mlp = layer.get("mlp")
            ffn = _feed_forward(dim, mlp, p + "mlp.", f"{where}.mlp") if mlp is not None else None
        except ValueError as e:
            raise ConfigError(f"{where}: {e}") from None
        extra = [("post_mixer_norm", "norm", _norm(dim, eps, p + "norm1b", p + "ls1"))]
        if ffn is not None:
            extra.append(("post_ffn_norm", "norm", _norm(dim, eps, p + "norm2b", p + "ls2")))
        else:
            optional += [p + "norm2", p + "norm2b", p + "ls2"]
        layers.append(LayerSpec(block="sandwich", mixer=mixer, mixer_norm=_norm(dim, eps, p + "norm1"), ffn=ffn,
                                ffn_norm=_norm(dim, eps, p + "norm2") if ffn is not None else None, extra=tuple(extra)))

    scale = float((config.get("embedding") or {}).get("scale", 1.0))
    return ModelArgs(
        architecture="Pegurax",
        dim=dim,
        vocab_size=vocab,
        max_positions=MAX_POSITIONS,
        tie_embeddings=True,
        embedding_name="embed",
        output_name=None,
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=_norm(dim, eps, "final.norm"),
        embedder=PartSpec("table", TableEmbeddingParams(vocab, dim, scale), {"table": "embed"}),
        optional_tensors=tuple(optional),
    )


register_architecture("Pegurax", pegurax_model_args)
