"""Pegurax through the engine against the plain implementation of ``plain_pegurax.py``: each mechanism
alone, whole prompts against token-by-token decoding, portions down to two tokens, unequal batches,
pages and slots used again, keys at both sides of every chunk's edge and at page borders, states that
carry what was long ago, the first tokens of a sequence, long decoding, sizes that pad or equal one,
and greedy generation through ``Fastgen.generate``."""

import copy
import queue
from pathlib import Path

import numpy as np
import pytest
import torch

import helpers as H
import plain_pegurax as pp
from fastgen_b200.config import ConfigError, PartSpec, model_args_from_config
from fastgen_b200.weights import write_random_model

DEV = "cuda:0"


def _attn(heads, kv, dim, vdim, scale, chunk=None, dims=None, base=10000.0, scaling=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale)
    if chunk:
        m["mask"] = dict(size=chunk)
    if dims:
        m["rot"] = dict(dims=dims, base=base)
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return m


def _delta(heads, kv, dim, vdim, conv):
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv)


def _pair(left, right, left_scale, right_scale):
    return dict(type="parallel", mixer=dict(left=left, right=right, left_scale=left_scale, right_scale=right_scale))


def _mamba(inner, state, dt_rank, conv):
    return dict(type="mamba1", mixer=dict(inner=inner, state=state, dt_rank=dt_rank, conv=conv))


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(experts, top, ff):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


# chunks of no multiple of a page; a part of a head turned; value heads larger and smaller than query heads;
# two of five experts; a layer without a feed-forward; fewer query/key heads than heads in the delta rule; a
# scan whose step sizes and states pad
PA = dict(
    architecture="Pegurax", vocab=203, width=96, norm=dict(eps=1e-5), embedding=dict(scale=2.5),
    layers=[
        dict(_pair(_attn(6, 3, 16, 32, 0.3, 21, 8, 5000.0, (4.0, 64, 8.0, 1.0)), _delta(4, 2, 24, 40, 3), 0.6, 1.4),
             mlp=_moe(5, 2, 40)),
        dict(_mamba(72, 5, 3, 4), mlp=_dense(88)),
        dict(_pair(_attn(4, 1, 32, 16, 0.2, 50, 32, 1e4, (16.0, 128, 16.0, 2.0)), _delta(2, 2, 40, 8, 2), 1.1, 0.3), mlp=None),
        dict(_mamba(40, 16, 8, 2), mlp=_moe(3, 3, 24)),
    ],
)
# a scan first; one expert of one; convolutions of one tap (nothing to keep); one head of everything; chunks
# shorter than a page; widths that are no multiple of eight; no embedding scale
PB = dict(
    architecture="Pegurax", vocab=97, width=60, norm=dict(eps=1e-6),
    layers=[
        dict(_mamba(33, 1, 1, 1), mlp=_moe(1, 1, 20)),
        dict(_pair(_attn(1, 1, 16, 16, 0.4, 5, 16, 100.0, (2.0, 32, 4.0, 1.0)), _delta(1, 1, 33, 5, 1), 1.0, 1.0), mlp=_dense(36)),
        dict(_mamba(50, 40, 12, 8), mlp=None),
    ],
)
# head sizes of the tcgen05 kernel, chunks that hold several of its key tiles and end inside one; a state of
# 128 rows; experts that all serve every token
PC = dict(
    architecture="Pegurax", vocab=130, width=128, norm=dict(eps=1e-5), embedding=dict(scale=0.5),
    layers=[
        dict(_pair(_attn(4, 2, 64, 64, 0.15, 150, 48, 1e5, (8.0, 256, 32.0, 1.0)), _delta(2, 1, 128, 16, 4), 0.7, 0.9),
             mlp=_moe(6, 1, 64)),
        dict(_mamba(96, 24, 10, 3), mlp=_moe(4, 2, 32)),
        dict(_pair(_attn(2, 1, 128, 64, 0.1, 96, 128, 1e6, (2.0, 64, 8.0, 0.5)), _delta(4, 4, 64, 64, 4), 0.9, 0.5), mlp=_dense(96)),
    ],
)
# nothing turned, no chunks, a rotation without a scaling
PD = dict(
    architecture="Pegurax", vocab=64, width=48, norm=dict(eps=1e-5),
    layers=[
        dict(_pair(_attn(3, 1, 16, 16, 0.25), _delta(3, 3, 16, 16, 4), 1.0, 0.5), mlp=_moe(9, 4, 8)),
        dict(_pair(_attn(2, 2, 16, 16, 0.25, 33, 4, 50.0), _delta(3, 1, 8, 12, 4), 0.5, 1.0), mlp=_dense(24)),
    ],
)
CONFIGS = {"pa": (PA, 3), "pb": (PB, 5), "pc": (PC, 8), "pd": (PD, 9)}
MARKED = 8  # channels that ``clear_choices`` sets aside


def make_dir(tmp_path, name, std=0.1):
    """A folder of random weights.  The short convolutions are made strong enough to leave numbers of about
    one, so that nothing of a mixer drowns in an epsilon."""
    from safetensors.torch import load_file, save_file

    cfg, seed = CONFIGS[name]
    d = write_random_model(Path(tmp_path) / name, cfg, seed, dtype=torch.bfloat16, norm_jitter=0.3, std=std)
    f = Path(d) / "model.safetensors"
    tensors = load_file(str(f))
    for key in tensors:
        if key.endswith(".conv"):
            tensors[key] = tensors[key] * 6
        if key.endswith((".q", ".k", ".v", ".g", ".a", ".b", ".in")) and "mix" in key:
            tensors[key] = tensors[key] * 2
    save_file({k: t.contiguous() for k, t in tensors.items()}, str(f))
    return d


def clear_choices(tensors, cfg, seed):
    """Routers whose choices no rounding turns: the first channels of the stream keep the embedding's number,
    one of two opposite ones (no layer adds to them, the output does not read them), and a router reads
    them alone, with evenly spaced weights.  So a token's experts follow from its id, in one of two orders,
    with weights that still depend on the whole stream through its norm."""
    g = torch.Generator().manual_seed(seed)
    dim = cfg["width"]
    sign = torch.randint(0, 2, (cfg["vocab"], 1), generator=g).float() * 2 - 1
    pattern = torch.tensor([1.0, -1.0] * (MARKED // 2))
    scale = float((cfg.get("embedding") or {}).get("scale", 1.0))
    tensors["embed"][:, :MARKED] = (sign * pattern * 4.0 / scale).to(tensors["embed"].dtype)
    tensors["final.norm"][:MARKED] = 0
    for i, layer in enumerate(cfg["layers"]):
        for n in ("ls1", "ls2"):
            if f"l{i}.{n}" in tensors:
                tensors[f"l{i}.{n}"][:MARKED] = 0
        if (layer.get("mlp") or {}).get("kind") == "moe":
            e = layer["mlp"]["router"]["experts"]
            at = (torch.randperm(e, generator=g).float() - (e - 1) / 2) / max(e - 1, 1) * 4.0
            router = torch.zeros(e, dim)
            router[:, :MARKED] = at[:, None] * pattern[None, :] / 16.0
            tensors[f"l{i}.mlp.router"] = router.to(tensors[f"l{i}.mlp.router"].dtype)
            tensors[f"l{i}.norm2"][:MARKED] = 1.0


def model_dir(tmp_path, name, dtype):
    """The model folder of a configuration.  In bfloat16 the engine's activations differ from the plain
    implementation's by a percent, which turns a token's choice of experts wherever two scores are that
    close, so the folder of the bfloat16 runs has routers of clear choices.  Choices of random routers are
    held in float32, and in bfloat16 by ``test_routed_experts_alone``."""
    from safetensors.torch import load_file, save_file

    if dtype == torch.float32:
        return make_dir(tmp_path, name)
    d = make_dir(Path(tmp_path) / "apart", name)
    f = Path(d) / "model.safetensors"
    tensors = load_file(str(f))
    clear_choices(tensors, *CONFIGS[name])
    save_file({k: t.contiguous() for k, t in tensors.items()}, str(f))
    return d


_plain = {}


def plain_logits(folder, tokens):
    key = (str(folder), tuple(tokens))
    if key not in _plain:
        cfg, w = pp.read_model(folder)
        _plain[key] = pp.forward(cfg, w, list(tokens)).numpy()
    return _plain[key]


# The bfloat16 rule of this design's models: a row of logits may differ from the plain one by T_L2 of the
# row's l2 norm and, in its worst entry, by T_MAX of the row's largest logit, and a request's rows by T_MEAN of
# their l2 norms on average.  A sub-layer's output passes a norm before it joins the stream, and so does the
# delta rule's read-out, so where one of them happens to be small its roundings grow: the plain implementation
# itself, with the inputs and results of its products rounded to bfloat16, is off by 0.01 of a row's norm at the
# median and by up to 0.08 at its worst rows.  float32 rows are held to ``helpers.check_row``'s 1e-4.
T_L2, T_MAX, T_MEAN = 0.16, 0.16, 0.025


def check_row(row, ref, dtype, what):
    if dtype == torch.float32:
        return H.check_row(row, ref, dtype, what)
    l2 = float(np.linalg.norm(row - ref) / max(np.linalg.norm(ref), 1e-30))
    mx = float(np.abs(row - ref).max()) / max(float(np.abs(ref).max()), 1e-30)
    assert l2 <= T_L2, f"{what}: l2 error {l2:.4f} of the row's norm (allowed {T_L2})"
    assert mx <= T_MAX, f"{what}: worst entry off by {mx:.4f} of the largest logit (allowed {T_MAX})"
    return l2


def compare(folder, requests, got, dtype):
    for rid, toks in requests.items():
        ref = plain_logits(folder, toks)
        assert set(got[rid]) == set(range(len(toks))), f"{rid}: positions missing"
        errors = [check_row(row, ref[p], dtype, f"{rid} pos {p}") for p, row in got[rid].items()]
        if dtype == torch.bfloat16 and len(errors) >= 8:
            assert np.mean(errors) <= T_MEAN, f"{rid}: l2 error {np.mean(errors):.4f} on average (allowed {T_MEAN})"


def _requests(vocab, lengths, seed):
    return {f"r{i}": H.random_tokens(vocab, n, seed + i) for i, n in enumerate(lengths)}


# ---------------------------------------------------------------------------------
# the description and the cache bookkeeping (no GPU)
# ---------------------------------------------------------------------------------
def test_description_reads_every_size_from_the_configuration():
    args = model_args_from_config(PA)
    assert (args.dim, args.vocab_size, args.streams, len(args.layers), args.tie_embeddings) == (96, 203, None, 4, True)
    assert args.embedder.params.scale == 2.5 and model_args_from_config(PB).embedder.params.scale == 1.0
    pair = args.layers[0].mixer.params
    left, right = pair.left.params, pair.right.params
    assert (pair.left_scale, pair.right_scale) == (0.6, 1.4)
    assert (left.n_heads, left.n_kv_heads, left.head_dim, left.v_head_dim, left.softmax_scale) == (6, 3, 16, 32, 0.3)
    assert left.chunk == 21 and left.window is None and left.sink_score == 0.0 and not left.sink and not left.bias
    assert left.qk_norm == "projection" and left.qk_norm_eps == 1e-5 and left.qk_layout == "half_split"
    rope = left.position.params
    assert (rope.rot_dims, rope.theta, rope.scaling.factor, rope.scaling.original_max_positions) == (8, 5000.0, 4.0, 64.0)
    assert (rope.scaling.fast, rope.scaling.slow) == (8.0, 1.0)
    assert (right.n_heads, right.n_kv_heads, right.head_dim, right.v_head_dim, right.conv) == (4, 2, 24, 40, 3)
    assert right.head_decay and right.full_gate and right.gate_act == "silu"
    scan = args.layers[1].mixer.params
    assert (scan.inner, scan.state, scan.dt_rank, scan.conv) == (72, 5, 3, 4)
    assert args.layers[1].ffn.params.ffn_dim == 88 and args.layers[1].ffn.params.act == "relu"
    moe = args.layers[0].ffn.params
    assert (moe.n_experts, moe.top, moe.ffn_dim, moe.score) == (5, 2, 40, "sigmoid")
    assert moe.weigh_input and not moe.correction and not moe.renormalize
    assert args.layers[2].ffn is None and [n for n, _, _ in args.layers[2].extra] == ["post_mixer_norm"]
    assert all(l.block == "sandwich" for l in args.layers)
    assert [(e.layer, e.kv_from) for e in args.schedule] == [(i, None) for i in range(4)]
    assert all(not l.mixer_norm.params.bias and not l.mixer_norm.params.scale for l in args.layers)
    assert all(spec.params.scale and not spec.params.bias for l in args.layers for _, _, spec in l.extra)
    plain = model_args_from_config(PD).layers[0].mixer.params.left.params
    assert plain.chunk is None and plain.position.kind == "none"


def test_description_errors_name_the_place():
    def bad(change):
        cfg = copy.deepcopy(PA)
        change(cfg["layers"])
        return cfg

    for change, words in (
        (lambda l: l[2].update(type="attention_9"), "attention_9"),
        (lambda l: l[0]["mixer"]["right"].pop("conv"), r"layers\[0\]\.mixer\.right.*conv"),
        (lambda l: l[0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), r"layers\[0\].*slow"),
        (lambda l: l[0]["mlp"]["router"].update(top=6), r"layers\[0\]"),
        (lambda l: l[1]["mlp"].update(kind="dense_9"), "dense_9"),
        (lambda l: l[1]["mixer"].pop("dt_rank"), r"layers\[1\].*dt_rank"),
        (lambda l: l[0]["mixer"]["left"].update(heads=5), r"layers\[0\]"),
        (lambda l: l[0]["mixer"]["left"]["mask"].update(size=0), "size"),
    ):
        with pytest.raises(ConfigError, match=words):
            model_args_from_config(bad(change))


def test_random_folder_holds_exactly_the_tensors_of_the_description(tmp_path):
    from safetensors.torch import load_file

    tensors = load_file(str(make_dir(tmp_path, "pa") / "model.safetensors"))
    names = set(tensors)
    assert {"embed", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.ls1", "l0.ls2", "l0.mix.left.q.norm",
            "l0.mix.left.k.norm", "l0.mix.left.o", "l0.mix.right.q.conv", "l0.mix.right.a", "l0.mix.right.A_log",
            "l0.mix.right.dt_bias", "l0.mix.right.b", "l0.mix.right.g", "l0.mix.right.norm", "l0.mlp.router", "l0.mlp.e4.down",
            "l1.mix.in", "l1.mix.conv", "l1.mix.conv.b", "l1.mix.x", "l1.mix.dt", "l1.mix.dt.b", "l1.mix.A_log", "l1.mix.D",
            "l1.mix.o", "l1.mlp.gate", "l1.mlp.up", "l1.mlp.down"} <= names
    assert not {"head", "l2.norm2", "l2.norm2b", "l2.ls2", "l0.mlp.e5.up", "l0.mlp.correction", "l1.mix.left.q"} & names
    assert tensors["l1.mix.x"].shape == (13, 72) and tensors["l1.mix.dt"].shape == (72, 3)
    assert tensors["l1.mix.A_log"].shape == (72, 5) and tensors["l0.mix.right.a"].shape == (4, 96)
    assert tensors["l0.mix.right.dt_bias"].shape == (4,) and tensors["l0.mix.right.g"].shape == (160, 96)
    assert tensors["l0.mix.left.q.norm"].shape == (96,) and tensors["l0.mix.left.k.norm"].shape == (48,)


def test_a_layer_without_a_feed_forward_may_ship_its_unused_norms(tmp_path):
    from fastgen_b200.engine.model import Model
    from fastgen_b200.weights.loader import WeightError, load_weights
    from safetensors.torch import load_file, save_file

    d = make_dir(tmp_path, "pa")
    f = d / "model.safetensors"
    tensors = load_file(str(f))
    args = model_args_from_config(PA)
    specs = Model(args, ops=None).weight_specs()
    for n in ("l2.norm2", "l2.norm2b", "l2.ls2"):
        tensors[n] = torch.ones(96, dtype=torch.bfloat16)
    save_file(tensors, str(f))
    assert set(load_weights(d, specs, "cpu", ignore=args.optional_tensors)) == {s.name for s in specs}
    tensors["l1.extra"] = torch.ones(3, dtype=torch.bfloat16)
    save_file(tensors, str(f))
    with pytest.raises(WeightError, match="l1.extra"):
        load_weights(d, specs, "cpu", ignore=args.optional_tensors)


def test_frequencies_and_magnitude():
    from fastgen_b200.config.pegurax import _rope
    from fastgen_b200.parts import make_position

    for dims, base, sc in ((8, 5000.0, (4.0, 64, 8.0, 1.0)), (32, 1e4, (16.0, 128, 16.0, 2.0)), (48, 1e5, (8.0, 256, 32.0, 1.0)),
                           (2, 100.0, (2.0, 32, 4.0, 1.0)), (64, 5e5, (32.0, 4096, 32.0, 1.0)), (16, 1e4, None),
                           (12, 1e3, (3.0, 16, 64.0, 32.0)), (16, 10.0, (2.0, 1e6, 2.0, 0.1))):
        rot = dict(dims=dims, base=base)
        if sc:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), sc))
        part = make_position(_rope(rot, 64, "test"))
        want, magnitude = pp.yarn(base, dims, rot.get("scaling"))
        table = part.table("cpu").double()  # a head of 64: 32 pairs, those that do not turn have frequency zero
        assert torch.allclose(table[: dims // 2], want, rtol=2e-6) and not table[dims // 2 :].any(), (dims, base, sc)
        assert abs(part.magnitude() - magnitude) < 1e-12


def test_chunks_give_their_pages_back():
    """Pages of 8 and chunks of 20: once a chunk has ended, the pages that hold only its positions are free,
    the one that the next chunk begins in stays; the block table agrees at every length."""
    from fastgen_b200.cache import CacheManager
    from fastgen_b200.parts import CacheSpec

    for page, chunk in ((8, 20), (8, 8), (8, 3), (16, 16), (4, 1), (8, 64), (8, 1000)):
        spec = CacheSpec(1, 16, chunk=chunk)
        cache = CacheManager([spec], [None], [None], page_size=page, n_pages=40, max_requests=2, max_length=160)
        for sizes in ((1,) * 130, (7, 1, 30, 2, 50, 1, 1, 28)):
            r, n = cache.admit("r"), 0
            for m in sizes:
                before = n
                cache.reserve(r, n + m)
                # everything that a query of this portion may see has a page
                first = before // chunk * chunk
                assert {p // page for p in range(first, n + m)} <= set(r.pages[0]), (page, chunk, n)
                n += m
                cache.advance(r, n)
                cache.check()
                held = set(r.pages[0])
                assert all((lp + 1) * page > n // chunk * chunk for lp in held), (page, chunk, n, held)
            cache.release("r")
            assert cache.free_pages() == [40]
    with pytest.raises(ValueError, match="chunk"):
        CacheSpec(1, 16, window=4, chunk=4)


# ---------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------
def _ops(dtype):
    from fastgen_b200.csrc.ops import Ops

    return Ops(dtype, DEV)


def _context(slot, start, n):
    from fastgen_b200.engine.step import StepContext

    ctx = StepContext(DEV)
    ctx.host_seq_slot, ctx.host_seq_cached, ctx.host_seq_start = [slot], [start], [0, n]
    ctx.pos = torch.arange(start, start + n, dtype=torch.int32, device=DEV)
    ctx.req = torch.full((n,), slot, dtype=torch.int32, device=DEV)
    ctx.seq_slot = torch.tensor([slot], dtype=torch.int32, device=DEV)
    ctx.seq_start = torch.tensor([0, n], dtype=torch.int32, device=DEV)
    ctx.seq_cached = torch.tensor([start], dtype=torch.int32, device=DEV)
    ctx.n_tokens, ctx.n_seqs = n, 1
    return ctx


def _value(out):
    """A part's output as one float64 tensor (a sum that has not been formed is formed)."""
    from fastgen_b200.parts.base import ScaledSum

    if isinstance(out, ScaledSum):
        assert out.row is None
        return sum(c * t.double() for t, c in out.terms)
    return out.double()


def _run_mixer(mixer, cache, x, portions, dtype, rid="r"):
    """One request through a mixer in portions; returns the outputs and the request."""
    req = cache.admit(rid)
    outs, start = [], 0
    for n in portions:
        cache.reserve(req, start + n)
        cache.flush_tables()
        ctx = _context(req.slot, start, n)
        outs.append(_value(mixer.forward(x[start:start + n].to(DEV, dtype), ctx, cache.memory(0))))
        cache.advance(req, start + n)
        start += n
    assert start == x.shape[0]
    return torch.cat(outs).cpu(), req


def _draw_all(part, g, std, tweak):
    from fastgen_b200.weights.random_init import draw

    w = {}
    for s in part.weight_specs():
        t = draw(s, g, 0.4)
        if s.init[0] == "normal" and s.init[1] == 0.02:
            t = t * (std / 0.02)
        w[s.name] = t.bfloat16()
    if tweak:
        tweak(w)
    return w


def _alone(build, m, dim, dtype, g, page=8, n_pages=24, std=0.3, tweak=None, eps=1e-5):
    """A mixer (``build`` one of the architecture's builders) with random tensors, bound, with a cache of its own."""
    from fastgen_b200.cache import CacheManager
    from fastgen_b200.parts import make_mixer

    ops = _ops(dtype)
    mixer = make_mixer(build(dim, eps, m, "mix.", "test"))
    w = _draw_all(mixer, g, std, tweak)
    mixer.bind({local: w[name].to(DEV) for local, name in mixer.names.items()}, ops)
    cache = CacheManager([mixer.cache_spec()], [mixer.state_spec()], [None], page, n_pages, 2, page * n_pages,
                         dtype=dtype, device=DEV, tensor_map_factory=ops.make_kv_tensor_maps)
    return mixer, cache, {k: v.double() for k, v in w.items()}, ops


def _attention_alone(m, dim, dtype, g, **kw):
    from fastgen_b200.config.pegurax import _chunked_attention

    return _alone(_chunked_attention, m, dim, dtype, g, **kw)


def _delta_alone(m, dim, dtype, g, **kw):
    from fastgen_b200.config.pegurax import _gated_delta

    return _alone(_gated_delta, m, dim, dtype, g, **kw)


def _mamba_alone(m, dim, dtype, g, **kw):
    from fastgen_b200.config.pegurax import _selective_scan

    return _alone(_selective_scan, m, dim, dtype, g, **kw)


def _tol(dtype):
    return 2e-5 if dtype == torch.float32 else 2.5e-2


def _close(out, ref, dtype, scale=None):
    scale = float(ref.abs().max()) if scale is None else scale
    err = float((out - ref).abs().max())
    assert err <= _tol(dtype) * scale, f"off by {err / scale:.2e} of the largest value (allowed {_tol(dtype):.1e})"


DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])


def _layer_norm(dim, eps, g, ops, scale=False, bias=False):
    from fastgen_b200.parts import LayerNormParams, make_norm

    norm = make_norm(PartSpec("layernorm", LayerNormParams(dim, eps, bias=bias, scale=scale), {"weight": "w", "scale": "s", "bias": "b"}))
    w, s, b = 1 + 0.3 * torch.randn(dim, generator=g), 0.7 * torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    norm.bind({"weight": w.to(DEV), "scale": s.to(DEV), "bias": b.to(DEV)}, ops)

    def plain(x):
        y = pp.centred_norm(x, w.double(), eps) + (b.double() if bias else 0.0)
        return y * s.double() if scale else y
    return norm, plain


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("dim", [1, 7, 96, 200, 1030, 3072, 5000, 8192, 8200])
@pytest.mark.parametrize("terms", [1, 2, 4])
def test_norms_on_both_sides_of_a_sum(dtype, dim, terms):
    """``h += scale * norm(sum of the summands)`` and the norm that opens the next sub-layer, in one kernel
    (rows of any width up to 8,192; wider ones in several): a mean far from zero, with and without biases;
    with rows gathered ``h`` stays."""
    from fastgen_b200.parts.base import ScaledSum

    ops = _ops(dtype)
    g = torch.Generator().manual_seed(dim + terms)
    t, eps = 9, 1e-3
    ys = [(torch.randn(t, dim, generator=g) + 2.0).to(dtype) for _ in range(terms)]
    coefs = [0.8, -0.5, 1.7, 0.1][:terms]
    x = 3 * torch.randn(t, dim, generator=g) - 40.0
    for bias in (False, True):
        close, plain_close = _layer_norm(dim, eps, g, ops, scale=True, bias=bias)
        nxt, plain_next = _layer_norm(dim, eps, g, ops, bias=bias)
        delta = ys[0].to(DEV) if terms == 1 else ScaledSum([(y.to(DEV), c) for y, c in zip(ys, coefs)])
        total = ys[0].double() if terms == 1 else sum(c * y.double() for y, c in zip(ys, coefs))
        new = x.double() + plain_close(total)
        h = x.clone().to(DEV)
        got = nxt.add_forward(h, delta, delta_norm=close)
        assert got.dtype == dtype
        assert float((h.double().cpu() - new).abs().max()) <= 1e-5 * float(new.abs().max())
        want = plain_next(new)
        _close(got.double().cpu(), want, dtype, max(1.0, float(want.abs().max())) * (20 if dtype == torch.float32 else 1))
        rows = torch.tensor([7, 0, 7, 8], dtype=torch.int32, device=DEV)
        h2 = x.clone().to(DEV)
        got = nxt.add_forward(h2, delta, rows=rows, delta_norm=close)
        _close(got.double().cpu(), want[[7, 0, 7, 8]], dtype, max(1.0, float(want.abs().max())) * (20 if dtype == torch.float32 else 1))
        assert torch.equal(h2.cpu(), x)
    ops.check_status()


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("kind", ["rmsnorm", "dynamic_tanh"])
def test_a_sum_passes_the_norm_that_closes_it(dtype, kind):
    """Norms without a kernel of their own for it: the summands are formed, normed and then added, also where
    the stream is written back."""
    from fastgen_b200.parts import DynamicTanhParams, RMSNormParams, make_norm
    from fastgen_b200.parts.base import ScaledSum

    ops = _ops(dtype)
    g = torch.Generator().manual_seed(2)
    dim = 64
    spec = (PartSpec("rmsnorm", RMSNormParams(dim, 1e-5), {"weight": "w"}) if kind == "rmsnorm"
            else PartSpec("dynamic_tanh", DynamicTanhParams(dim), {"weight": "w", "bias": "b", "alpha": "a"}))
    made = []
    for _ in range(2):
        norm = make_norm(spec)
        w, b, a = 1 + 0.3 * torch.randn(dim, generator=g), torch.randn(dim, generator=g), torch.tensor(0.7)
        norm.bind({"weight": w.to(DEV), "bias": b.to(DEV), "alpha": a.to(DEV)}, ops)
        plain = ((lambda y, w=w: pp.unit_rms(y, 1e-5) * w.double()) if kind == "rmsnorm"
                 else (lambda y, w=w, b=b: torch.tanh(0.7 * y) * w.double() + b.double()))
        made.append((norm, plain))
    (close, plain_close), (nxt, plain_next) = made
    x = torch.randn(5, dim, generator=g)
    ys = [torch.randn(5, dim, generator=g).to(dtype) for _ in range(2)]
    new = x.double() + plain_close(0.8 * ys[0].double() + 0.5 * ys[1].double())
    h = x.clone().to(DEV)
    got = nxt.add_forward(h, ScaledSum([(ys[0].to(DEV), 0.8), (ys[1].to(DEV), 0.5)]), delta_norm=close)
    assert float((h.double().cpu() - new).abs().max()) <= (2e-6 if dtype == torch.float32 else 2e-2) * float(new.abs().max())
    _close(got.double().cpu(), plain_next(new), dtype)


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("sizes", [
    # heads, key/value heads, key size, value size, scale, chunk, turned dimensions, base, scaling
    (6, 3, 16, 32, 0.3, 21, 8, 5000.0, (4.0, 64, 8.0, 1.0)),
    (4, 1, 32, 16, 0.2, 50, 32, 1e4, (16.0, 128, 16.0, 2.0)),
    (1, 1, 16, 16, 0.4, 5, 16, 100.0, (2.0, 32, 4.0, 1.0)),
    (3, 1, 24, 24, 0.3, 16, None, 1.0, None),                      # no positions at all, chunks of two pages
    (2, 2, 48, 40, 0.2, 1, 6, 50.0, (3.0, 16, 4.0, 1.0)),          # chunks of one: only the key itself and the sink
    (2, 1, 80, 80, 0.15, 33, 80, 1e4, None),
    (5, 5, 16, 16, 0.3, None, 4, 1e4, (8.0, 64, 8.0, 1.0)),        # no chunks
    (4, 2, 64, 64, 0.15, 40, 48, 1e5, (8.0, 256, 32.0, 1.0)),      # head sizes of the tcgen05 kernel
    (4, 4, 64, 32, 0.15, 64, 64, 1e5, (8.0, 256, 32.0, 1.0)),
    (2, 1, 128, 128, 0.1, 70, 128, 1e6, (2.0, 64, 8.0, 0.5)),
    (20, 1, 64, 64, 0.15, 30, 32, 1e4, (4.0, 64, 8.0, 1.0)),       # more heads a group than the single-token kernel's rows
    (2, 2, 192, 64, 0.1, 37, 64, 1e4, (4.0, 64, 8.0, 1.0)),        # mma.sync on cp.async tiles at a multiple of 64
])
def test_chunked_attention_alone(dtype, sizes):
    """Queries and keys normed over the whole projection, a part of each head turned (dimension i with
    dimension i + half) and grown by the magnitude, chunks, one more summand in the denominator: a portion,
    single tokens and short portions across pages of eight; then the pages are freed and taken again."""
    heads, kv, d, dv, scale, chunk, dims, base, scaling = sizes
    g = torch.Generator().manual_seed(heads * 100 + d)
    m = _attn(heads, kv, d, dv, scale, chunk, dims, base, scaling)
    mixer, cache, w, ops = _attention_alone(m, 40, dtype, g)
    x = torch.randn(150, 40, generator=g).to(dtype)
    ref = pp.chunked_attention(x.double(), m, w, "mix.", 1e-5)
    out, req = _run_mixer(mixer, cache, x, (75, 1, 1, 7, 1, 2, 3, 1, 26) + (1,) * 20 + (13,), dtype)
    ops.check_status()
    _close(out, ref, dtype)
    cache.release("r")
    out2, _ = _run_mixer(mixer, cache, x[:30], (2, 1, 27), dtype, rid="again")
    _close(out2, ref[:30], dtype, float(ref.abs().max()))


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("d", [16, 64, 128])
@pytest.mark.parametrize("chunk,page", [(128, 16), (100, 16), (129, 64), (24, 8)])
def test_keys_at_both_sides_of_a_chunks_edge(dtype, d, chunk, page):
    """The only keys with scores sit on the last place of a chunk and on the first of the next.  Queries at the
    end of a chunk see the key at its start; the queries after the edge see neither the one before it nor
    anything of the chunk before: in prompt portions that cross the edge, start on it or end on it, and decoded
    alone.  A chunk that is one place off, or counted from a portion's start, gives other outputs."""
    heads, n = 2, 3 * chunk + 5
    g = torch.Generator().manual_seed(chunk + d)
    m = _attn(heads, 1, d, d, 12.0 / d, chunk, 8, 1e4, (4.0, 4096, 32.0, 1.0))

    def tweak(w):
        for h in range(heads):
            w["mix.q"][h * d + d - 1, :] = 0
            w["mix.q"][h * d + d - 1, 0] = 4.0
        w["mix.k"][d - 1, :] = 0
        w["mix.k"][d - 1, 1] = 4.0
        w["mix.q.norm"][:] = 1.0
        w["mix.k.norm"][:] = 1.0
    mixer, cache, w, ops = _attention_alone(m, 24, dtype, g, page=page, n_pages=-(-n // page) + 2, std=0.05, tweak=tweak)
    x = 0.3 * torch.randn(n, 24, generator=g)
    x[:, :2] = 0.0
    x[:, 0] = 2.0  # every token asks
    for edge in (chunk, 2 * chunk, 3 * chunk):
        x[edge - 1, 1] = x[edge, 1] = 3.0
    x[0, 1] = 3.0
    x = x.to(dtype)
    ref = pp.chunked_attention(x.double(), m, w, "mix.", 1e-5)
    for off in (-1, 1):
        other = pp.chunked_attention(x.double(), dict(m, mask=dict(size=chunk + off)), w, "mix.", 1e-5)
        for p in (chunk - 1, chunk, 2 * chunk - 1, 2 * chunk):
            if (off > 0) == (p % chunk == 0):  # (a longer chunk shows after the edge, a shorter one before it)
                assert float((other[p] - ref[p]).abs().max()) > 0.1 * float(ref[p].abs().max()), (off, p)
    for portions in ((n,), (chunk - 1, 2, chunk - 1, n - 2 * chunk), (chunk, chunk + 1, n - 2 * chunk - 1),
                     (chunk - 3,) + (1,) * 6 + (chunk - 6,) + (1,) * 6 + (n - 2 * chunk - 3,)):
        out, _ = _run_mixer(mixer, cache, x, portions, dtype)
        ops.check_status()
        _close(out, ref, dtype)
        cache.release("r")


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("d", [16, 64])
def test_far_key_inside_its_chunk(dtype, d):
    """One key at the start of a chunk of 400 has a score above all others; queries near the chunk's end find it,
    the first query of the next chunk does not: in a prompt and decoded alone, the key on the first of many pages."""
    heads, chunk, n = 2, 400, 420
    g = torch.Generator().manual_seed(21)
    m = _attn(heads, 1, d, d, 12.0 / d, chunk, 8, 1e4, (4.0, 4096, 32.0, 1.0))

    def tweak(w):
        for h in range(heads):
            w["mix.q"][h * d + d - 1, :] = 0
            w["mix.q"][h * d + d - 1, 0] = 4.0
        w["mix.k"][d - 1, :] = 0
        w["mix.k"][d - 1, 1] = 4.0
    mixer, cache, w, ops = _attention_alone(m, 24, dtype, g, page=16, n_pages=32, std=0.05, tweak=tweak)
    x = 0.3 * torch.randn(n, 24, generator=g)
    x[:, :2] = 0.0
    x[2, 1] = 3.0
    for q in (360, chunk - 1, chunk):
        x[q, 0] = 3.0
    x = x.to(dtype)
    ref = pp.chunked_attention(x.double(), m, w, "mix.", 1e-5)
    x0 = x.clone()
    x0[2] = 0
    without = pp.chunked_attention(x0.double(), m, w, "mix.", 1e-5)
    assert all(float((ref[q] - without[q]).abs().max()) > 0.3 * float(ref[q].abs().max()) for q in (360, chunk - 1))
    assert torch.equal(ref[chunk], without[chunk])
    for portions in ((300, 120), (300,) + (1,) * 110 + (10,)):
        out, _ = _run_mixer(mixer, cache, x, portions, dtype)
        ops.check_status()
        for q in (360, chunk - 1, chunk):
            assert float((out[q] - ref[q]).abs().max()) <= _tol(dtype) * float(ref[q].abs().max()), q
        _close(out, ref, dtype)
        cache.release("r")


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("d", [16, 64, 128])
def test_the_constant_sink_joins_the_denominator_once(dtype, d):
    """Scores far below zero: almost all of the weight is the sink's, so the output is nearly zero; scores around
    zero at the first tokens of a chunk: the sink takes half, a third, a quarter.  Without it the outputs are
    several times as large; in a prompt (also one whose keys are worked on in several stretches) and decoded."""
    m = _attn(2, 1, d, d, 0.5 / d, 40, 8, 1e4)
    g = torch.Generator().manual_seed(3)
    for how in ("zero", "low"):
        def tweak(w):
            w["mix.q"][:] = 0
            w["mix.k"][:] = 0
            if how == "low":  # every score is -8
                w["mix.q"][d - 1 :: d, 0] = 1.0
                w["mix.k"][d - 1 :: d, 0] = -1.0
                w["mix.q.norm"][:] = 4.0
                w["mix.k.norm"][:] = 4.0
        mixer, cache, w, ops = _attention_alone(m, 24, dtype, g, tweak=tweak, n_pages=32)
        x = torch.randn(130, 24, generator=g)
        x[:, 0] = 2.0
        x = x.to(dtype)
        ref = pp.chunked_attention(x.double(), m, w, "mix.", 1e-5)
        v = (x.double() @ w["mix.v"].T)[40]
        if how == "zero":
            first = torch.cat([v, v]) @ w["mix.o"].T / 2  # a chunk's first token: its own value and the sink, half each
            assert float((ref[40] - first).abs().max()) < 1e-9
        for portions in ((130,), (38, 1, 1, 1, 1, 30, 2) + (1,) * 20 + (36,)):
            out, _ = _run_mixer(mixer, cache, x, portions, dtype)
            ops.check_status()
            _close(out, ref, dtype)
            cache.release("r")


@pytest.mark.gpu
@DTYPES
def test_the_magnitude_grows_turned_dimensions_only(dtype):
    """A head whose score comes half from turned and half from unturned dimensions: growing all of them, or none,
    gives another output."""
    g = torch.Generator().manual_seed(8)
    m = _attn(2, 2, 16, 16, 0.6, 64, 8, 50.0, (40.0, 64, 8.0, 1.0))
    mixer, cache, w, ops = _attention_alone(m, 32, dtype, g)
    x = torch.randn(60, 32, generator=g).to(dtype)
    ref = pp.chunked_attention(x.double(), m, w, "mix.", 1e-5)
    grown = 0.1 * np.log(40.0) + 1.0
    w_all = dict(w, **{"mix.q.norm": w["mix.q.norm"].clone()})
    for h in range(2):
        w_all["mix.q.norm"][h * 16 + 8 : h * 16 + 16] *= grown * grown
    w_none = dict(w, **{"mix.q.norm": w["mix.q.norm"].clone()})
    for h in range(2):
        w_none["mix.q.norm"][h * 16 : h * 16 + 8] /= grown * grown
    for other in (w_all, w_none):
        alt = pp.chunked_attention(x.double(), m, other, "mix.", 1e-5)
        assert float((alt - ref).abs().max()) > 0.1 * float(ref.abs().max())
    out, _ = _run_mixer(mixer, cache, x, (40, 1, 1, 18), dtype)
    ops.check_status()
    _close(out, ref, dtype)


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("sizes", [(4, 2, 24, 40, 3), (1, 1, 33, 1, 1), (6, 3, 8, 24, 8), (2, 1, 200, 12, 4), (3, 3, 16, 16, 4),
                                   (2, 2, 64, 9, 2), (4, 1, 128, 32, 4), (1, 1, 256, 64, 2), (8, 8, 32, 128, 4)])
def test_gated_delta_rule_alone(dtype, sizes):
    """Convolutions, unit norms, one decay per head, the corrected write, read-out, norm and SiLU gate: a prompt
    portion, single tokens and short portions through the state of a slot; then the slot is used again and
    starts from zero."""
    g = torch.Generator().manual_seed(sum(sizes))
    m = _delta(*sizes)
    mixer, cache, w, ops = _delta_alone(m, 72, dtype, g)
    x = torch.randn(60, 72, generator=g).to(dtype)
    ref = pp.gated_delta_rule(x.double(), m, w, "mix.", 1e-5)
    out, req = _run_mixer(mixer, cache, x, (30, 1, 1, 7, 1, 2, 3, 1, 14), dtype)
    ops.check_status()
    _close(out, ref, dtype)
    slot = req.slot
    cache.release("r")
    out2, req2 = _run_mixer(mixer, cache, x[:20], (1, 2, 17), dtype, rid="again")
    assert req2.slot == slot
    _close(out2, ref[:20], dtype, float(ref.abs().max()))


@pytest.mark.gpu
@DTYPES
def test_delta_state_carries_what_was_long_ago_and_decays_per_head(dtype):
    """Next to no decay in one head, an immediate one in the other: a value written 150 tokens back still makes
    most of the first head's read-out, and swapping the heads' decays gives another result."""
    g = torch.Generator().manual_seed(4)
    m = _delta(2, 1, 16, 8, 2)

    def tweak(w):
        w["mix.A_log"] = torch.tensor([-12.0, 2.0]).bfloat16()
        w["mix.g"] = w["mix.g"] * 3
    mixer, cache, w, ops = _delta_alone(m, 32, dtype, g, tweak=tweak, std=0.2, n_pages=32)
    x = 0.05 * torch.randn(170, 32, generator=g)
    x[5] = 2.0 * torch.randn(32, generator=g)
    x = x.to(dtype)
    ref = pp.gated_delta_rule(x.double(), m, w, "mix.", 1e-5)
    x0 = x.clone()
    x0[5] = 0
    for other, ww in ((x0, w), (x, dict(w, **{"mix.A_log": w["mix.A_log"].flip(0)}))):
        alt = pp.gated_delta_rule(other.double(), m, ww, "mix.", 1e-5)
        assert float((ref[160] - alt[160]).abs().max()) > 0.1 * float(ref[160].abs().max())
    out, _ = _run_mixer(mixer, cache, x, (4, 3, 90, 2) + (1,) * 50 + (21,), dtype)
    ops.check_status()
    _close(out, ref, dtype)
    assert float((out[160] - ref[160]).abs().max()) <= 2 * _tol(dtype) * float(ref[160].abs().max())


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("sizes", [(72, 5, 3, 4), (40, 16, 8, 2), (33, 1, 1, 1), (50, 40, 12, 8), (96, 24, 10, 3), (64, 32, 16, 4),
                                   (17, 64, 5, 4), (24, 100, 2, 2), (16, 128, 8, 4), (9, 200, 7, 3), (8, 256, 4, 2), (200, 8, 6, 4)])
def test_selective_scan_alone(dtype, sizes):
    """Convolution with a bias, low-rank step sizes, decays per channel and state number, B and C of the token,
    skip and gate: a prompt portion, single tokens and short portions through the state of a slot; then the slot
    is used again and starts from zero."""
    g = torch.Generator().manual_seed(sum(sizes))
    m = _mamba(*sizes)["mixer"]
    mixer, cache, w, ops = _mamba_alone(m, 48, dtype, g)
    x = torch.randn(70, 48, generator=g).to(dtype)
    ref = pp.mamba(x.double(), m, w, "mix.")
    out, req = _run_mixer(mixer, cache, x, (33, 1, 1, 8, 1, 2, 3, 1, 20), dtype)
    ops.check_status()
    _close(out, ref, dtype)
    slot = req.slot
    cache.release("r")
    out2, req2 = _run_mixer(mixer, cache, x[:20], (1, 2, 17), dtype, rid="again")
    assert req2.slot == slot
    _close(out2, ref[:20], dtype, float(ref.abs().max()))


@pytest.mark.gpu
@DTYPES
def test_scan_state_carries_what_was_long_ago_per_number(dtype):
    """One number of every channel's state hardly decays, all others do at once: what one token wrote 150 tokens
    back still shows through that number, and through no other place of the table of decays."""
    g = torch.Generator().manual_seed(12)
    m = _mamba(40, 20, 4, 3)["mixer"]
    slow = 13

    def tweak(w, at=slow):
        a = torch.full((40, 20), 3.0)
        a[:, at] = -9.0
        w["mix.A_log"] = a.bfloat16()
        w["mix.D"] = torch.zeros(40).bfloat16()
        w["mix.dt.b"] = torch.zeros(40).bfloat16()
    mixer, cache, w, ops = _mamba_alone(m, 32, dtype, g, tweak=tweak, n_pages=32)
    x = 0.1 * torch.randn(170, 32, generator=g)
    x[5] = 3.0 * torch.randn(32, generator=g)
    x = x.to(dtype)
    ref = pp.mamba(x.double(), m, w, "mix.")
    x0 = x.clone()
    x0[5] = 0
    w2 = {}
    tweak(w2, at=slow + 1)
    for other, ww in ((x0, w), (x, dict(w, **{k: v.double() for k, v in w2.items()}))):
        alt = pp.mamba(other.double(), m, ww, "mix.")
        assert float((ref[160] - alt[160]).abs().max()) > 0.2 * float(ref[160].abs().max())
    out, _ = _run_mixer(mixer, cache, x, (4, 3, 90, 2) + (1,) * 50 + (21,), dtype)
    ops.check_status()
    _close(out, ref, dtype)
    late = float(ref[150:].abs().max())
    assert float((out[150:] - ref[150:]).abs().max()) <= 2 * _tol(dtype) * late


@pytest.mark.gpu
@DTYPES
def test_a_scan_of_many_sequences(dtype):
    """Sequences of 1, 40, 1 and 17 tokens in one launch, slots out of order, a padding sequence among them: each
    gets what it gets alone (bitwise)."""
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(5)
    inner, N, slots = 70, 24, 5
    lengths, order = [1, 40, 0, 1, 17], [3, 0, -1, 4, 1]
    t = sum(lengths)
    rand = lambda *s: torch.randn(*s, generator=g)
    x, dt, z, low = (rand(t, n).to(DEV, dtype) for n in (inner, inner, inner, 2 * N + 8))
    bias, d, a = rand(inner).to(DEV), rand(inner).to(DEV), (-rand(inner, N).exp()).to(DEV)
    state0 = rand(slots, inner * N + 10).to(DEV)

    def context(starts, slot):
        ctx = _context(0, 0, 1)
        ctx.seq_slot = torch.tensor(slot, dtype=torch.int32, device=DEV)
        ctx.seq_start = torch.tensor(starts, dtype=torch.int32, device=DEV)
        ctx.n_seqs = len(slot)
        return ctx
    starts = [0]
    for n in lengths:
        starts.append(starts[-1] + n)
    together = state0.clone()
    y = ops.selective_scan(x, dt, low, 8, z, bias, a, d, together, context(starts, order), N)
    alone = state0.clone()
    for b, slot in enumerate(order):
        if slot < 0:
            continue
        s, e = starts[b], starts[b + 1]
        one = ops.selective_scan(x[s:e], dt[s:e], low[s:e], 8, z[s:e], bias, a, d, alone, context([0, e - s], [slot]), N)
        assert torch.equal(one, y[s:e]), b
    assert torch.equal(together, alone)
    assert torch.equal(together[2], state0[2]) and torch.equal(together[:, inner * N :], state0[:, inner * N :])


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("ff", [36, 88, 104])
@pytest.mark.parametrize("tokens", [1, 7, 90])
def test_dense_feed_forward_with_a_relu_gate(dtype, ff, tokens):
    from fastgen_b200.config.pegurax import _feed_forward
    from fastgen_b200.parts import make_feed_forward

    ops = _ops(dtype)
    g = torch.Generator().manual_seed(ff)
    part = make_feed_forward(_feed_forward(64, _dense(ff), "mlp.", "test"))
    w = _draw_all(part, g, 0.3, None)
    part.bind({local: w[name].to(DEV) for local, name in part.names.items()}, ops)
    w = {k: v.double() for k, v in w.items()}
    x = torch.randn(tokens, 64, generator=g).to(dtype)
    ref = pp.gated_mlp(x.double(), w, "mlp.", torch.relu)
    silu = pp.gated_mlp(x.double(), w, "mlp.", pp.silu)
    assert float((silu - ref).abs().max()) > 0.05 * float(ref.abs().max())
    _close(part.forward(x.to(DEV), _context(0, 0, tokens)).double().cpu(), ref, dtype)


def _experts_alone(mlp, dim, dtype, g, std=0.3, tweak=None):
    from fastgen_b200.config.pegurax import _feed_forward
    from fastgen_b200.parts import make_feed_forward

    ops = _ops(dtype)
    ff = make_feed_forward(_feed_forward(dim, mlp, "mlp.", "test"))
    w = _draw_all(ff, g, std, tweak)
    ff.bind({local: w[name].to(DEV) for local, name in ff.names.items()}, ops)
    return ff, {k: v.double() for k, v in w.items()}, ops


def _clear(x, mlp, w, margin):
    """Tokens whose last chosen expert leads the best one left out by more than ``margin`` (in logits)."""
    z = torch.sort(x @ w["mlp.router"].T, dim=-1, descending=True).values
    top = mlp["router"]["top"]
    if top == z.shape[1]:
        return torch.ones(x.shape[0], dtype=torch.bool)
    return (z[:, top - 1] - z[:, top]) > margin


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("sizes", [(5, 3, 40), (7, 1, 24), (1, 1, 56), (3, 3, 32), (12, 2, 96), (9, 4, 8), (33, 5, 16), (64, 8, 24),
                                   (6, 2, 20)])
@pytest.mark.parametrize("tokens", [1, 3, 70, 600])
def test_routed_experts_alone(dtype, sizes, tokens):
    """Sigmoid scores in float32, the largest chosen, each multiplying its expert's input: one expert, all
    experts, more than a warp has lanes; one token, a few, more tokens than experts, and a prompt's worth (whose
    products in bfloat16 are the grouped ones over the experts' gathered rows, some experts without a row)."""
    experts, top, ff = sizes
    g = torch.Generator().manual_seed(experts * 10 + top)
    mlp = _moe(experts, top, ff)
    part, w, ops = _experts_alone(mlp, 48, dtype, g)
    x = torch.randn(tokens, 48, generator=g).to(dtype)
    ref = pp.routed_experts(x.double(), mlp, w, "mlp.")
    out = _value(part.forward(x.to(DEV), _context(0, 0, tokens))).cpu()
    ops.check_status()
    ok = _clear(x.double(), mlp, w, 1e-4)  # both see the same rounded input: float32 sums are that close
    assert int(ok.sum()) >= (tokens * 2 + 2) // 3
    _close(out[ok], ref[ok], dtype, float(ref.abs().max()))


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("tokens", [5, 40, 300])
def test_the_weight_multiplies_the_experts_input(dtype, tokens):
    """Scores around a tenth: weighing the output instead of the input, dividing by the chosen scores' sum, or
    leaving the weight out would each give another output."""
    g = torch.Generator().manual_seed(31)
    experts, top = 6, 2
    mlp = _moe(experts, top, 32)

    def tweak(w):
        r = 0.05 * torch.randn(experts, 48, generator=g)
        r[:, 0] = torch.tensor([-2.0, -2.3, -1.7, -2.6, -2.1, -1.9])
        w["mlp.router"] = r.bfloat16()
    part, w, ops = _experts_alone(mlp, 48, dtype, g, tweak=tweak)
    x = torch.randn(tokens, 48, generator=g)
    x[:, 0] = 1.0
    x = x.to(dtype)
    xd = x.double()
    ref = pp.routed_experts(xd, mlp, w, "mlp.")
    s = torch.sigmoid(xd @ w["mlp.router"].T)
    picked = torch.topk(s, top, dim=-1).indices
    for how in ("output", "renormalized", "none"):
        alt = torch.zeros_like(ref)
        for t in range(tokens):
            wts = s[t, picked[t]]
            wts = wts / wts.sum() if how == "renormalized" else wts
            for e, wt in zip(picked[t], wts):
                row, p = xd[t : t + 1], f"mlp.e{int(e)}."
                alt[t] += (wt * pp.gated_mlp(row, w, p, pp.silu) if how == "output"
                           else pp.gated_mlp(row * (wt if how == "renormalized" else 1.0), w, p, pp.silu))[0]
        assert float((alt - ref).abs().max()) > 0.2 * float(ref.abs().max()), how
    out = _value(part.forward(x.to(DEV), _context(0, 0, tokens))).cpu()
    ops.check_status()
    ok = _clear(xd, mlp, w, 1e-4)
    _close(out[ok], ref[ok], dtype, float(ref[ok].abs().max()))


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("act", ["gelu_tanh", "relu2"])
@pytest.mark.parametrize("tokens", [3, 70, 600])
def test_weights_on_the_inputs_of_experts_without_a_gate(dtype, act, tokens):
    from fastgen_b200.parts import RoutedExpertsParams, make_feed_forward

    ops = _ops(dtype)
    g = torch.Generator().manual_seed(7)
    params = RoutedExpertsParams(48, 40, 5, 2, correction=False, score="sigmoid", act=act, weigh_input=True)
    part = make_feed_forward(PartSpec("routed_experts", params, {"router": "r", "w3": "e{}.up", "w2": "e{}.down"}))
    w = _draw_all(part, g, 0.3, None)
    part.bind({local: w[name].to(DEV) for local, name in part.names.items()}, ops)
    w = {k: v.double() for k, v in w.items()}
    x = torch.randn(tokens, 48, generator=g).to(dtype)
    xd = x.double()
    s = torch.sigmoid(xd @ w["r"].T)
    picked = torch.topk(s, 2, dim=-1).indices
    f = {"gelu_tanh": lambda z: torch.nn.functional.gelu(z, approximate="tanh"), "relu2": lambda z: torch.relu(z) ** 2}[act]
    ref = torch.zeros(tokens, 48, dtype=torch.float64)
    for e in range(5):
        y = f((s[:, e : e + 1] * xd) @ w[f"e{e}.up"].T) @ w[f"e{e}.down"].T
        ref += y * (picked == e).any(-1, keepdim=True)
    out = _value(part.forward(x.to(DEV), _context(0, 0, tokens))).cpu()
    ops.check_status()
    z = torch.sort(xd @ w["r"].T, dim=-1, descending=True).values
    ok = (z[:, 1] - z[:, 2]) > 1e-4
    _close(out[ok], ref[ok], dtype, float(ref.abs().max()))


@pytest.mark.gpu
def test_scores_that_round_to_one_are_ranked_by_their_logits():
    """Logits beyond 17, whose sigmoids are all one in float32."""
    ops = _ops(torch.float32)
    logits = torch.tensor([[18.0, 25.0, 19.0, 30.0, -5.0], [40.0, 20.0, 21.0, 19.0, 50.0]], device=DEV)
    ids, weights = ops.moe_route(logits, None, 2, _context(0, 0, 2), score="sigmoid")
    assert ids.tolist() == [[3, 1], [4, 0]] and torch.allclose(weights.cpu(), torch.ones(2, 2))


@pytest.mark.gpu
@DTYPES
def test_two_mixers_side_by_side(dtype):
    """Both halves read the same input; the sum takes each half with its own scale; the attention of the pair has
    the pages, the delta rule the slot's state."""
    from fastgen_b200.config.pegurax import _pair as build

    g = torch.Generator().manual_seed(41)
    m = PA["layers"][0]["mixer"]
    mixer, cache, w, ops = _alone(build, m, 56, dtype, g, std=0.25)
    x = torch.randn(50, 56, generator=g).to(dtype)
    ref = pp.two_mixers(x.double(), m, w, "mix.", 1e-5)
    left = pp.chunked_attention(x.double(), m["left"], w, "mix.left.", 1e-5)
    right = pp.gated_delta_rule(x.double(), m["right"], w, "mix.right.", 1e-5)
    assert float((ref - (left + right)).abs().max()) > 0.05 * float(ref.abs().max())
    out, _ = _run_mixer(mixer, cache, x, (20, 1, 1, 2, 5, 1, 20), dtype)
    ops.check_status()
    _close(out, ref, dtype)


# ---------------------------------------------------------------------------------
# whole models through the engine
# ---------------------------------------------------------------------------------
@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", ["pa", "pb", "pc", "pd"])
@pytest.mark.parametrize("plan", ["whole", "decode", "portions", "mixed"])
def test_replay(tmp_path, name, dtype, plan):
    """Whole prompts (of one and two tokens too), prompts with a decoded tail, portions of 2 to 17 tokens, and
    mixed batches of up to four requests whose pages and slots are used again, all against the plain
    implementation run on whole sequences."""
    d = model_dir(tmp_path, name, dtype)
    vocab = CONFIGS[name][0]["vocab"]
    page = 16
    if plan == "mixed":
        requests = _requests(vocab, [70, 33, 1, 90, 18, 64, 47, 2], 40)
        steps = H.plan_mixed(requests, seed=5)
    else:
        long = 330 if name == "pc" else 150
        requests = _requests(vocab, [1, 2, 37, long] if plan != "portions" else [2, 95], 20)
        steps = {"whole": H.plan_whole, "decode": lambda r: H.plan_decode_tail(r, 45), "portions": H.plan_portions}[plan](requests)
    outputs, engine = H.run_engine(d, dtype, steps, page, H.max_live_tokens(steps, page) + 2 * page)
    compare(d, requests, H.collect(steps, outputs), dtype)
    assert engine.cache.n_live == 0 and all(f == g.pool.n_pages for f, g in zip(engine.cache.free_pages(), engine.cache.groups))


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", ["pa", "pc"])
def test_batching_changes_nothing(tmp_path, dtype, name):
    """A request's logits in a batch of unequal requests equal those it gets alone (bitwise in float32, where
    every sum has a fixed order; within rounding in bfloat16)."""
    d = model_dir(tmp_path, name, dtype)
    requests = _requests(CONFIGS[name][0]["vocab"], [41, 5, 77, 20], 60)
    alone = H.plan_portions(requests, sizes=(9, 1, 1, 30))
    out_a, _ = H.run_engine(d, dtype, alone, 8, H.max_live_tokens(alone, 8) + 32)
    got_a = H.collect(alone, out_a)
    mixed = H.plan_mixed(requests, seed=2)
    out_m, _ = H.run_engine(d, dtype, mixed, 8, H.max_live_tokens(mixed, 8) + 32)
    got_m = H.collect(mixed, out_m)
    for rid, toks in requests.items():
        for p in range(len(toks)):
            if dtype == torch.float32:
                assert np.array_equal(got_a[rid][p], got_m[rid][p]), (rid, p)
            else:
                check_row(got_m[rid][p], got_a[rid][p], dtype, f"{rid} {p}")


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", ["pa", "pc"])
def test_steps_replayed_from_graphs_change_nothing(tmp_path, dtype, name):
    """Steps captured as CUDA graphs (single tokens, and prompt portions padded to a few shapes) give what the
    same steps give launched kernel by kernel: states and convolution inputs are advanced by the replays only,
    never by a capture, and padding lanes choose no expert."""
    d = model_dir(tmp_path, name, dtype)
    requests = _requests(CONFIGS[name][0]["vocab"], [41, 5, 77, 20], 61)
    mixed = H.plan_mixed(requests, seed=3)
    room = H.max_live_tokens(mixed, 8) + 32
    out_g, eng = H.run_engine(d, dtype, mixed, 8, room, max_step_tokens=64)
    assert eng.graphs is not None and eng.step_graphs is not None and eng.step_graphs.replays > 0
    out_p, _ = H.run_engine(d, dtype, mixed, 8, room, num_cuda_graphs=0)
    got_g, got_p = H.collect(mixed, out_g), H.collect(mixed, out_p)
    for rid, toks in requests.items():
        for p in range(len(toks)):
            if dtype == torch.float32:
                assert np.array_equal(got_g[rid][p], got_p[rid][p]), (rid, p)
            else:
                check_row(got_g[rid][p], got_p[rid][p], dtype, f"{rid} {p}")


@pytest.mark.gpu
@DTYPES
def test_long_decoding(tmp_path, dtype):
    """200 tokens decoded one by one after a two-token prompt, over many chunks and pages of eight; the pages of
    chunks that have ended are handed out again while the request lives."""
    d = model_dir(tmp_path, "pa", dtype)
    requests = _requests(203, [202], 77)
    steps = H.plan_decode_tail(requests, 200)
    outputs, engine = H.run_engine(d, dtype, steps, 8, 232)
    compare(d, requests, H.collect(steps, outputs), dtype)


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", ["pa", "pb"])
def test_slots_used_again_start_from_zero(tmp_path, dtype, name):
    """Two slots only: six requests pass through them one after the other, some ending in the middle of a step of
    the others; a state or a convolution input left by a slot's earlier request would show in the first tokens
    of the next."""
    d = model_dir(tmp_path, name, dtype)
    requests = _requests(CONFIGS[name][0]["vocab"], [30, 9, 41, 3, 26, 12], 81)
    steps = H.plan_mixed(requests, seed=7, max_live=2)
    outputs, engine = H.run_engine(d, dtype, steps, 8, H.max_live_tokens(steps, 8) + 16, max_requests=2)
    compare(d, requests, H.collect(steps, outputs), dtype)
    assert engine.cache.n_live == 0


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", ["pa", "pb"])
def test_greedy_generation_through_the_entry_point(tmp_path, dtype, name):
    """``Fastgen.generate`` with its scheduler (portions of 16 tokens, batches of 3, graphs) against greedy decoding
    with the plain implementation."""
    from fastgen_b200.engine import Fastgen, GenArgs, HfLoader, Packet

    d = model_dir(tmp_path, name, dtype)
    cfg, w = pp.read_model(d)
    vocab = cfg["vocab"]
    prompts = [H.random_tokens(vocab, n, 90 + n) for n in (7, 1, 40, 23)]
    fg = Fastgen.build(HfLoader(d), GenArgs(use_sampling=False, max_gen=12, cache_block=16, max_seq=128, max_batch=3,
                                            max_prefill=16),
                       tp_mesh=None, device=torch.device(DEV), dtype=dtype)
    q = queue.Queue()
    for i, p in enumerate(prompts):
        q.put(Packet(thread_id=i, tokens=p))
    q.put(None)
    got = {pkt.thread_id: pkt.tokens for pkt in fg.generate(q)}
    fg.destroy()
    for i, p in enumerate(prompts):
        assert len(got[i]) == 12
        if dtype == torch.float32:
            assert got[i] == pp.greedy(cfg, w, p, 12), i
        else:
            seq = list(p)
            for tok in got[i]:
                logits = pp.forward(cfg, w, seq)[-1]
                assert float(logits[tok]) >= float(logits.max()) - 0.03 * float(logits.abs().max())
                seq.append(tok)


# ---------------------------------------------------------------------------------
# the rule itself, and configurations drawn at random
# ---------------------------------------------------------------------------------
def _edit(layers, kind, change):
    for layer in layers:
        if layer["type"] == kind:
            change(layer["mixer"])


def test_faults_break_the_bfloat16_rule(tmp_path):
    """Negative controls, planted in the plain implementation: a chunk one place longer, a missing magnitude, a
    frequency law without its ramp, a value head's scale, an expert's weight left out, a lost skip, a decay that is
    a tenth off.  Each puts rows far outside what the bfloat16 comparison allows."""
    d = model_dir(tmp_path, "pa", torch.bfloat16)
    cfg, w = pp.read_model(d)
    tokens = H.random_tokens(cfg["vocab"], 100, 7)
    ref = pp.forward(cfg, w, tokens)

    def off(config=cfg, tensors=w):
        got = pp.forward(config, tensors, tokens)
        return float(((got - ref).norm(dim=-1) / ref.norm(dim=-1)).mean())

    def changed(change):
        c = copy.deepcopy(cfg)
        change(c["layers"])
        return c
    left = lambda f: (lambda layers: _edit(layers, "parallel", lambda m: f(m["left"])))
    faults = {
        "chunk": off(changed(left(lambda m: m["mask"].update(size=m["mask"]["size"] + 1)))),
        "no chunks": off(changed(left(lambda m: m.pop("mask")))),
        "no scaling": off(changed(left(lambda m: m["rot"].pop("scaling")))),
        "ramp": off(changed(left(lambda m: m["rot"]["scaling"].update(fast=1e6, slow=1e-6)))),
        "score scale": off(changed(left(lambda m: m.update(scale=m["scale"] * 1.2)))),
        "left scale": off(changed(lambda layers: _edit(layers, "parallel", lambda m: m.update(left_scale=1.0)))),
        "skip": off(tensors={k: torch.zeros_like(t) if k.endswith("mix.D") else t for k, t in w.items()}),
        "delta decay": off(tensors={k: t + 0.3 if k.endswith("right.A_log") else t for k, t in w.items()}),
        "scan decay": off(tensors={k: t + 1.0 if k.endswith("mix.A_log") and "right" not in k else t for k, t in w.items()}),
        "step bias": off(tensors={k: t + 0.5 if k.endswith("dt.b") else t for k, t in w.items()}),
        "layer scale": off(tensors={k: torch.ones_like(t) if k.endswith("ls1") else t for k, t in w.items()}),
    }
    assert all(v > T_MEAN for v in faults.values()), faults


def _random_config(seed):
    import random

    r = random.Random(seed)
    width = r.choice([40, 64, 72, 96, 120])

    def attn():
        kv = r.choice([1, 2, 3])
        d = r.choice([8, 16, 20, 32, 48, 64, 96, 128])
        turned = r.choice([d, d // 2, 2, None])
        sc = r.choice([None, (r.uniform(1.5, 40), r.choice([32, 64, 512]), r.choice([4.0, 32.0]), r.choice([0.5, 1.0]))])
        return _attn(kv * r.choice([1, 2, 4]), kv, d, r.choice([d, 8, 24, 64]), r.uniform(0.5, 2.0) * d ** -0.5,
                     r.choice([None, 3, 16, 31, 64, 97]), turned // 2 * 2 if turned else None, r.choice([50.0, 1e4, 1e6]), sc)

    def delta():
        kv = r.choice([1, 2, 3])
        return _delta(kv * r.choice([1, 2, 3]), kv, r.choice([8, 24, 32, 40, 64, 130]), r.choice([6, 16, 40, 64]), r.choice([1, 2, 4, 5]))

    def mlp():
        if r.random() < 0.15:
            return None
        if r.random() < 0.3:
            return _dense(r.choice([20, 64, 104]))
        e = r.choice([1, 2, 5, 8, 16])
        return _moe(e, r.choice([1, 2, e]) if e > 1 else 1, r.choice([8, 20, 48]))
    layers = []
    for _ in range(r.choice([1, 2, 3])):
        if r.random() < 0.5:
            layer = _pair(attn(), delta(), r.uniform(0.3, 1.5), r.uniform(0.3, 1.5))
        else:
            layer = _mamba(r.choice([24, 50, 80, 128]), r.choice([1, 4, 16, 20, 32, 64, 100]), r.choice([1, 3, 8, 11]), r.choice([1, 2, 4, 7]))
        layers.append(dict(layer, mlp=mlp()))
    return dict(architecture="Pegurax", vocab=r.choice([50, 131, 256]), width=width, norm=dict(eps=r.choice([1e-6, 1e-5, 1e-3])),
                embedding=dict(scale=r.uniform(0.5, 6.0)), layers=layers)


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("seed", range(100, 116))
def test_configurations_drawn_at_random(tmp_path, dtype, seed):
    """One to three layers of sizes drawn at random, mixed batches with pages and slots that are used again."""
    cfg = _random_config(seed)
    name = f"random{seed}"
    CONFIGS[name] = (cfg, seed)
    try:
        d = model_dir(tmp_path, name, dtype)
        requests = _requests(cfg["vocab"], [60, 17, 1, 110, 33, 2], seed)
        steps = H.plan_mixed(requests, seed=seed)
        page = (4, 8, 16, 64)[seed % 4]
        outputs, engine = H.run_engine(d, dtype, steps, page, H.max_live_tokens(steps, page) + page)
        compare(d, requests, H.collect(steps, outputs), dtype)
    finally:
        del CONFIGS[name]
