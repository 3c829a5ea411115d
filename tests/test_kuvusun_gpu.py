"""Kuvusun through the engine against the plain implementation of ``plain_kuvusun.py``: each mechanism
alone, whole prompts against token-by-token decoding, portions down to two tokens, unequal batches,
pages and slots used again, keys far away and at page borders, the first tokens of a sequence, long
decoding, sizes that pad or equal one, and greedy generation through ``Fastgen.generate``."""

import copy
import queue
import random
from pathlib import Path

import numpy as np
import pytest
import torch

import helpers as H
import plain_kuvusun as pk
from fastgen_b200.config import ConfigError, PartSpec, model_args_from_config
from fastgen_b200.weights import write_random_model
from test_tanupel_gpu import _close, _context, _draw_all, _ops, _run_mixer, _tol, _value

DEV = "cuda:0"


def _plain(heads, dim, vdim, q_rank, kv_rank, scale):
    return dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale)


def _turned(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(dims=rot_dim, base=base))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(experts, top, ff, shared=None):
    mlp = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared:
        mlp["shared"] = dict(ff=shared)
    return mlp


def _layer(mixer, mlp):
    return dict(type="latent_attention_2" if "rot_dim" in mixer else "latent_attention", mixer=mixer, mlp=mlp)


# two layers read a third one's cache with heads of their own; a layer without a feed-forward; a shared
# expert of another width; three parts a norm
KA = dict(
    architecture="Kuvusun", vocab=211, width=96, norm=dict(eps=1e-5, groups=3),
    layers=[
        _layer(_plain(3, 24, 40, 56, 80, 0.2), _moe(5, 2, 40, 24)),
        _layer(_turned(4, 16, 8, 24, 48, 0.25, 5000.0), _dense(136)),
        _layer(_turned(2, 40, 8, 16, 48, 0.15, 5000.0, kv_from=1), _moe(7, 3, 16, 72)),
        _layer(_plain(2, 16, 16, 32, 48, 0.3), None),
        _layer(_turned(6, 8, 8, 8, 48, 0.3, 5000.0, kv_from=1), _dense(40)),
    ],
)
# one part a norm; one head, one expert, all experts, no shared expert; a turned part of one pair
KB = dict(
    architecture="Kuvusun", vocab=97, width=64, norm=dict(eps=1e-6, groups=1),
    layers=[
        _layer(_turned(1, 32, 2, 48, 32, 0.2, 100.0), _moe(1, 1, 56)),
        _layer(_plain(1, 64, 8, 8, 16, 0.15), _moe(4, 4, 24)),
        _layer(_turned(5, 8, 32, 64, 128, 0.2), None),
    ],
)
# sizes that fit no kernel's favourite: a width that is no multiple of eight, parts of 25 columns, ranks
# and heads that are no multiple of eight, odd head sizes
KC = dict(
    architecture="Kuvusun", vocab=173, width=100, norm=dict(eps=1e-5, groups=4),
    layers=[
        _layer(_plain(3, 13, 21, 20, 36, 0.25), _dense(60)),
        _layer(_turned(3, 7, 6, 11, 20, 0.3, 777.0), _moe(9, 4, 28, 20)),
        _layer(_turned(2, 15, 6, 5, 20, 0.25, 777.0, kv_from=1), _moe(3, 1, 36, 12)),
    ],
)
# sixteen parts of eight columns; more heads than a block of the kernels has rows at four tokens; a
# layer that reads the cache of the layer before the one before it
KD = dict(
    architecture="Kuvusun", vocab=130, width=128, norm=dict(eps=1e-5, groups=16),
    layers=[
        _layer(_turned(20, 16, 16, 16, 136, 0.2, 2000.0), _moe(16, 5, 8, 8)),
        _layer(_plain(24, 8, 16, 72, 24, 0.3), _dense(200)),
        _layer(_turned(20, 24, 16, 8, 136, 0.15, 2000.0, kv_from=0), _moe(2, 1, 88, 40)),
        _layer(_turned(3, 16, 4, 32, 64, 0.2, 1e6), _moe(33, 7, 8)),
    ],
)
CONFIGS = {"ka": (KA, 3), "kb": (KB, 5), "kc": (KC, 8), "kd": (KD, 9)}


def make_dir(tmp_path, name, std=0.1):
    cfg, seed = CONFIGS[name]
    return write_random_model(Path(tmp_path) / name, cfg, seed, dtype=torch.bfloat16, norm_jitter=0.3, std=std)


def model_dir(tmp_path, name, dtype):
    """The model folder of a configuration (see ``alike``)."""
    return make_dir(tmp_path, name) if dtype == torch.float32 else alike(make_dir(Path(tmp_path) / "alike", name))


def alike(d):
    """In bfloat16 the engine's activations differ from the plain implementation's by a percent, which
    turns a token's choice of experts wherever two logits are that close, so in the folder of the
    bfloat16 runs all experts of a layer are the same expert: whichever are chosen, their weights add up
    to one and the output is the same.  Choices that depend on the token are held in float32, and in
    bfloat16 by ``test_routed_experts_alone``."""
    from safetensors.torch import load_file, save_file

    f = Path(d) / "model.safetensors"
    tensors = load_file(str(f))
    for key in list(tensors):
        parts = key.split(".")
        if len(parts) == 4 and parts[1] == "mlp" and parts[2].startswith("e") and parts[2][1:].isdigit():
            tensors[key] = tensors[f"{parts[0]}.mlp.e0.{parts[3]}"].clone()
    save_file(tensors, str(f))
    return d


_known = {}


def plain_logits(model_dir, tokens):
    key = (str(model_dir), tuple(tokens))
    if key not in _known:
        cfg, w = pk.read_model(model_dir)
        _known[key] = pk.forward(cfg, w, list(tokens)).numpy()
    return _known[key]


# The bfloat16 rule of this design's models: a row of logits may differ from the plain one by K_L2 of the
# row's l2 norm and, in its worst entry, by K_MAX of the row's largest logit.  A norm on a sub-layer's
# output magnifies the rounding of an output (or of one part of it) that happens to be small: rounding
# the inputs and results of the plain implementation's products to bfloat16, and nothing else, moves the
# rows of these models by 0.01 in the middle, 0.033 for one row in a hundred and 0.055 at worst.  So of the
# rows of a comparison a share of K_SHARE may be up to K_FAR times as far as the rule.  float32 rows are
# all held to ``helpers.check_row``'s 1e-4.
K_L2, K_MAX, K_SHARE, K_FAR = 0.045, 0.055, 0.03, 2.5


def check_rows(trios, dtype):
    """``trios``: (what, row, row it should be)."""
    dist = []
    for what, row, ref in trios:
        if dtype == torch.float32:
            H.check_row(row, ref, dtype, what)
            continue
        l2 = float(np.linalg.norm(row - ref)) / max(float(np.linalg.norm(ref)), 1e-30)
        mx = float(np.abs(row - ref).max()) / max(float(np.abs(ref).max()), 1e-30)
        dist.append((max(l2 / K_L2, mx / K_MAX), what))
    if dist:
        worst = max(dist)
        assert worst[0] <= K_FAR, f"{worst[1]}: {worst[0]:.2f} times the rule's distance (at most {K_FAR})"
        over = [x for x in dist if x[0] > 1.0]
        assert len(over) <= max(1, K_SHARE * len(dist)), f"{len(over)} of {len(dist)} rows beyond the rule, e.g. {over[:3]}"


def compare(model_dir, requests, got, dtype):
    trios = []
    for rid, toks in requests.items():
        ref = plain_logits(model_dir, toks)
        assert set(got[rid]) == set(range(len(toks))), f"{rid}: positions missing"
        trios += [(f"{rid} pos {p}", row, ref[p]) for p, row in got[rid].items()]
    check_rows(trios, dtype)


def _requests(vocab, lengths, seed):
    return {f"r{i}": H.random_tokens(vocab, n, seed + i) for i, n in enumerate(lengths)}


# ---------------------------------------------------------------------------------
# the description and the cache bookkeeping (no GPU)
# ---------------------------------------------------------------------------------
def test_description_reads_every_size_from_the_configuration():
    args = model_args_from_config(KA)
    assert (args.dim, args.vocab_size, args.streams, len(args.layers)) == (96, 211, None, 5)
    assert args.tie_embeddings and args.output_name is None
    plain, turned, reader = (args.layers[i].mixer.params for i in (0, 1, 2))
    assert (plain.n_heads, plain.head_dim, plain.rot_dim, plain.v_head_dim, plain.q_rank, plain.kv_rank) == (3, 24, 0, 40, 56, 80)
    assert plain.gate is None and plain.position.kind == "none" and plain.own_cache and plain.softmax_scale == 0.2
    assert (turned.n_heads, turned.head_dim, turned.rot_dim, turned.v_head_dim, turned.q_rank, turned.kv_rank) == (
        4, 16, 8, 24, None, 48)
    assert turned.gate == "value" and turned.rot_layout == "half_split" and turned.own_cache and turned.eps == 1e-5
    assert (turned.position.params.theta, turned.position.params.rot_dims, turned.position.params.scaling) == (5000.0, 8, None)
    assert not reader.own_cache and reader.n_heads == 2 and reader.head_dim == 40
    assert [e.kv_from for e in args.schedule] == [None, None, 1, None, 1]
    assert args.layers[3].ffn is None and args.layers[3].ffn_norm is None and "l3.norm2" in args.optional_tensors
    moe, dense = args.layers[2].ffn.params, args.layers[1].ffn.params
    assert (moe.n_experts, moe.top, moe.ffn_dim, moe.shared.params.ffn_dim) == (7, 3, 16, 72)
    assert (moe.score, moe.renormalize, moe.correction, moe.router_bias, moe.shared_gate, moe.act) == (
        "softmax", True, False, True, True, "silu_gate")
    assert (dense.ffn_dim, dense.act) == (136, "relu2")
    lone = model_args_from_config(KB).layers[0].ffn.params
    assert lone.shared is None and not lone.shared_gate and lone.router_bias
    for spec in (args.embed_norm, args.final_norm, args.layers[0].mixer_norm, args.layers[0].ffn_norm):
        assert spec.kind == "part_rmsnorm" and (spec.params.dim, spec.params.parts, spec.params.eps) == (96, 3, 1e-5)
    assert all(l.block == "postnorm" and not l.extra for l in args.layers)
    free = copy.deepcopy(KA)
    del free["norm"]["groups"]
    assert model_args_from_config(free).final_norm.params.parts == 1


def test_description_errors_name_the_place():
    def broken(change, match):
        bad = copy.deepcopy(KA)
        change(bad)
        with pytest.raises(ConfigError, match=match):
            model_args_from_config(bad)

    broken(lambda c: c["layers"][1].update(type="latent_attention_9"), "latent_attention_9")
    broken(lambda c: c["layers"][0]["mixer"].pop("q_rank"), r"layers\[0\]\.mixer.*q_rank")
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), r"layers\[1\]\.mixer")
    broken(lambda c: c["layers"][2]["mixer"].update(kv_from=0), r"layers\[2\]")  # of the other kind
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=2), r"layers\[4\]")  # has no cache of its own
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=4), r"layers\[4\]")
    broken(lambda c: c["layers"][2]["mixer"].update(kv_rank=56), "kv_rank")
    broken(lambda c: c["layers"][2]["mixer"]["rot"].update(base=1.0), "rot")
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=6), r"layers\[0\]")
    broken(lambda c: c["layers"][0]["mlp"].update(kind="moe_9"), "moe_9")
    broken(lambda c: c["norm"].update(groups=5), "groups")
    broken(lambda c: c.pop("norm"), "norm")


def test_random_folder_holds_exactly_the_tensors_of_the_description(tmp_path):
    from safetensors.torch import load_file

    tensors = load_file(str(make_dir(tmp_path, "ka") / "model.safetensors"))
    want = {"embed", "embed.norm", "final.norm"}
    for i, layer in enumerate(KA["layers"]):
        p, mlp = f"l{i}.", layer["mlp"]
        want |= {p + "norm1"} | ({p + "norm2"} if mlp else set())
        names = ["q", "g"] if layer["type"] == "latent_attention_2" else ["dq", "dq.norm", "uq"]
        if "kv_from" not in layer["mixer"]:
            names += ["dkv", "dkv.norm"]
        want |= {f"{p}mix.{n}" for n in names + ["uk", "uv", "o"]}
        if mlp and mlp["kind"] == "dense":
            want |= {p + "mlp.up", p + "mlp.down"}
        elif mlp:
            want |= {p + "mlp.router", p + "mlp.router.b", p + "mlp.shared.sg"}
            want |= {f"{p}mlp.{e}.{n}" for e in [f"e{k}" for k in range(mlp["router"]["experts"])] + ["shared"]
                     for n in ("gate", "up", "down")}
    assert set(tensors) == want
    assert tensors["l1.mix.q"].shape == (4 * 24, 96) and tensors["l1.mix.g"].shape == (4 * 24, 96)
    assert tensors["l1.mix.dkv"].shape == (56, 96) and tensors["l0.mix.dkv"].shape == (80, 96)
    assert tensors["l2.mlp.shared.sg"].shape == (1, 96) and tensors["l2.mlp.router.b"].shape == (7,)


def test_readers_share_a_cache_and_have_none_of_their_own():
    """Five runs, three caches of two entry sizes; pages and slots come back and are taken again."""
    from fastgen_b200.cache import CacheManager
    from fastgen_b200.engine.model import Model

    model = Model(model_args_from_config(KA), ops=None)
    specs = model.cache_specs()
    assert [s.head_dim for s in specs] == [80, 56, 56, 48, 56] and all(s.n_pools == 1 and s.window is None for s in specs)
    assert all(s is None for s in model.state_specs()) and model.kv_from() == [None, None, 1, None, 1]
    assert model.cache_bytes_per_token(2) == 2 * (80 + 56 + 48)
    cache = CacheManager(specs, model.state_specs(), model.kv_from(), page_size=8, n_pages=12, max_requests=2, max_length=64)
    a = cache.admit("a")
    cache.reserve(a, 20)
    cache.advance(a, 20)
    b = cache.admit("b")
    cache.reserve(b, 9)
    cache.advance(b, 9)
    cache.check()
    slot = a.slot
    cache.release("a")
    c = cache.admit("c")
    assert c.slot == slot
    cache.reserve(c, 40)
    cache.advance(c, 40)
    cache.check()
    cache.release("b")
    cache.release("c")
    assert all(f == g.pool.n_pages for f, g in zip(cache.free_pages(), cache.groups))


def test_turned_rows_are_reordered_once_for_the_kernels():
    """The reordering of a projection's turned rows: turning adjacent pairs of the reordered product is
    turning the checkpoint's halves, and everything in front of the turned part stays."""
    from fastgen_b200.config.kuvusun import _MIXERS
    from fastgen_b200.parts import make_mixer

    m = _turned(3, 5, 6, 4, 16, 0.3, 50.0)
    mixer = make_mixer(_MIXERS["latent_attention_2"](12, 1e-5, m, "mix.", "test"))
    w = torch.arange(3 * 11 * 12, dtype=torch.float64).view(33, 12)
    new = mixer._turn_rows(w, 3).view(3, 11, 12)
    old = w.view(3, 11, 12)
    assert torch.equal(new[:, :5], old[:, :5])
    for i in range(3):
        assert torch.equal(new[:, 5 + 2 * i], old[:, 5 + i]) and torch.equal(new[:, 6 + 2 * i], old[:, 8 + i])


# ---------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(96, 3), (64, 1), (100, 4), (128, 16), (200, 8), (105, 7), (48, 48), (2048, 2), (40, 20),
                                   (4100, 1), (96, 12), (110, 5)])
def test_norm_in_parts(dtype, sizes):
    """The norm alone; the norm of a sub-layer's output joining the stream; the stream opened by a norm;
    both norms at the model's end, with rows gathered (the stream stays).  Parts of very unequal sizes:
    one statistic over the whole row would give something else."""
    from fastgen_b200.parts import PartRMSNormParams, RMSNormParams, ScaledSum, make_norm

    dim, parts = sizes
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(dim + parts)
    weights = [1 + 0.4 * torch.randn(dim, generator=g) for _ in range(2)]
    norms = []
    for w in weights:
        n = make_norm(PartSpec("part_rmsnorm", PartRMSNormParams(dim, 1e-5, parts), {"weight": "w"}))
        n.bind({"weight": w.to(DEV)}, ops)
        norms.append(n)
    loud = torch.exp(torch.linspace(-2, 2, parts)).repeat_interleave(dim // parts)
    t = 9
    x = 3 * torch.randn(t, dim, generator=g)
    y = (torch.randn(t, dim, generator=g) * loud).to(dtype)
    want_y = pk.part_norm(y.double(), weights[0].double(), parts, 1e-5)
    if parts > 1 and dim > parts:
        whole = pk.part_norm(y.double(), weights[0].double(), 1, 1e-5)
        assert float((whole - want_y).abs().max()) > 0.3 * float(want_y.abs().max())

    _close(norms[0].forward(y.to(DEV)).double().cpu(), want_y, dtype)
    exact = norms[0].forward(y.to(DEV), out_dtype=torch.float32)
    assert float((exact.double().cpu() - want_y).abs().max()) <= 2e-6 * float(want_y.abs().max())
    h = x.clone().to(DEV)
    got = norms[0].close(h, y.to(DEV))
    new = x.double() + want_y
    assert float((h.double().cpu() - new).abs().max()) <= 2e-6 * float(new.abs().max())
    assert got.dtype == dtype and torch.equal(got, h.to(dtype)) and got.data_ptr() != h.data_ptr()
    # a sum that was not formed, closed by the norm
    h = x.clone().to(DEV)
    norms[0].close(h, ScaledSum([(y.to(DEV), 0.5), (y.to(DEV), 0.5)]))
    assert float((h.double().cpu() - new).abs().max()) <= 2e-6 * float(new.abs().max())

    src = (2 * torch.randn(t, dim, generator=g)).to(DEV)
    h = torch.full((t, dim), float("nan"), device=DEV)
    got = norms[1].close(h, src, fresh=True)
    want = pk.part_norm(src.double().cpu(), weights[1].double(), parts, 1e-5)
    assert float((h.double().cpu() - want).abs().max()) <= 2e-6 * float(want.abs().max())
    assert torch.equal(got, h.to(dtype))

    want = pk.part_norm(new, weights[1].double(), parts, 1e-5)
    h = x.clone().to(DEV)
    _close(norms[1].add_forward(h, y.to(DEV), delta_norm=norms[0]).double().cpu(), want, dtype)
    rows = torch.tensor([7, 0, 7, 8], dtype=torch.int32, device=DEV)
    h = x.clone().to(DEV)
    got = norms[1].add_forward(h, y.to(DEV), rows=rows, delta_norm=norms[0])
    _close(got.double().cpu(), want[[7, 0, 7, 8]], dtype)
    assert torch.equal(h.cpu(), x)
    # no summand; and a summand that another kind of norm closes
    _close(norms[1].add_forward(h, None).double().cpu(), pk.part_norm(x.double(), weights[1].double(), parts, 1e-5), dtype)
    other = make_norm(PartSpec("rmsnorm", RMSNormParams(dim, 1e-5), {"weight": "w"}))
    other.bind({"weight": weights[0].to(DEV)}, ops)
    got = norms[1].add_forward(h, y.to(DEV), rows=rows, delta_norm=other)
    mixed = x.double() + pk.unit_rms(y.double(), 1e-5) * weights[0].double()
    _close(got.double().cpu(), pk.part_norm(mixed, weights[1].double(), parts, 1e-5)[[7, 0, 7, 8]], dtype)
    ops.check_status()


def _mixer_and_cache(m, dim, dtype, g, page=8, n_pages=16, std=0.3, tweak=None, eps=1e-5):
    """A mixer of the given sizes with random tensors, bound, with a cache of its own."""
    from fastgen_b200.cache import CacheManager
    from fastgen_b200.config.kuvusun import _MIXERS
    from fastgen_b200.parts import make_mixer

    ops = _ops(dtype)
    mixer = make_mixer(_MIXERS["latent_attention_2" if "rot_dim" in m else "latent_attention"](dim, eps, m, "mix.", "test"))
    w = _draw_all(mixer, g, std, tweak)
    mixer.bind({local: w[name].to(DEV) for local, name in mixer.names.items()}, ops)
    cache = CacheManager([mixer.cache_spec()], [mixer.state_spec()], [None], page, n_pages, 2, page * n_pages,
                         dtype=dtype, device=DEV, tensor_map_factory=ops.make_kv_tensor_maps)
    return mixer, cache, {k: v.double() for k, v in w.items()}, ops


def _plain_mixer(x, m, w, eps=1e-5):
    turned = "rot_dim" in m
    fn = pk.turned_latent_attention if turned else pk.latent_attention
    return fn(x, w, "mix.", m, eps, pk.latent_entries(x, w, "mix.", m, eps, turned))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [
    (4, 16, 24, 40, 48), (1, 64, 8, 8, 16), (3, 13, 21, 20, 36), (24, 8, 16, 72, 24), (2, 32, 32, 64, 200),
    (5, 48, 16, 24, 320), (70, 8, 8, 32, 64), (2, 128, 64, 96, 512), (1, 1, 1, 1, 1)])
def test_latent_attention_without_positions_alone(dtype, sizes):
    """Query latent, cached latent, no turned part and no gate: a prompt portion, single tokens and
    portions of two and three through the cache, against the form that makes every head's keys and
    values."""
    g = torch.Generator().manual_seed(sum(sizes))
    heads, d, dv, qr, rank = sizes
    # scores of size two: products of std 0.2 of unit latents, d of them added
    m = _plain(*sizes, 2.0 / (0.2 * qr ** 0.5 * 0.2 * rank ** 0.5 * d ** 0.5))
    mixer, cache, w, ops = _mixer_and_cache(m, 72, dtype, g, std=0.2)
    assert mixer.cache_spec().n_pools == 1 and mixer.cache_spec().head_dim >= m["kv_rank"]
    x = torch.randn(60, 72, generator=g).to(dtype)
    ref = _plain_mixer(x.double(), m, w)
    # no positions: the same tokens in another order give the last query the same output
    turned = torch.cat([x[:59].flip(0), x[59:]]).double()
    assert float((_plain_mixer(turned, m, w)[-1] - ref[-1]).abs().max()) < 1e-9
    for rid, portions in (("a", (30, 1, 1, 7, 2, 3, 1, 15)), ("b", (60,))):
        out, _ = _run_mixer(mixer, cache, x, portions, dtype, rid=rid)
        ops.check_status()
        _close(out, ref, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [
    (4, 16, 8, 24, 48), (1, 32, 2, 48, 32), (3, 7, 6, 11, 20), (20, 24, 16, 8, 136), (2, 32, 64, 32, 256),
    (5, 16, 32, 40, 384), (66, 8, 4, 8, 40), (2, 64, 64, 128, 512), (1, 1, 2, 1, 1)])
def test_latent_attention_with_a_turned_part_alone(dtype, sizes):
    """Queries straight from the input, a turned part (halves) of queries and of one key that the heads
    share, a gate on every output number."""
    g = torch.Generator().manual_seed(sum(sizes))
    heads, d, r, dv, rank = sizes
    # scores of size two: products of std 0.2 of a unit input and of a unit latent
    m = _turned(*sizes, 2.0 / (0.2 * 72 ** 0.5 * 0.2 * max(rank, 72) ** 0.5 * (d + r) ** 0.5), 300.0)
    mixer, cache, w, ops = _mixer_and_cache(m, 72, dtype, g, std=0.2)
    x = torch.randn(60, 72, generator=g).to(dtype)
    ref = _plain_mixer(x.double(), m, w)
    scale = float(ref.abs().max())
    if sizes[4] > 1:
        # what a missing rotation, another base or a missing gate would change
        still = _plain_mixer(x.double(), dict(m, rot=dict(dims=m["rot_dim"], base=1e30)), w)
        ungated = _plain_mixer(x.double(), m, dict(w, **{"mix.g": 0 * w["mix.g"]}))
        assert m["rot_dim"] == 2 or float((still - ref).abs().max()) > 0.05 * scale
        assert float((2 * ungated - ref).abs().max()) > 0.2 * scale
    for rid, portions in (("a", (30, 1, 1, 7, 2, 3, 1, 15)), ("b", (60,))):
        out, _ = _run_mixer(mixer, cache, x, portions, dtype, rid=rid)
        ops.check_status()
        _close(out, ref, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["plain", "turned"])
@pytest.mark.parametrize("rank", [32, 20])
def test_far_key_shows(dtype, kind, rank):
    """One entry hundreds of positions back takes nearly all of a query's weight, across many pages:
    through the latent of the mixer without positions, and through the turned key part of the other;
    for tokens decoded alone and inside a portion.  (A rank of 20 runs on the CUDA cores in bfloat16.)"""
    n, d, heads = 420, 16, 2
    g = torch.Generator().manual_seed(12)
    turned = kind == "turned"
    m = _turned(heads, d, 4, 16, rank, 0.4, 1e6) if turned else _plain(heads, d, 16, 24, rank, 0.06)

    def tweak(w):
        if turned:  # slow turns: the far score does not fade
            w["mix.dkv"][rank:, :] = 0
            w["mix.dkv"][rank:, 0] = 1.0    # the first input coordinate drives the shared key part,
            w["mix.q"][:] = 0.02 * torch.randn(w["mix.q"].shape, generator=g).bfloat16()
            for h in range(heads):
                w["mix.q"][h * (d + 4) + d : (h + 1) * (d + 4), 1] = 2.0  # the second one the queries
        else:
            # the latent is normed, so a loud key is one that points elsewhere: along latent coordinate 0
            w["mix.dkv"][0, 0] = 8.0
            w["mix.dq"][0, 1] = 8.0
            w["mix.uk"][:, 0] = 1.0
            w["mix.uq"][:, 0] = 0.5
    mixer, cache, w, ops = _mixer_and_cache(m, 32, dtype, g, page=16, n_pages=32, std=0.05, tweak=tweak)
    x = 0.3 * torch.randn(n, 32, generator=g)
    x[:, :2] = 0.0
    far, q1, q2 = 3, n - 1, n - 40
    x[far, 0] = 4.0
    x[q1, 1] = x[q2, 1] = 4.0
    x = x.to(dtype)
    ref = _plain_mixer(x.double(), m, w)
    x0 = x.clone()
    x0[far, 0] = 0
    other = _plain_mixer(x0.double(), m, w)
    for i in (q1, q2):
        assert float((ref[i] - other[i]).abs().max()) > 0.15 * float(ref[i].abs().max()), i
    for rid, portions in (("a", (300, 100) + (1,) * 20), ("b", (2,) + (1,) * 8 + (410,))):
        out, _ = _run_mixer(mixer, cache, x, portions, dtype, rid=rid)
        ops.check_status()
        for i in (q1, q2):
            _close(out[i], ref[i], dtype)
        _close(out, ref, dtype)
        cache.release(rid)


LOUD = (0, 7, 8, 31, 32, 63, 64, 65, 95)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("mode", ["prompt", "decoded"])
def test_keys_at_page_and_tile_borders(dtype, mode):
    """Keys with a score far above the others sit on the first and last places of pages and of the
    kernels' key tiles, the sequence's first token among them: every query from such a key on leans on
    it, the query before it does not see it.  Losing one, or seeing one too early, shows."""
    g = torch.Generator().manual_seed(23)
    n, d, r, rank = 96, 16, 4, 48
    m = _turned(3, d, r, 16, rank, 1.0, 1e6)

    def tweak(w):
        w["mix.q"][:] = 0.05 * torch.randn(w["mix.q"].shape, generator=g).bfloat16()
        for h in range(3):
            w["mix.q"][h * (d + r) + d : (h + 1) * (d + r), 1] = 1.0
        w["mix.dkv"][rank:, :] = 0
        w["mix.dkv"][rank:, 0] = 1.0
    mixer, cache, w, ops = _mixer_and_cache(m, 24, dtype, g, page=8, n_pages=16, std=0.2, tweak=tweak)
    x = torch.randn(n, 24, generator=g)
    x[:, 0] = 0.0
    x[:, 1] = 1.0
    for i in LOUD:
        x[i, 0] = 1.5
    x = x.to(dtype)
    ref = _plain_mixer(x.double(), m, w)
    for i in LOUD[1:]:
        x0 = x.clone()
        x0[i, 0] = 0
        other = _plain_mixer(x0.double(), m, w)
        assert float((other[i] - ref[i]).abs().max()) > 0.05 * float(ref[i].abs().max()), i
        assert torch.equal(other[i - 1], ref[i - 1])
    plans = ((8, 24, 8, 7, 1, 16, 32), (96,), (27, 2, 3, 64)) if mode == "prompt" else ((7, 1, 1, 23) + (1,) * 64,)
    for portions in plans:
        out, _ = _run_mixer(mixer, cache, x, portions, dtype)
        ops.check_status()
        _close(out, ref, dtype)
        cache.release("r")


@pytest.mark.gpu
@pytest.mark.parametrize("page", [8, 64, 256])
@pytest.mark.parametrize("sizes", [(5, 64, 0), (7, 64, 24), (32, 256, 32), (3, 256, 0), (24, 128, 10), (5, 192, 6), (24, 512, 64),
                                   (8, 512, 0), (130, 256, 64), (1, 64, 4), (7, 384, 40)])
def test_prompt_kernel_on_tensor_memory(monkeypatch, sizes, page):
    """The tcgen05 kernel of prompt portions by itself, at once and on cached entries, with and without a
    gate per head, for latents of one and of two output halves, tiles of 64 and of 32 keys, more heads
    than a block has rows, turned parts that fill no group of columns and start at no 16 bytes; against
    float64 sums over the same bfloat16 entries.  A loud key sits on every border of a tile or page, and
    the pages' free places hold large numbers that no query may see."""
    from fastgen_b200.cache import CacheManager
    from fastgen_b200.csrc import ops as ops_module
    from fastgen_b200.parts import CacheSpec

    heads, rank, rot = sizes
    monkeypatch.setattr(ops_module, "LATENT_TC5_BLOCKS", 1)
    ops = _ops(torch.bfloat16)
    lib = ops_module.latent(rank, rot)
    assert lib.fg_latent_tc5_rows() == 128
    g = torch.Generator().manual_seed(heads + rank + rot)
    width = -(-(rank + rot) // 8) * 8
    total = 210
    cache = CacheManager([CacheSpec(1, width, None, n_pools=1)], [None], [None], page, -(-total // page) + 2, 2, 2 * total,
                         dtype=torch.bfloat16, device=DEV, tensor_map_factory=ops.make_kv_tensor_maps)
    req = cache.admit("r")
    cache.reserve(req, total)
    cache.flush_tables()
    mem = cache.memory(0)
    entries = torch.randn(total, width, generator=g).bfloat16()
    for j in (0, 31, 32, 63, 64, 127, 128, 191, 192):
        entries[j, :rank] *= 2
    entries[:, rank + rot :] = 0
    mem.k_pages[:] = 1000.0
    table = mem.block_table[req.slot].tolist()
    for j in range(total):
        mem.k_pages[table[j // page], 0, j % page] = entries[j].to(DEV)
    scale = 2.0 / (rank + rot) ** 0.5
    keys = entries.double()
    for start, n, gated in ((0, 210, False), (77, 133, True), (190, 20, False)):
        qa = torch.randn(heads, n, rank, generator=g).bfloat16()
        q = torch.randn(n, heads, rot + 6, generator=g).bfloat16().to(DEV)
        gate = torch.randn(n, heads, generator=g).bfloat16()
        out = torch.full((heads, n, rank), float("nan"), dtype=torch.bfloat16, device=DEV)
        launched = ops_module.Ops.launches
        assert ops._latent_tc5(lib, qa.to(DEV), q[:, :, 6:] if rot else qa.to(DEV).permute(1, 0, 2), out,
                               gate.to(DEV) if gated else None, mem, _context(req.slot, start, n), heads, rank, rot, scale)
        assert ops_module.Ops.launches == launched + 1
        ops.check_status()
        s = torch.einsum("hnd,kd->hnk", qa.double(), keys[:, :rank])
        if rot:
            s = s + torch.einsum("nhd,kd->hnk", q[:, :, 6:].double().cpu(), keys[:, rank : rank + rot])
        later = torch.arange(total)[None, :] > torch.arange(start, start + n)[:, None]
        ref = torch.softmax((s * scale).masked_fill(later[None], float("-inf")), dim=-1) @ keys[:, :rank]
        if gated:
            ref = ref * torch.sigmoid(gate.double()).T[:, :, None]
        _close(out.double().cpu(), ref, torch.bfloat16)
        # (a row's own rounding, not the largest row's)
        err = (out.double().cpu() - ref).norm(dim=-1) / ref.norm(dim=-1)
        assert float(err.max()) < 0.01, float(err.max())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_reader_uses_the_other_layers_entries(dtype):
    """A mixer without a latent projection reads the entries that another one wrote, with its own heads,
    maps, queries and gate, and writes nothing."""
    from fastgen_b200.cache import CacheManager
    from fastgen_b200.config.kuvusun import _MIXERS
    from fastgen_b200.parts import make_mixer

    ops = _ops(dtype)
    g = torch.Generator().manual_seed(6)
    dim = 40
    ms = [_turned(2, 16, 8, 24, 48, 0.2, 500.0), _turned(5, 24, 8, 8, 48, 0.3, 500.0, kv_from=0)]
    mixers, ws = [], []
    for m in ms:
        mixer = make_mixer(_MIXERS["latent_attention_2"](dim, 1e-5, m, "mix.", "test"))
        w = _draw_all(mixer, g, 0.25, None)
        mixer.bind({local: w[name].to(DEV) for local, name in mixer.names.items()}, ops)
        mixers.append(mixer)
        ws.append({k: v.double() for k, v in w.items()})
    assert "mix.dkv" not in ws[1] and "mix.dkv.norm" not in ws[1]
    cache = CacheManager([m.cache_spec() for m in mixers], [None, None], [None, 0], 8, 16, 2, 128, dtype=dtype, device=DEV,
                         tensor_map_factory=ops.make_kv_tensor_maps)
    xs = [torch.randn(50, dim, generator=g).to(dtype) for _ in range(2)]  # the two layers' inputs differ
    entries = pk.latent_entries(xs[0].double(), ws[0], "mix.", ms[0], 1e-5, True)
    refs = [pk.turned_latent_attention(x.double(), w, "mix.", m, 1e-5, entries) for x, w, m in zip(xs, ws, ms)]
    req = cache.admit("r")
    outs, start = [[], []], 0
    for n in (20, 1, 1, 2, 5, 1, 20):
        cache.reserve(req, start + n)
        cache.flush_tables()
        ctx = _context(req.slot, start, n)
        for e, mixer in enumerate(mixers):
            assert cache.memory(e).writes == (e == 0)
            outs[e].append(mixer.forward(xs[e][start : start + n].to(DEV, dtype), ctx, cache.memory(e)).double().cpu())
        cache.advance(req, start + n)
        start += n
    ops.check_status()
    for out, ref in zip(outs, refs):
        _close(torch.cat(out), ref, dtype)


def _feed_forward_alone(mlp, dim, dtype, g, std=0.3, tweak=None):
    from fastgen_b200.config.kuvusun import _feed_forward
    from fastgen_b200.parts import make_feed_forward

    ops = _ops(dtype)
    ff = make_feed_forward(_feed_forward(dim, mlp, "mlp.", "test"))
    w = _draw_all(ff, g, std, tweak)
    ff.bind({local: w[name].to(DEV) for local, name in ff.names.items()}, ops)
    return ff, {k: v.double() for k, v in w.items()}, ops


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(136, 1), (136, 9), (60, 70), (200, 300)])
def test_squared_relu_alone(dtype, sizes):
    ff, tokens = sizes
    g = torch.Generator().manual_seed(ff)
    part, w, ops = _feed_forward_alone(_dense(ff), 56, dtype, g)
    x = torch.randn(tokens, 56, generator=g).to(dtype)
    ref = pk.squared_relu_mlp(x.double(), w, "mlp.")
    out = _value(part.forward(x.to(DEV), _context(0, 0, tokens))).cpu()
    ops.check_status()
    _close(out, ref, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(5, 2, 40, 24), (1, 1, 56, None), (4, 4, 24, None), (9, 4, 28, 20), (7, 3, 16, 72), (16, 5, 8, 8),
                                   (33, 7, 8, 40), (64, 6, 24, 8), (2, 1, 88, 40), (256, 9, 8, 16)])
@pytest.mark.parametrize("tokens", [1, 3, 70, 600])
def test_routed_experts_alone(dtype, sizes, tokens):
    """Logits with a bias, the largest chosen, the softmax over the chosen ones, gated experts, the shared
    expert times its gate; one expert, all experts, more experts than a warp has lanes; one token, a
    few, more tokens than experts, and a prompt's worth."""
    experts, top, ff, shared = sizes
    g = torch.Generator().manual_seed(experts * 10 + top)
    mlp = _moe(experts, top, ff, shared)
    part, w, ops = _feed_forward_alone(mlp, 48, dtype, g)
    x = torch.randn(tokens, 48, generator=g).to(dtype)
    ref = pk.experts_mlp(x.double(), w, "mlp.", mlp)
    out = part.forward(x.to(DEV), _context(0, 0, tokens))
    assert isinstance(out, torch.Tensor) and out.dtype == dtype  # (one tensor: the gated shared output is in it)
    ops.check_status()
    # choices that rest on no close call: both see the same rounded input, float32 sums are that close
    z = torch.sort(x.double() @ w["mlp.router"].T + w["mlp.router.b"], dim=-1, descending=True).values
    ok = (z[:, top - 1] - z[:, top]) > 1e-4 if top < experts else torch.ones(tokens, dtype=torch.bool)
    assert int(ok.sum()) >= (tokens * 2 + 2) // 3
    _close(out.double().cpu()[ok], ref[ok], dtype, float(ref.abs().max()))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_bias_and_the_chosen_softmax_show(dtype):
    """A router whose product favours experts 0 and 1 and whose bias turns the choice to 2 and 3; the rest
    hold as much weight as those: choosing without the bias, weighting without it, or a softmax over all
    experts would each give another output.  So would a shared expert without its gate."""
    g = torch.Generator().manual_seed(31)
    mlp = _moe(6, 2, 32, 16)

    def tweak(w):
        rows = torch.zeros(6, 48)
        rows[:, 0] = torch.tensor([2.0, 1.9, 1.0, 0.5, 1.2, 1.1])  # for x[0] = 1
        w["mlp.router"] = rows.bfloat16()
        w["mlp.router.b"] = torch.tensor([-1.5, -1.4, 1.0, 0.75, 0.0, 0.0]).bfloat16()
        w["mlp.shared.sg"] = torch.zeros(1, 48).bfloat16()
        w["mlp.shared.sg"][0, 0] = -1.0
        for n in ("gate", "up", "down"):
            w[f"mlp.shared.{n}"] *= 2
    part, w, ops = _feed_forward_alone(mlp, 48, dtype, g, tweak=tweak)
    x = 0.5 * torch.randn(40, 48, generator=g)
    x[:, 0] = 1.0
    x = x.to(dtype)
    xd = x.double()
    ref = pk.experts_mlp(xd, w, "mlp.", mlp)
    z = (xd @ w["mlp.router"].T + w["mlp.router.b"])[0]
    y = [pk.silu_mlp(xd, w, f"mlp.e{e}.") for e in range(6)]
    s = pk.silu_mlp(xd, w, "mlp.shared.")
    gate = torch.sigmoid(torch.tensor(-1.0, dtype=torch.float64))
    mix = lambda weights, coef: sum(c * y[e] for e, c in weights.items()) + coef * s
    two = torch.softmax(z[2:4], 0)
    assert float((mix({2: two[0], 3: two[1]}, gate) - ref).abs().max()) < 1e-9
    raw = xd[0] @ w["mlp.router"].T
    no_bias = torch.softmax(raw[:2], 0)
    unbiased = torch.softmax(raw[2:4], 0)
    everyone = torch.softmax(z, 0)
    for wrong in (mix({0: no_bias[0], 1: no_bias[1]}, gate), mix({2: unbiased[0], 3: unbiased[1]}, gate),
                  mix({2: everyone[2], 3: everyone[3]}, gate), mix({2: two[0], 3: two[1]}, 1.0)):
        assert float((wrong - ref).abs().max()) > 2 * _tol(dtype) * float(ref.abs().max())
    out = _value(part.forward(x.to(DEV), _context(0, 0, 40))).cpu()
    ops.check_status()
    _close(out, ref, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [96, 33, 1, 1024])
def test_column_gate(dtype, width):
    """A gate with a number of its own for every column, read from the middle of a wider tensor; very
    large gates of either sign give one and zero."""
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(width)
    t = 13
    x = torch.randn(t, width, generator=g).to(dtype)
    wide = 2 * torch.randn(t, width + 24, generator=g)
    wide[3] = 300.0
    wide[4] = -300.0
    wide = wide.to(dtype)
    ctx = _context(0, 0, t)
    want = x.double() * torch.sigmoid(wide[:, 8 : 8 + width].double())
    out = ops.head_gate(x.clone().to(DEV), wide.to(DEV)[:, 8 : 8 + width], ctx.req, width, 1)
    ops.check_status()
    _close(out.double().cpu(), want, dtype)
    assert torch.equal(out[3].cpu(), x[3]) and not out[4].any()


# ---------------------------------------------------------------------------------
# whole models through the engine
# ---------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["ka", "kb", "kc", "kd"])
@pytest.mark.parametrize("plan", ["whole", "decode", "portions", "mixed"])
def test_replay(tmp_path, name, dtype, plan):
    """Whole prompts (of one and two tokens too), prompts with a decoded tail, portions of 2 to 17 tokens,
    and mixed batches of up to four requests whose pages and slots are used again, all against the
    plain implementation run on whole sequences."""
    d = model_dir(tmp_path, name, dtype)
    vocab = CONFIGS[name][0]["vocab"]
    page = 16
    if plan == "mixed":
        requests = _requests(vocab, [70, 33, 1, 90, 18, 64, 47, 2], 40)
        steps = H.plan_mixed(requests, seed=5)
    else:
        requests = _requests(vocab, [1, 2, 37, 150] if plan != "portions" else [2, 95], 20)
        steps = {"whole": H.plan_whole, "decode": lambda r: H.plan_decode_tail(r, 45), "portions": H.plan_portions}[plan](requests)
    outputs, engine = H.run_engine(d, dtype, steps, page, H.max_live_tokens(steps, page) + 2 * page)
    compare(d, requests, H.collect(steps, outputs), dtype)
    assert engine.cache.n_live == 0 and all(f == g.pool.n_pages for f, g in zip(engine.cache.free_pages(), engine.cache.groups))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["ka", "kc"])
def test_layer_by_layer(tmp_path, name, dtype):
    """The residual stream after every layer, read where the next block (or the last norm) closes it."""
    from fastgen_b200.engine import Engine, Model, StepEntry
    from fastgen_b200.parts import split_pending

    d = model_dir(tmp_path, name, dtype)
    cfg, w = pk.read_model(d)
    toks = H.random_tokens(cfg["vocab"], 29, 5)
    want = []
    pk.forward(cfg, w, toks, want)
    model = Model.load(d, dtype, DEV)
    seen = []
    for i, block in enumerate(model.blocks):
        def forward(h, pending, ctx, memory, inner=block.forward):
            h, pending = inner(h, pending, ctx, memory)
            delta, norm = split_pending(pending)
            seen.append((h.double() + norm.forward(delta, out_dtype=torch.float32).double()).cpu())
            return h, pending
        block.forward = forward
    engine = Engine(model, page_size=16, n_pages=4, max_requests=1, max_length=64, num_cuda_graphs=0)
    engine.admit("a")
    engine.step([StepEntry("a", toks, [28])])
    engine.ops.check_status()
    assert len(seen) == len(want) == len(cfg["layers"])
    for got, ref in zip(seen, want):
        _close(got, ref, dtype)


def _random_config(seed):
    """A configuration drawn at random: both mixers in any order, readers of an earlier cache, sizes that
    pad and sizes that do not, every kind of feed-forward, one to many parts a norm."""
    rng = random.Random(seed)
    layers, sources = [], []
    for i in range(rng.randint(3, 7)):
        heads, dim, vdim = rng.choice([1, 2, 4, 6, 9]), rng.choice([8, 16, 20, 32]), rng.choice([8, 16, 33, 64])
        if rng.random() < 0.45:
            m = _plain(heads, dim, vdim, rng.choice([24, 32, 50, 64]), rng.choice([30, 32, 64, 128, 264]), 0.15)
        elif sources and rng.random() < 0.5:
            src = rng.choice(sources)
            b = layers[src]["mixer"]
            m = _turned(heads, dim, b["rot_dim"], vdim, b["kv_rank"], 0.12, b["rot"]["base"], kv_from=src)
        else:
            m = _turned(heads, dim, rng.choice([2, 8, 10, 32]), vdim, rng.choice([28, 32, 64, 128, 256]), 0.12,
                        rng.choice([100.0, 1e4, 1e6]))
            sources.append(i)
        experts = rng.choice([1, 2, 6, 16, 40])
        mlp = rng.choice([None, _dense(rng.choice([64, 100])),
                          _moe(experts, rng.randint(1, min(experts, 8)), rng.choice([16, 20, 56]), rng.choice([None, 24, 60]))])
        layers.append(_layer(m, mlp))
    width = rng.choice([64, 96, 120, 200])
    groups = rng.choice([q for q in (1, 2, 3, 4, 5, 8, 10) if width % q == 0])
    return dict(architecture="Kuvusun", vocab=rng.choice([97, 211, 256]), width=width, norm=dict(eps=1e-5, groups=groups),
                layers=layers)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("seed", [11, 13, 25, 35, 37, 42])
def test_configurations_drawn_at_random(tmp_path, dtype, seed):
    """Mixed batches of a model whose layers and sizes are drawn at random."""
    cfg = _random_config(seed)
    d = write_random_model(Path(tmp_path) / "m", cfg, seed, dtype=torch.bfloat16, norm_jitter=0.3, std=0.08)
    if dtype != torch.float32:
        d = alike(d)
    requests = _requests(cfg["vocab"], [150, 33, 1, 90, 18, 2], 40 + seed)
    steps = H.plan_mixed(requests, seed=seed)
    outputs, engine = H.run_engine(d, dtype, steps, 64, H.max_live_tokens(steps, 64) + 64)
    compare(d, requests, H.collect(steps, outputs), dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["ka", "kd"])
def test_batching_changes_nothing(tmp_path, dtype, name):
    """A request's logits in a batch of unequal requests equal those it gets alone (bitwise in float32,
    where every sum has a fixed order; within rounding in bfloat16)."""
    d = model_dir(tmp_path, name, dtype)
    requests = _requests(CONFIGS[name][0]["vocab"], [41, 5, 77, 20], 60)
    alone = H.plan_portions(requests, sizes=(9, 1, 1, 30))
    out_a, _ = H.run_engine(d, dtype, alone, 8, H.max_live_tokens(alone, 8) + 32)
    got_a = H.collect(alone, out_a)
    mixed = H.plan_mixed(requests, seed=2)
    out_m, _ = H.run_engine(d, dtype, mixed, 8, H.max_live_tokens(mixed, 8) + 32)
    got_m = H.collect(mixed, out_m)
    trios = []
    for rid, toks in requests.items():
        for p in range(len(toks)):
            if dtype == torch.float32:
                assert np.array_equal(got_m[rid][p], got_a[rid][p]), (rid, p)
            trios.append((f"{rid} pos {p}", got_m[rid][p], got_a[rid][p]))
    check_rows(trios, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["ka", "kb", "kd"])
def test_steps_replayed_from_graphs_change_nothing(tmp_path, dtype, name):
    """Steps captured as CUDA graphs (single tokens, and prompt portions padded to a few shapes) give
    what the same steps give launched kernel by kernel; padding lanes choose no expert."""
    d = model_dir(tmp_path, name, dtype)
    requests = _requests(CONFIGS[name][0]["vocab"], [41, 5, 77, 20], 61)
    mixed = H.plan_mixed(requests, seed=3)
    room = H.max_live_tokens(mixed, 8) + 32
    out_g, eng = H.run_engine(d, dtype, mixed, 8, room, max_step_tokens=64)
    assert eng.graphs is not None and eng.step_graphs is not None and eng.step_graphs.replays > 0
    out_p, _ = H.run_engine(d, dtype, mixed, 8, room, num_cuda_graphs=0)
    got_g, got_p = H.collect(mixed, out_g), H.collect(mixed, out_p)
    trios = []
    for rid, toks in requests.items():
        for p in range(len(toks)):
            if dtype == torch.float32:
                assert np.array_equal(got_g[rid][p], got_p[rid][p]), (rid, p)
            trios.append((f"{rid} pos {p}", got_g[rid][p], got_p[rid][p]))
    check_rows(trios, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_many_live_requests(tmp_path, dtype):
    """More live requests than a block of the attention kernel has tokens, prompts beside single tokens,
    then single tokens only while the batch walks down through every size."""
    d = model_dir(tmp_path, "kd", dtype)
    requests = _requests(130, [30 + 7 * (i % 5) for i in range(18)], 300)
    steps = H.plan_many(requests, seed=4, max_live=12)
    outputs, engine = H.run_engine(d, dtype, steps, 16, H.max_live_tokens(steps, 16) + 32, max_requests=12)
    compare(d, requests, H.collect(steps, outputs), dtype)


@pytest.mark.gpu
def test_portions_on_either_side_of_the_prompt_kernels_threshold(tmp_path):
    """A model whose latents the tcgen05 kernel takes, in bfloat16: long portions run there, short ones and
    single tokens on the kernel that cuts a tile's keys into stretches, all on the same cached entries."""
    from fastgen_b200.csrc.ops import Ops

    cfg = dict(architecture="Kuvusun", vocab=150, width=120, norm=dict(eps=1e-5, groups=2), layers=[
        _layer(_turned(40, 16, 16, 8, 64, 0.2, 3000.0), _dense(72)), _layer(_plain(33, 16, 8, 40, 128, 0.2), _dense(64)),
        _layer(_turned(20, 8, 16, 16, 64, 0.25, 3000.0, kv_from=0), None)])
    d = write_random_model(Path(tmp_path) / "m", cfg, 4, dtype=torch.bfloat16, norm_jitter=0.3, std=0.1)
    taken = []
    inner = Ops._latent_tc5

    def spy(self, *args):
        taken.append(inner(self, *args))
        return taken[-1]
    requests = _requests(150, [260, 170], 21)
    try:
        Ops._latent_tc5 = spy
        for sizes in ((260,), (150, 1, 1, 2, 3, 103), (17, 130, 1, 9, 103)):
            steps = H.plan_portions(requests, sizes=sizes)
            outputs, _ = H.run_engine(d, torch.bfloat16, steps, 16, H.max_live_tokens(steps, 16) + 32)
            compare(d, requests, H.collect(steps, outputs), torch.bfloat16)
    finally:
        Ops._latent_tc5 = inner
    assert any(taken) and not all(taken)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_long_decoding(tmp_path, dtype):
    """200 tokens decoded one by one after a two-token prompt, over many pages of eight."""
    d = model_dir(tmp_path, "ka", dtype)
    requests = _requests(211, [202], 77)
    steps = H.plan_decode_tail(requests, 200)
    outputs, engine = H.run_engine(d, dtype, steps, 8, 232)
    compare(d, requests, H.collect(steps, outputs), dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["ka", "kc"])
def test_greedy_generation_through_the_entry_point(tmp_path, dtype, name):
    """``Fastgen.generate`` with its scheduler (portions of 16 tokens, batches of 3, graphs) against
    greedy decoding with the plain implementation."""
    from fastgen_b200.engine import Fastgen, GenArgs, HfLoader, Packet

    d = model_dir(tmp_path, name, dtype)
    cfg, w = pk.read_model(d)
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
            assert got[i] == pk.greedy(cfg, w, p, 12), i
        else:
            seq = list(p)
            for tok in got[i]:
                logits = pk.forward(cfg, w, seq)[-1]
                assert float(logits[tok]) >= float(logits.max()) - 0.03 * float(logits.abs().max())
                seq.append(tok)
