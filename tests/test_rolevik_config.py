"""Rolevik configuration and spec building (no GPU): keys, validation, tensor names and shapes, cache and state registration,
pages given back by chunks, work items under chunks, and the plain implementation's own mechanisms."""
import copy
import math

import pytest
import torch

import plain_rolevik as plain
from rolevik_cases import (CASE_A, CASE_B, CASE_C, CASE_D, CASE_E, CASES, attn, delta, make_folder, model, par, read_folder, tokens_for)

from openinfer_b200.cache.manager import RELEASED, CacheManager, KvNeed
from openinfer_b200.config.base import ConfigError, load_config, resolve_architecture
from openinfer_b200.parts.model import Model


def build(cfg):
    entry = resolve_architecture(cfg)
    config = entry.config_cls.from_dict(cfg)
    return config, entry.build_spec(config)


def test_registry_and_what_the_spec_takes_from_the_configuration():
    config, spec = build(CASE_A)
    assert type(config).__name__ == "RolevikConfig"
    assert spec.residual_dtype == "float32" and spec.vocab_size == 211 and spec.hidden_size == 64
    assert (spec.embedding_scale, spec.logit_scale, spec.head_name) == (9.0, 0.7, None)
    assert (spec.final_norm.kind, spec.final_norm.eps) == ("layer", 1e-5)
    assert [b.kind for b in spec.blocks] == ["branchnorm"] * 4
    first, second, third, last = spec.blocks
    m = first.mixer
    assert (m.kind, m.channels, m.blocks, m.conv_taps, m.rate) == ("rglru", 40, 5, 4, 8.0)
    f = first.feed_forward
    assert (f.routing, f.experts, f.identity, f.top, f.groups, f.keep_groups, f.weight_scale, f.activation) == \
        ("softmax_groups", 6, 2, 2, 4, 2, 1.7, "silu")
    assert (f.shared.intermediate_size, f.shared.activation) == (40, "silu")
    left, right = second.mixer.left, second.mixer.right
    assert (left.num_heads, left.num_kv_heads, left.qk_dim, left.v_dim, left.head_dim, left.softmax_scale) == (4, 2, 16, 24, 24, 0.4)
    assert (left.window, left.chunked, left.qkv_bias, left.joint_norm_eps, left.qk_norm) == (21, True, True, 1e-5, None)
    assert (left.position.rotary_dim, left.position.theta, left.position.interleaved) == (8, 1000.0, False)
    assert (right.num_heads, right.num_kv_heads, right.qk_dim, right.v_dim, right.conv_taps) == (4, 2, 8, 20, 3)
    assert (right.decay_per, right.gate_activation) == ("head", "silu")
    assert (second.mixer.left_scale, second.mixer.right_scale, second.mixer.out_norm_eps) == (0.5, 0.5, 1e-5)
    assert (second.feed_forward.kind, second.feed_forward.activation) == ("gated_mlp", "gelu_tanh")
    assert third.feed_forward is None and third.feed_forward_scale is None and third.mixer_scale is not None
    assert last.feed_forward.shared is None
    b = build(CASE_B)[1].blocks
    assert b[0].mixer.left.window is None and not b[0].mixer.left.chunked and b[1].mixer.left.position.kind == "none"
    assert (b[0].feed_forward.identity, b[0].feed_forward.groups, b[0].feed_forward.weight_scale) == (0, 1, 1.0)
    assert type(config).from_dict(config.to_dict()) == config


@pytest.mark.parametrize("name", list(CASES))
def test_tensor_names_and_shapes(name):
    cfg = CASES[name][0]
    exp = Model(build(cfg)[1], torch.bfloat16).expected_tensors()
    W = cfg["width"]
    want = {"embed": (cfg["vocab"], W), "final.norm": (W,)}

    def gated(p, F):
        want.update({p + "gate": (F, W), p + "up": (F, W), p + "down": (W, F)})

    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        want[p + "norm1"] = want[p + "ls1"] = (W,)
        if layer["type"] == "rglru":
            C, B, n = m["width"], m["blocks"], m["width"] // m["blocks"]
            for t in ("y", "x"):
                want.update({p + f"mix.{t}": (C, W), p + f"mix.{t}.b": (C,)})
            want.update({p + "mix.conv": (C, m["conv"]), p + "mix.conv.b": (C,), p + "mix.lam": (C,), p + "mix.o": (W, C)})
            for t in ("ra", "ri"):
                want.update({p + f"mix.{t}": (B, n, n), p + f"mix.{t}.b": (B, n)})
        else:
            a, d = m["left"], m["right"]
            H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            for t, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
                want.update({q + t: (rows, W), q + t + ".b": (rows,)})
            want.update({q + "q.norm": (H * D,), q + "k.norm": (G * D,), q + "o": (W, H * V), q + "out": (W,)})
            H, G, D, V, q = d["heads"], d["kv_heads"], d["dim"], d["vdim"], p + "mix.right."
            for t, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                want.update({q + t: (rows, W), q + t + ".conv": (rows, d["conv"])})
            want.update({q + "b": (H, W), q + "a": (H, W), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (V,), q + "g": (H * V, W),
                         q + "o": (W, H * V), q + "out": (W,)})
        f = layer["mlp"]
        if f:
            want[p + "norm2"] = want[p + "ls2"] = (W,)
            if f["kind"] == "dense":
                gated(p + "mlp.", f["ff"])
            else:
                n = f["router"]["experts"] + f["router"].get("identity", 0)
                want.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
                for e in range(f["router"]["experts"]):
                    gated(p + f"mlp.e{e}.", f["expert"]["ff"])
                if f.get("shared"):
                    gated(p + "mlp.shared.", f["shared"]["ff"])
    assert {k: tuple(v.shape) for k, v in exp.items()} == want


def test_random_folders_load_back(tmp_path):
    path = make_folder(str(tmp_path / "m"), CASE_D, 3)
    cfg, tensors = read_folder(path)
    assert cfg["architecture"] == "Rolevik" and load_config(path).width == 36
    assert tensors["l1.mix.ra"].shape == (3, 11, 11) and all(t.dtype == torch.bfloat16 for t in tensors.values())


def test_cache_and_state_registration():
    m, cache = Model(build(CASE_A)[1], torch.bfloat16), CacheManager(page_size=16)
    m.bind_cache(cache)
    assert [g.need for g in cache.groups] == [KvNeed(2, 24, 21, chunked=True), KvNeed(1, 24, 48, chunked=True)]
    assert [(n.shape, n.phases) for n in cache.state_needs] == [
        ((40,), 1), ((3, 40), 2),                            # the recurrent unit and its filter
        ((4, 160), 2), ((2, 2 * 16 + 80), 2),                # the delta rule and its filter (q | k | v)
        ((3, 240), 2), ((1, 2 * 60 + 36), 2), ((96,), 1), ((1, 96), 2)]
    m, cache = Model(build(CASE_B)[1], torch.bfloat16), CacheManager(page_size=16)
    m.bind_cache(cache)
    assert [g.need for g in cache.groups] == [KvNeed(6, 16), KvNeed(1, 40, 1, chunked=True), KvNeed(5, 16, 16, chunked=True)]
    m, cache = Model(build(CASE_E)[1], torch.bfloat16), CacheManager(page_size=16)
    m.bind_cache(cache)
    assert not cache.groups and len(cache.state_needs) == 4
    # two chunk sizes and a window of the same number are groups of their own
    cache = CacheManager(page_size=16)
    handles = [cache.add_kv_layer(n) for n in (KvNeed(1, 8, 5, chunked=True), KvNeed(1, 8, 5), KvNeed(1, 8, 5, chunked=True))]
    assert [(h.group, h.layer) for h in handles] == [(0, 0), (1, 0), (0, 1)]


@pytest.mark.parametrize("chunk,page", [(7, 4), (16, 16), (21, 16), (1, 2), (64, 16), (100, 8)])
def test_pages_behind_a_chunk_go_back(chunk, page):
    """After every step exactly the pages that hold a key the next query can still see are kept."""
    cache = CacheManager(page_size=page)
    cache.add_kv_layer(KvNeed(1, 8, chunk, chunked=True))
    cache.allocate(64, 1)
    cache.open("r")
    at = 0
    for n in (3, 1, 1, 2, 30, 1, 17, 2, 64, 1, 1, 1, 5):
        cache.reserve("r", n)
        cache.commit("r")
        at += n
        first = at - at % chunk                     # the next query sees the keys from here on
        table = cache.block_table("r", 0)
        for i, p in enumerate(table):
            assert (p == RELEASED) == ((i + 1) * page <= first), (at, i)
        cache.check()
    cache.close("r")
    assert cache.min_free_pages() == 64


def test_work_items_under_chunks():
    from openinfer_b200.kernels.attention import KEYS_PER_TILE, decode_splits, first_visible, plan_items
    assert [first_visible(p, -7) for p in (0, 6, 7, 13, 14)] == [0, 0, 7, 7, 14]
    assert [first_visible(p, 7) for p in (0, 6, 7, 13)] == [0, 0, 1, 7] and first_visible(99, None) == 0 and first_visible(99, 0) == 0
    for chunk in (5, 64, 100):
        tiles, _, _, _, _ = plan_items([300, 41], [300, 700], 2, 4, -chunk, 148, rows_per_cta=128)
        assert sorted({(b, t) for b, t, _, _ in tiles.tolist()}) == [(b, t) for b, n in ((0, 300), (1, 41)) for t in range(0, n, 64)]
        for b, t0, s, ns in tiles.tolist():
            pos0 = (0, 659)[b] + t0
            span = -(-(pos0 + min(64, (300, 41)[b] - t0) - (first_visible(pos0, -chunk) & ~(KEYS_PER_TILE - 1))) // KEYS_PER_TILE)
            assert 0 <= s < ns <= max(1, span)
    # a row's keys are cut no finer than its chunk allows
    assert decode_splits(1, 1, 148, 100000, chunk=64) == decode_splits(1, 1, 148, 64)
    assert decode_splits(1, 1, 148, None, 100000, chunk=256) == decode_splits(1, 1, 148, 256)


def _bad(change):
    cfg = copy.deepcopy(CASE_A)
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].__setitem__("type", "lru"), "not known"),
    (lambda c: c["layers"][0]["mixer"].pop("width"), "width"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("blocks", 3), "does not divide"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("conv", 0), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][1]["mixer"]["left"].__setitem__("kv_heads", 3), "do not divide"),
    (lambda c: c["layers"][1]["mixer"]["right"].__setitem__("kv_heads", 3), "do not divide"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 7), "even"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 18), "at most dim"),
    (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "table"), "kind must be"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"].pop("expert"), "expert"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("groups", {"count": 3, "keep": 1}), "cannot give"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("groups", {"count": 4, "keep": 5}), "cannot give"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("groups", {"count": 8, "keep": 1}), "cannot give"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("identity", -1), "identity"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c.__setitem__("layers", []), "at least one layer"),
    (lambda c: c.__setitem__("width", 0), "positive"),
])
def test_bad_configs_are_refused(change, message):
    with pytest.raises(ConfigError) as e:
        build(_bad(change))
    assert message in str(e.value)


def test_specs_the_parts_cannot_serve_are_refused():
    from openinfer_b200.parts.registry import build_block, build_feed_forward, build_mixer
    from openinfer_b200.parts.spec import (AttentionSpec, BlockSpec, DepthAverageSpec, GatedDeltaSpec, LayerScaleSpec, MinGruSpec, NormSpec,
                                           RgLruSpec, RoutedExpertsSpec)
    good = dict(hidden_size=32, num_heads=4, num_kv_heads=2, head_dim=16, joint_norm_eps=1e-5)
    build_mixer(AttentionSpec(**good))
    for bad in (dict(qk_norm=NormSpec(size=16)), dict(unit_norm_after_rotation_eps=1e-5), dict(conv_taps=2),
                dict(window=8, chunked=True, keep_first=2)):
        with pytest.raises(ValueError):
            build_mixer(AttentionSpec(**{**good, **bad}))
    for bad in (dict(blocks=5), dict(conv_taps=0), dict(channels=0)):
        with pytest.raises(ValueError):
            build_mixer(RgLruSpec(**{**dict(hidden_size=32, channels=12, blocks=3, conv_taps=2), **bad}))
    with pytest.raises(ValueError):
        build_mixer(GatedDeltaSpec(hidden_size=32, num_heads=2, num_kv_heads=1, qk_dim=8, v_dim=8, conv_taps=2, decay_per="row"))
    experts = dict(hidden_size=32, intermediate_size=8, experts=6, top=2, activation="silu", routing="softmax_groups", identity=2, groups=4, keep_groups=1)
    build_feed_forward(RoutedExpertsSpec(**experts))
    for bad in (dict(groups=3), dict(top=3), dict(routing="softmax_top"), dict(identity=-1)):
        with pytest.raises(ValueError):
            build_feed_forward(RoutedExpertsSpec(**{**experts, **bad}))
    norm = NormSpec(kind="layer", size=32)
    with pytest.raises(ValueError):                           # an average over depth joins by the rms kernel only
        build_block(BlockSpec(kind="branchnorm", mixer=MinGruSpec(hidden_size=32, channels=8), input_norm=norm, mixer_scale=LayerScaleSpec(size=32),
                              depth_average=DepthAverageSpec(terms=2)))
    with pytest.raises(ValueError):                           # blocks that fuse an rms norm do not take a layer norm for one
        build_block(BlockSpec(kind="shared_norm", mixer=MinGruSpec(hidden_size=32, channels=8), input_norm=norm))


# ---------------------------------------------------------------------------------------------- the plain implementation
def test_plain_mechanisms():
    f64 = torch.float64
    # the layer norm: no mean, unit variance
    y = plain.layer_norm(torch.randn(3, 50, dtype=f64) * 4 + 7, torch.ones(50, dtype=f64), 0.0)
    assert torch.allclose(y.mean(-1), torch.zeros(3, dtype=f64), atol=1e-12) and torch.allclose((y * y).mean(-1), torch.ones(3, dtype=f64))
    # the turn of halves: position zero stands still, the rest of the head passes
    x = torch.randn(3, 2, 6, dtype=f64)
    y = plain.turn_halves(x, torch.tensor([0, 1, 5]), 10.0, 4)
    a = torch.tensor(5 * 10.0 ** -0.5, dtype=f64)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    assert torch.allclose(y[2, 1, 1], x[2, 1, 1] * torch.cos(a) - x[2, 1, 3] * torch.sin(a))
    assert torch.allclose(y[2, 1, 3], x[2, 1, 3] * torch.cos(a) + x[2, 1, 1] * torch.sin(a))
    # chunks
    seen = plain.chunk_mask(7, 3)
    assert seen.sum(dim=1).tolist() == [1, 2, 3, 1, 2, 3, 1] and not seen[3, 2] and plain.chunk_mask(4, None)[3].all()
    # softmax attention with equal scores is a mean over the keys seen
    v = torch.randn(7, 1, 2, dtype=f64)
    o = plain.softmax_attention(torch.zeros(7, 2, 3, dtype=f64), torch.zeros(7, 1, 3, dtype=f64), v, 1.0, seen)
    assert torch.allclose(o[4, :2], v[3:5, 0].mean(0)) and torch.allclose(o[4, :2], o[4, 2:])
    # the filter: the last column is the current row's
    y = plain.causal_filter(torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[3.0, 2.0]]), torch.tensor([0.5]))
    assert y[:, 0].tolist() == [2.5, 23.5, 230.5]
    # the delta rule: a full correction writes the value itself along a unit key, and the read-out sees it
    k = plain.unit(torch.tensor([[[3.0, 4.0]]], dtype=f64).repeat(2, 1, 1))
    vals = torch.tensor([[[1.0, 2.0]], [[5.0, -1.0]]], dtype=f64)
    one = torch.ones(2, 1, dtype=f64)
    o = plain.delta_rule(k, k, vals, one, 0.5 * one)
    assert torch.allclose(o, vals, atol=1e-6)
    o = plain.delta_rule(k, k, vals, torch.tensor([[1.0], [0.0]], dtype=f64), 0.5 * one)
    assert torch.allclose(o[1], 0.5 * vals[0], atol=1e-6)
    # the recurrent unit: r = 0 keeps, a large r forgets
    u, r = torch.tensor([[1.0], [9.0], [3.0]], dtype=f64), torch.tensor([[1.0], [0.0], [1.0]], dtype=f64)
    lam = torch.tensor([20.0], dtype=f64)
    S = plain.rglru_states(u, r, torch.ones_like(u), lam)[:, 0]
    assert torch.allclose(S, torch.tensor([1.0, 1.0, 3.0], dtype=f64))
    lam = torch.tensor([-1.5], dtype=f64)
    a = math.exp(-8 * 0.3 * math.log1p(math.exp(-1.5)))
    S = plain.rglru_states(u[:1], 0.3 * torch.ones(1, 1, dtype=f64), 0.5 * torch.ones(1, 1, dtype=f64), lam, S=torch.tensor([2.0], dtype=f64))
    assert math.isclose(S.item(), a * 2.0 + math.sqrt(1 - a * a) * 0.5, rel_tol=1e-12)
    # the gates: parts do not see one another
    w = torch.randn(2, 3, 3, dtype=f64)
    uu = torch.randn(1, 6, dtype=f64)
    g = plain.block_gates(uu, w, torch.zeros(2, 3, dtype=f64))
    assert torch.allclose(g[0, 3:], torch.sigmoid(w[1] @ uu[0, 3:]))


def test_plain_choice_of_experts():
    z = torch.log(torch.tensor([[0.30, 0.02, 0.28, 0.25, 0.10, 0.05]], dtype=torch.float64))
    c = torch.zeros(6, dtype=torch.float64)
    s, e = plain.choose(z, c, 2, 1, 1)
    assert torch.allclose(s.sum(), torch.ones((), dtype=torch.float64)) and sorted(e[0].tolist()) == [0, 2]
    assert sorted(plain.choose(z, c, 2, 3, 1)[1][0].tolist()) == [0, 1]           # the best group is the one with the single best member
    assert sorted(plain.choose(z, c, 2, 3, 2)[1][0].tolist()) == [0, 2]
    c[5], c[0], c[1] = 0.9, -0.9, -0.9                                            # the correction moves the choice, not the scores
    s2, e2 = plain.choose(z, c, 2, 3, 1)
    assert torch.equal(s, s2) and sorted(e2[0].tolist()) == [4, 5]
    # every choice score below zero: the groups left out stay out
    assert sorted(plain.choose(z, c - 2.0, 2, 3, 1)[1][0].tolist()) == [4, 5]
    assert math.isclose(plain.choice_margin(z, torch.zeros(6, dtype=torch.float64), 2, 1, 1).item(), 0.03, rel_tol=1e-9)
    assert math.isclose(plain.choice_margin(z, torch.zeros(6, dtype=torch.float64), 1, 3, 1).item(), 0.02, rel_tol=1e-9)


def test_plain_forward_is_causal_and_every_mechanism_moves_the_logits(tmp_path):
    path = make_folder(str(tmp_path / "m"), CASE_A, 5)
    cfg, tensors = read_folder(path)
    toks = tokens_for(cfg, 60, 1)
    ref = plain.forward(cfg, tensors, toks)
    other = plain.forward(cfg, tensors, toks[:40] + [(t + 1) % cfg["vocab"] for t in toks[40:]])
    assert torch.allclose(ref[:40], other[:40], rtol=0, atol=1e-12) and not torch.allclose(ref[40:], other[40:])
    size = ref.pow(2).mean().sqrt().item()

    def moved(change_cfg=None, change_tensors=None):
        c, t = copy.deepcopy(cfg), dict(tensors)
        if change_cfg:
            change_cfg(c)
        if change_tensors:
            change_tensors(t)
        return (plain.forward(c, t, toks) - ref).abs().max().item() / size

    def scaled(name, by=-1.0):
        return lambda t: t.__setitem__(name, t[name] * by)

    assert moved(lambda c: c.__setitem__("logit_scale", 0.71)) > 1e-4
    assert moved(lambda c: c["embedding"].__setitem__("scale", 8.9)) > 1e-4
    assert moved(lambda c: c["layers"][1]["mixer"]["left"].__setitem__("scale", 0.5)) > 1e-4
    assert moved(lambda c: c["layers"][1]["mixer"]["left"]["mask"].__setitem__("size", 22)) > 1e-4
    assert moved(lambda c: c["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 10)) > 1e-4
    assert moved(lambda c: c["layers"][2]["mixer"]["left"]["rot"].__setitem__("base", 51.0)) > 1e-4
    assert moved(lambda c: c["layers"][0]["mlp"]["router"].__setitem__("scale", 1.6)) > 1e-4
    assert moved(lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("keep", 1)) > 1e-4
    assert moved(lambda c: c["norm"].__setitem__("eps", 1e-2)) > 1e-4
    for name in ("l0.mix.y", "l0.mix.y.b", "l0.mix.x.b", "l0.mix.conv", "l0.mix.conv.b", "l0.mix.ra", "l0.mix.ra.b", "l0.mix.ri", "l0.mix.ri.b",
                 "l0.mix.lam", "l0.mlp.router", "l0.mlp.correction", "l0.mlp.shared.up", "l1.mix.left.q.b", "l1.mix.left.k.b", "l1.mix.left.v.b",
                 "l1.mix.left.q.norm", "l1.mix.left.k.norm", "l1.mix.left.out", "l1.mix.right.out", "l1.mix.right.k.conv", "l1.mix.right.v.conv",
                 "l1.mix.right.b", "l1.mix.right.a", "l1.mix.right.A_log", "l1.mix.right.dt_bias", "l1.mix.right.g", "l1.mix.right.norm",
                 "l1.mlp.gate", "l1.norm1", "l1.norm2", "l1.ls1", "l1.ls2", "final.norm"):
        assert moved(None, scaled(name, 0.5)) > 1e-6, name


def test_the_cases_share_no_sizes_by_accident():
    widths = [c["width"] for c, _ in CASES.values()]
    assert len(set(widths)) >= 5
    lefts = [l["mixer"]["left"] for c, _ in CASES.values() for l in c["layers"] if l["type"] == "parallel"]
    assert {a["heads"] // a["kv_heads"] for a in lefts} >= {1, 2, 3, 4, 8} and any(a["dim"] < a["vdim"] for a in lefts)
    assert model(5, 6, [par(attn(1, 1, 2, 2, 1.0), delta(1, 1, 2, 2, 1))])["logit_scale"] == 1.0
    assert CASE_C["layers"][0]["mixer"]["left"]["mask"]["size"] % 16 == 0
