"""Linurax configuration and spec building (no GPU): keys, validation, tensor names and shapes, cache and state registration,
the planning of the attention's work items, and the plain implementation's own mechanisms."""
import copy

import numpy as np
import pytest
import torch

import plain_linurax as plain
from linurax_cases import CASES, CASE_A, CASE_B, CASE_D, CASE_E, CASE_F, make_folder, read_folder, tokens_for

from openinfer_b200.cache.manager import CacheManager, KvNeed
from openinfer_b200.config.base import ConfigError, load_config, resolve_architecture
from openinfer_b200.parts.model import Model


def build(cfg):
    entry = resolve_architecture(cfg)
    config = entry.config_cls.from_dict(cfg)
    return config, entry.build_spec(config)


def test_registry_and_what_the_spec_takes_from_the_configuration():
    config, spec = build(CASE_A)
    assert type(config).__name__ == "LinuraxConfig"
    assert spec.residual_dtype == "float32" and spec.vocab_size == 211 and spec.hidden_size == 64
    assert spec.embedding_scale == 30.0 and spec.head_name is None and spec.final_norm.eps == 1e-5
    assert [b.kind for b in spec.blocks] == ["branchnorm"] * 4
    first, att, att2, last = spec.blocks
    assert (first.mixer.kind, first.mixer.channels, first.feed_forward) == ("mingru", 40, None)
    m = att.mixer
    assert (m.kind, m.num_heads, m.num_kv_heads, m.qk_dim, m.v_dim, m.score_scale) == ("sigmoid_attention", 4, 2, 16, 16, 0.4)
    assert m.values_from_keys and m.mix_heads and m.score_bias and m.output_gate and m.joint_norm_eps == 1e-5
    assert m.position.interleaved and (m.position.rotary_dim, m.position.theta) == (8, 1000.0)
    assert (att.feed_forward.intermediate_size, att.feed_forward.activation) == (48, "silu")
    assert att2.feed_forward is None and att2.post_norm is None and last.feed_forward.intermediate_size == 72
    assert build(CASE_B)[1].blocks[1].mixer.position.kind == "none"
    assert type(config).from_dict(config.to_dict()) == config


@pytest.mark.parametrize("name", list(CASES))
def test_tensor_names_and_shapes(name):
    cfg = CASES[name][0]
    exp = Model(build(cfg)[1], torch.bfloat16).expected_tensors()
    W = cfg["width"]
    want = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        want[p + "norm1"] = (W,)
        if layer["type"] == "mingru":
            C = m["width"]
            want.update({p + "mix.z": (C, W), p + "mix.z.b": (C,), p + "mix.x": (C, W), p + "mix.x.b": (C,), p + "mix.g": (C, W),
                         p + "mix.o": (W, C)})
        else:
            H, G, D = m["heads"], m["kv_heads"], m["dim"]
            want.update({p + "mix.q": (H * D, W), p + "mix.k": (G * D, W), p + "mix.q.norm": (H * D,), p + "mix.k.norm": (G * D,),
                         p + "mix.talk": (H, H), p + "mix.pb": (H,), p + "mix.g": (H * D, W), p + "mix.o": (W, H * D)})
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            want.update({p + "norm2": (W,), p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    assert {k: tuple(v.shape) for k, v in exp.items()} == want


def test_random_folders_load_back(tmp_path):
    path = make_folder(str(tmp_path / "m"), CASE_D, 3)
    cfg, tensors = read_folder(path)
    assert cfg["architecture"] == "Linurax" and load_config(path).width == 36
    assert tensors["l0.mix.talk"].shape == (3, 3) and all(t.dtype == torch.bfloat16 for t in tensors.values())


def test_cache_and_state_registration():
    model = Model(build(CASE_A)[1], torch.bfloat16)
    cache = CacheManager(page_size=16)
    model.bind_cache(cache)
    assert [g.need for g in cache.groups] == [KvNeed(2, 16), KvNeed(1, 24)]
    assert [(n.shape, n.dtype, n.phases) for n in cache.state_needs] == [((40,), "float32", 1), ((96,), "float32", 1)]
    for cfg, groups, states in ((CASE_E, 0, 2), (CASE_F, 2, 0)):
        model, cache = Model(build(cfg)[1], torch.bfloat16), CacheManager(page_size=16)
        model.bind_cache(cache)
        assert (len(cache.groups), len(cache.state_needs)) == (groups, states)
    # heads of 10 and 6 numbers are cached in rows of 16 and 8
    model, cache = Model(build(CASE_D)[1], torch.bfloat16), CacheManager(page_size=16)
    model.bind_cache(cache)
    assert [g.need.head_dim for g in cache.groups] == [16, 8]


def _bad(change):
    cfg = copy.deepcopy(CASE_A)
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].__setitem__("type", "gru"), "not known"),
    (lambda c: c["layers"][0]["mixer"].pop("width"), "width"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 3), "do not divide"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("vdim", 8), "must equal dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 18), "at most dim"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "moe"), "kind must be"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c.__setitem__("layers", []), "at least one layer"),
    (lambda c: c.__setitem__("width", 0), "positive"),
])
def test_bad_configs_are_refused(change, message):
    with pytest.raises(ConfigError) as e:
        build(_bad(change))
    assert message in str(e.value)


def test_specs_the_mixer_cannot_serve_are_refused():
    from openinfer_b200.parts.registry import build_mixer
    from openinfer_b200.parts.spec import PositionSpec, SigmoidAttentionSpec
    good = dict(hidden_size=32, num_heads=4, num_kv_heads=2, qk_dim=16, v_dim=16)
    build_mixer(SigmoidAttentionSpec(**good))
    for bad in (dict(num_kv_heads=3), dict(values_from_keys=True, v_dim=8), dict(qk_dim=600),
                dict(position=PositionSpec(kind="rope", rotary_dim=8, max_positions=64))):
        with pytest.raises(ValueError):
            build_mixer(SigmoidAttentionSpec(**{**good, **bad}))


def test_work_items_cover_every_key_once():
    """Whatever the batch: every portion of two tokens or more is cut into tiles, every tile's and every single token's keys
    into slices numbered from zero, rows of several slices own disjoint places for their partial results."""
    from openinfer_b200.kernels.sigmoid_attention import plan_items
    for q_lens, kv_lens, tt in (([1], [1], 16), ([2048], [2048], 16), ([3, 1, 40, 1], [3, 900, 1000, 1], 8), ([17, 16], [17, 700], 32),
                                ([5000], [9000], 16)):
        tiles, decode, splits, base, part_rows = plan_items(q_lens, kv_lens, tt, 148)
        starts = np.concatenate([[0], np.cumsum(q_lens)])
        seen = {}
        for b, t0, s, ns in tiles.tolist():
            assert q_lens[b] > 1 and t0 % tt == 0 and t0 < q_lens[b] and 0 <= s < ns
            seen.setdefault((b, t0), []).append(s)
            rows = slice(starts[b] + t0, starts[b] + min(t0 + tt, q_lens[b]))
            assert (splits[rows] == ns).all()
        assert set(seen) == {(b, t0) for b, n in enumerate(q_lens) if n > 1 for t0 in range(0, n, tt)}
        for b, _, s, ns in decode.tolist():
            assert q_lens[b] == 1 and splits[starts[b]] == ns
            seen.setdefault(b, []).append(s)
        assert all(sorted(v) == list(range(len(v))) for v in seen.values())
        assert all(b in seen for b, n in enumerate(q_lens) if n == 1)
        taken = [p for t in range(len(splits)) if splits[t] > 1 for p in range(base[t], base[t] + splits[t])]
        assert sorted(taken) == list(range(part_rows))


def test_plain_mechanisms():
    # the turn of neighbours: number pairs, position zero stands still, the rest of the head passes
    x = torch.randn(3, 2, 6, dtype=torch.float64)
    y = plain.turn_neighbours(x, torch.tensor([0, 1, 5]), 10.0, 4)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    a = torch.tensor(5 * 10.0 ** -0.5)
    assert torch.allclose(y[2, 1, 2], x[2, 1, 2] * torch.cos(a) - x[2, 1, 3] * torch.sin(a))
    # mixing: one head's scores are another's
    q, k = torch.randn(4, 2, 3, dtype=torch.float64), torch.randn(4, 1, 3, dtype=torch.float64)
    plainly = plain.talking_scores(q, k, 0.5, torch.eye(2, dtype=torch.float64))
    swapped = plain.talking_scores(q, k, 0.5, torch.tensor([[0.0, 1.0], [2.0, 0.0]], dtype=torch.float64))
    assert torch.allclose(swapped[0], plainly[1]) and torch.allclose(swapped[1], 2.0 * plainly[0])
    assert torch.allclose(plainly[1, 2, 1], 0.5 * (q[2, 1] * k[1, 0]).sum())
    # weights do not sum to one and do not see later keys
    w = plain.sigmoid_weights(torch.zeros(1, 3, 3), torch.tensor([0.0]))
    assert torch.equal(w[0], 0.5 * torch.ones(3, 3).tril())
    # the recurrence: a closed gate keeps, an open one takes the candidate on either side of zero
    z, u = torch.tensor([[1.0], [0.0], [0.25], [1.0]]), torch.tensor([[2.0], [9.0], [0.0], [-1.0]])
    S = plain.mingru_states(z, u)[:, 0]
    assert torch.allclose(S, torch.tensor([2.5, 2.5, 0.75 * 2.5 + 0.25 * 0.5, float(torch.sigmoid(torch.tensor(-1.0)))]))


def test_plain_forward_is_causal_and_every_mechanism_moves_the_logits(tmp_path):
    path = make_folder(str(tmp_path / "m"), CASE_A, 5)
    cfg, tensors = read_folder(path)
    toks = tokens_for(cfg, 60, 1)
    ref = plain.forward(cfg, tensors, toks)
    other = plain.forward(cfg, tensors, toks[:40] + [(t + 1) % cfg["vocab"] for t in toks[40:]])
    assert torch.equal(ref[:40], other[:40]) and not torch.allclose(ref[40:], other[40:])
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

    assert moved(lambda c: c["embedding"].__setitem__("scale", 29.0)) > 1e-4
    assert moved(lambda c: c["layers"][1]["mixer"].__setitem__("scale", 0.5)) > 1e-4
    assert moved(lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 10)) > 1e-4
    assert moved(lambda c: c["layers"][2]["mixer"]["rot"].__setitem__("base", 51.0)) > 1e-4
    assert moved(lambda c: c["norm"].__setitem__("eps", 1e-2)) > 1e-4
    for name in ("l1.mix.talk", "l1.mix.pb", "l1.mix.g", "l2.mix.k", "l2.mix.q.norm", "l2.mix.k.norm", "l0.mix.z", "l0.mix.z.b",
                 "l0.mix.x.b", "l3.mix.g", "l3.mlp.gate", "l3.norm2", "l0.norm1", "final.norm"):
        assert moved(None, scaled(name, 0.5)) > 1e-5, name
