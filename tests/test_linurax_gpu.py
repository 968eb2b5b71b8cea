"""Linurax in the engine against the plain implementation: the design's kernels alone, every mechanism alone in a model of one
layer, the stream behind every layer, whole prompts, decoding through cache and state, portions, mixed batches, pages and slots
that are used again, far keys, keys at page and tile borders, first tokens, long decoding, greedy generation through the
scheduler, the command line and the trace program."""
import json
import subprocess
import sys

import pytest
import torch

import plain_linurax as plain
from linurax_cases import (CASES, assert_logits, attn, bfloat16_noise, float32_noise, gru, make_folder, model, oracle, read_folder,
                           tokens_for)
from helpers import (ROOT, count_page_handouts, replay_in_process, replay_trace_run, round64, trace_mixed, trace_portions,
                     trace_tail, trace_whole)

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {n: make_folder(str(tmp_path_factory.mktemp(f"lnx{n}")), cfg, seed) for n, (cfg, seed) in CASES.items()}


def runner_for(path, dtype, max_tokens=2048, max_requests=4, page_size=16, graphs=True):
    from openinfer_b200.engine.runner import ModelRunner
    r = ModelRunner.from_folder(path, dtype=dtype, max_tokens=max_tokens, max_requests=max_requests, page_size=page_size)
    r.cuda_graph = graphs
    return r


def compare(got, path, toks, dtype, what, rows=slice(None), noise=None):
    assert_logits(got, oracle(path, toks)[rows], dtype, what, noise=float32_noise(path, toks) if noise is None else noise,
                  noise16=bfloat16_noise(path, toks))


def check_trace(runner, path, requests, steps, dtype, what):
    got = replay_in_process(runner, steps)
    for rid, toks in requests.items():
        compare(got[rid], path, toks, dtype, f"{what}/{rid}")


def _dev(t, dtype=None):
    return t.to(device="cuda", dtype=dtype or t.dtype)


def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


def save(path, tensors):
    from safetensors.torch import save_file
    save_file({k: v.contiguous() for k, v in tensors.items()}, path + "/model.safetensors")


# ---------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,hd,qk,rot_half,own_values,page", [(4, 2, 16, 16, 4, False, 16), (3, 1, 16, 10, 3, False, 4),
                                                                    (5, 5, 40, 40, 0, False, 8), (9, 3, 64, 64, 32, True, 16),
                                                                    (1, 1, 8, 6, 1, False, 2), (20, 5, 128, 128, 64, False, 16)])
def test_joint_norm_rotation_and_store_kernel(dtype, nq, nkv, hd, qk, rot_half, own_values, page):
    """q and k normed over all heads together, neighbouring pairs turned, q in place, k to its page, and as the value the key
    as it was projected (or columns of its own); a padding row stores nothing."""
    from openinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(nq * 100 + hd)
    T, pages, td = 7, 9, TORCH[dtype]
    k_off = nq * hd
    v_off = k_off + nkv * hd if own_values else k_off
    cols = v_off + nkv * hd + 8
    head = torch.arange(hd) < qk

    def rows(heads):
        return torch.randn(T, heads, hd, generator=g) * head

    q, k, v = rows(nq) * 3, rows(nkv) * 2, rows(nkv)
    proj = torch.zeros(T, cols)
    proj[:, : nq * hd] = q.reshape(T, -1)
    if own_values:
        proj[:, v_off: v_off + nkv * hd] = v.reshape(T, -1)
    proj[:, k_off: k_off + nkv * hd] = k.reshape(T, -1)
    proj = proj.to(td)
    qw, kw = ((1 + 0.2 * torch.randn(h, hd, generator=g)) * head for h in (nq, nkv))
    pos = [0, 3, 11, 12, 4, 30, 31]
    slots = [1, 0, 2 * page + 1, -1, 8 * page + page - 1, 3 * page, 4 * page]
    base, n = 77.0, torch.arange(max(rot_half, 1), dtype=torch.float64)
    ang = torch.arange(32, dtype=torch.float64)[:, None] * base ** (-2.0 * n / max(2 * rot_half, 1))[None, :]
    cos, sin = (_dev(f(ang).float().contiguous()) if rot_half else None for f in (torch.cos, torch.sin))
    kc, vc = (torch.full((pages, page, nkv, hd), 9.0, dtype=td, device="cuda") for _ in range(2))
    x = _dev(proj.clone())
    ops.joint_norm_rope_store(x, nq, nkv, hd, qk, k_off, v_off, q_norm_w=_dev(qw.reshape(-1)), k_norm_w=_dev(kw.reshape(-1)), eps=1e-3,
                              cos=cos, sin=sin, positions=_i32(pos), slots=_i32(slots), k_cache=kc, v_cache=vc, page_stride=kc.stride(0),
                              page_size=page)
    p64 = proj.double()

    def ready(cols0, heads, w):
        z = p64[:, cols0: cols0 + heads * hd].view(T, heads, hd)[..., :qk].reshape(T, -1)
        z = plain.rms(z, w.double()[:, :qk].reshape(-1), 1e-3).view(T, heads, qk)
        return plain.turn_neighbours(z, torch.tensor(pos), base, 2 * rot_half) if rot_half else z

    tol = 2e-6 if dtype == "float32" else 2e-2
    rq, rk = ready(0, nq, qw), ready(k_off, nkv, kw)
    rv = p64[:, v_off: v_off + nkv * hd].view(T, nkv, hd)[..., :qk]
    gq = x[:, : nq * hd].double().cpu().view(T, nq, hd)[..., :qk]
    assert (gq - rq).abs().max().item() < tol * max(1.0, rq.abs().max().item())
    written = torch.zeros(pages, page, dtype=torch.bool)
    for t, s in enumerate(slots):
        if s < 0:
            continue
        written[s // page, s % page] = True
        assert (kc[s // page, s % page, :, :qk].double().cpu() - rk[t]).abs().max().item() < tol * max(1.0, rk.abs().max().item())
        assert torch.equal(vc[s // page, s % page, :, :qk].double().cpu(), rv[t])
        assert qk == hd or (kc[s // page, s % page, :, qk:] == 0).all()
    assert (kc.cpu()[~written] == 9.0).all() and (vc.cpu()[~written] == 9.0).all()
    assert torch.equal(x[:, nq * hd:].cpu(), proj[:, nq * hd:])          # the keys stay as they were projected


def _attention_case(nq, nkv, hd, q_lens, kv_lens, page, td, seed):
    """Random q, gate and paged keys and values; the scores spread over tens, so that single keys decide a row."""
    import random
    import types
    g = torch.Generator().manual_seed(seed)
    T, B = sum(q_lens), len(q_lens)
    per = [-(-k // page) for k in kv_lens]
    ids = list(range(sum(per) + 3))
    random.Random(seed).shuffle(ids)
    table, at = torch.zeros(B, max(per), dtype=torch.int32), 0
    for b, n in enumerate(per):
        table[b, :n] = torch.tensor(ids[at: at + n], dtype=torch.int32)
        at += n
    kc, vc = (torch.randn(len(ids), page, nkv, hd, generator=g).to(td) for _ in range(2))
    proj = torch.randn(T, (2 * nq + nkv) * hd, generator=g).to(td)
    mix = (torch.eye(nq) + 0.3 * torch.randn(nq, nq, generator=g)).to(torch.bfloat16).float()
    bias = torch.randn(nq, generator=g) - 6.0
    starts = [0]
    for n in q_lens:
        starts.append(starts[-1] + n)
    ctx = types.SimpleNamespace(
        num_requests=B, cache=types.SimpleNamespace(page_size=page), scratch={}, q_lens_host=list(q_lens), kv_lens_host=list(kv_lens),
        token_req=_i32([b for b, n in enumerate(q_lens) for _ in range(n)]),
        positions=_i32([p for n, k in zip(q_lens, kv_lens) for p in range(k - n, k)]), cu_seqlens=_i32(starts))
    group = types.SimpleNamespace(block_table=_dev(table), kv_lens=_i32(kv_lens))
    return proj, kc, vc, mix, bias, table, starts, ctx, group


@pytest.mark.parametrize("tensor_cores", [True, False])
@pytest.mark.parametrize("nq,nkv,hd", [(9, 3, 64), (4, 1, 32), (8, 8, 64), (16, 4, 128), (12, 4, 64), (32, 8, 128), (20, 5, 32), (3, 3, 128),
                                       (1, 1, 64), (16, 16, 128), (24, 2, 32), (5, 1, 24), (2, 2, 256)])
def test_attention_kernels_over_paged_keys(nq, nkv, hd, tensor_cores):
    """The tensor-core kernels and the general one, on shuffled pages: prompt portions behind cached keys beside single tokens,
    key slices and none, every grouping of heads."""
    from openinfer_b200.kernels import sigmoid_attention as sa
    taken = hd in (32, 64, 128)
    if tensor_cores and not taken:
        pytest.skip("the general kernel serves this head size")
    scale = 5.0 * hd ** -0.5
    for td in ((torch.bfloat16,) if tensor_cores else (torch.float32, torch.bfloat16)):
        for page, q_lens, kv_lens in ((16, [1], [1]), (32, [2], [2]), (16, [5, 1], [37, 513]), (16, [1, 40, 1, 3], [16, 300, 17, 3]), (48, [70], [130])):
            proj, kc, vc, mix, bias, table, starts, ctx, group = _attention_case(nq, nkv, hd, q_lens, kv_lens, page, td, nq + hd + page)
            d = [_dev(t) for t in (proj, kc, vc, mix, bias)]
            out = torch.zeros(sum(q_lens), nq * hd, dtype=td, device="cuda")
            gate = d[0][:, (nq + nkv) * hd:]
            args = (d[0], out, gate, d[1], d[2], d[1].stride(0), ctx, group, nq, nkv, hd, scale, d[3], d[4])
            if tensor_cores:
                assert sa._tensor_cores(*args)
            else:
                sa._general(*args)
            for b, (n, kv) in enumerate(zip(q_lens, kv_lens)):
                rows = slice(starts[b], starts[b] + n)
                pages = table[b, : -(-kv // page)].long()
                k, v = (c[pages].reshape(-1, nkv, hd)[:kv].double() for c in (kc, vc))
                q = torch.zeros(kv, nq, hd, dtype=torch.float64)
                q[kv - n:] = proj[rows, : nq * hd].double().view(n, nq, hd)
                w = plain.sigmoid_weights(plain.talking_scores(q, k, scale, mix.double()), bias.double())
                ref = torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(nq // nkv, dim=1))[kv - n:].reshape(n, -1)
                ref = ref * torch.sigmoid(proj[rows, (nq + nkv) * hd:].double())
                err = (out[rows].double().cpu() - ref).abs().max().item() / max(1e-3, ref.abs().max().item())
                assert err < (1e-5 if td == torch.float32 else 1.2e-2), f"{td} page {page} request {b}: {err}"


def test_scores_are_mixed_in_more_than_sixteen_bits():
    """Scores of hundreds that cancel in the mix: with 16-bit scores the weights would be off by far more than rounding."""
    from openinfer_b200.kernels import sigmoid_attention as sa
    nq, nkv, hd = 8, 2, 64
    proj, kc, vc, mix, bias, table, starts, ctx, group = _attention_case(nq, nkv, hd, [40], [40], 16, torch.bfloat16, 3)
    q = proj[:, : nq * hd].view(40, nq, hd)
    q[:, 1] = q[:, 0]                                    # heads 0 and 1 share a kv head: equal scores, mixed with opposite signs
    mix[0] = 0.0
    mix[0, 0], mix[0, 1], mix[0, 5] = 32.0, -31.875, 0.5
    bias[0] = -2.0
    d = [_dev(t) for t in (proj, kc, vc, mix, bias)]
    outs = []
    for run in (sa._tensor_cores, sa._general):
        out = torch.zeros(40, nq * hd, dtype=torch.bfloat16, device="cuda")
        run(d[0], out, None, d[1], d[2], d[1].stride(0), ctx, group, nq, nkv, hd, 1.0, d[3], d[4])
        outs.append(out[:, :hd].double().cpu())
    pages = table[0].long()
    k, v = (c[pages].reshape(-1, nkv, hd)[:40].double() for c in (kc, vc))

    def reference(round_scores):
        s = plain.talking_scores(q.double(), k, 1.0, torch.eye(nq, dtype=torch.float64))
        s = s.bfloat16().double() if round_scores else s
        w = plain.sigmoid_weights(torch.einsum("hg,gij->hij", mix.double(), s), bias.double())
        return torch.einsum("ij,jd->id", w[0], v[:, 0])

    ref = reference(False)
    size = ref.abs().max().item()
    for out in outs:
        assert (out - ref).abs().max().item() < 1.2e-2 * size
    s16 = plain.talking_scores(q.double(), k, 1.0, torch.eye(nq, dtype=torch.float64))
    s16[0] = s16[0].bfloat16().double()                  # one of the two cancelling scores rounded to 16 bits
    w = plain.sigmoid_weights(torch.einsum("hg,gij->hij", mix.double(), s16), bias.double())
    assert (torch.einsum("ij,jd->id", w[0], v[:, 0]) - ref).abs().max().item() > 0.1 * size


@pytest.mark.parametrize("out_dtype", DTYPES)
@pytest.mark.parametrize("channels", [1, 33, 64, 520])
def test_gated_scan_kernel(channels, out_dtype):
    """Portions over old state beside a single token and a padding request; runs of rows that end inside a run, at a run's and
    at a round's edge."""
    from openinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(channels)
    step = -(-channels // 8) * 8
    for lens in ([7, 1, 256, 130], [1, 300], [2, 515, 5], [1, 1, 1]):
        T, B = sum(lens) + 1, len(lens) + 1
        zug = torch.randn(T, 3 * step, generator=g) * 2
        zug[0, :channels] = 40.0                          # an open gate forgets everything in front of it
        bias, state = torch.randn(2, channels, generator=g), torch.randn(B + 1, channels, generator=g)
        starts = [0]
        for n in lens + [1]:
            starts.append(starts[-1] + n)
        slots = list(range(B, 0, -1))

        class Ctx:
            cu_seqlens = _i32(starts)
            token_req = _i32([b for b, n in enumerate(lens) for _ in range(n)] + [-1])
            state_slots, num_requests, decode_only, q_lens_host = _i32(slots), B, max(lens) == 1, lens + [1]

        def run():
            y, s = torch.empty(T, channels, device="cuda", dtype=TORCH[out_dtype]), _dev(state.clone())
            ops.mingru_scan(y, _dev(zug), step, _dev(bias), s, Ctx)
            return y.double().cpu(), s.cpu()

        y, s = run()
        for b, n in enumerate(lens):
            z = torch.sigmoid(zug[starts[b]: starts[b] + n, :channels].double() + bias[0].double())
            u = zug[starts[b]: starts[b] + n, step: step + channels].double() + bias[1].double()
            # the old state enters as a first row with an open gate (its candidate cannot be any number: added by hand)
            S = plain.mingru_states(z, u) + torch.cumprod(1.0 - z, dim=0) * state[slots[b]].double()
            ref = S * plain.silu(zug[starts[b]: starts[b] + n, 2 * step: 2 * step + channels].double())
            got = y[starts[b]: starts[b] + n]
            assert (got - ref).abs().max().item() < (3e-6 if out_dtype == "float32" else 1e-2) * max(1.0, ref.abs().max().item())
            assert (s[slots[b]].double() - S[-1]).abs().max().item() < 3e-6 * max(1.0, S.abs().max().item())
        assert torch.equal(s[0], state[0]) and torch.equal(s[slots[-1]], state[slots[-1]])      # nobody's slot, and the padding's


# ---------------------------------------------------------------------------------------------- mechanisms alone
def _one_layer(layer, width=48, vocab=83, **kw):
    return model(vocab, width, [layer], **{"scale": 20.0, **kw})


MECHANISMS = {
    "recurrence of one channel": _one_layer(gru(1)),
    "recurrence wider than the model": _one_layer(gru(200)),
    "recurrence with a feed-forward": _one_layer(gru(24, mlp=70)),
    "one head, no rotation": _one_layer(attn(1, 1, 16, 0.5)),
    "mixed heads on one key head": _one_layer(attn(4, 1, 16, 0.5)),
    "mixed heads, a key head each": _one_layer(attn(5, 5, 8, 0.7)),
    "rotation of the first two numbers": _one_layer(attn(2, 1, 16, 0.5, rot=(2, 40.0))),
    "rotation of part of a head": _one_layer(attn(3, 1, 24, 0.4, rot=(10, 1000.0))),
    "rotation of the whole head": _one_layer(attn(2, 2, 32, 0.4, rot=(32, 10000.0))),
    "a rotation base below ten": _one_layer(attn(2, 1, 16, 0.5, rot=(16, 3.0))),
    "attention with a feed-forward": _one_layer(attn(6, 3, 8, 0.7, rot=(8, 100.0), mlp=33)),
    "heads of 264 numbers": _one_layer(attn(2, 1, 264, 0.1, rot=(64, 10000.0))),
    "heads of 64, groups of three": _one_layer(attn(9, 3, 64, 0.25, rot=(64, 10000.0))),
    "heads of 128, groups of eight": _one_layer(attn(16, 2, 128, 0.15, rot=(64, 10000.0))),
    "embedding as it is": _one_layer(gru(24), scale=1.0),
    "a large eps": _one_layer(attn(2, 1, 16, 0.5), eps=0.5),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MECHANISMS))
def test_each_mechanism_alone(tmp_path, name, dtype):
    """A model of one layer with one mechanism: a whole prompt, then portions of 2, 1, 5 and 3 tokens and decoding."""
    cfg = MECHANISMS[name]
    path = make_folder(str(tmp_path / "m"), cfg, 7)
    requests = {"a": tokens_for(cfg, 75, 1), "b": tokens_for(cfg, 40, 2)}
    runner = runner_for(path, dtype, max_tokens=256)
    check_trace(runner, path, requests, trace_whole(requests), dtype, name)
    check_trace(runner, path, requests, trace_portions(requests, sizes=(2, 1, 5, 3, 30, 1, 1, 2)), dtype, name + "/portions")


def test_options_of_the_mixer_that_the_design_does_not_use():
    """Values of their own, no head mix, no bias, no norm, no gate: the mixer's other forms, against the same formulas."""
    from openinfer_b200.cache.manager import CacheManager
    from openinfer_b200.engine.runner import ModelRunner, StepEntry
    from openinfer_b200.parts.model import Model
    from openinfer_b200.parts.spec import BlockSpec, ModelSpec, NormSpec, SigmoidAttentionSpec
    from openinfer_b200.weights.random import random_tensors
    W, V, H, G, D, VD = 40, 61, 4, 2, 16, 10
    for extra in (dict(), dict(mix_heads=True), dict(output_gate=True, score_bias=True), dict(joint_norm_eps=1e-5)):
        norm = NormSpec(size=W, param_name="")
        spec = ModelSpec(vocab_size=V, hidden_size=W, order=(0,), final_norm=norm, embedding_name="embed", final_norm_name="final.norm",
                         head_name=None, residual_dtype="float32", embedding_scale=20.0, blocks=(BlockSpec(
                             kind="branchnorm", name="l0.", mixer_name="mix.", input_norm_name="norm1", input_norm=norm,
                             mixer=SigmoidAttentionSpec(hidden_size=W, num_heads=H, num_kv_heads=G, qk_dim=D, v_dim=VD, score_scale=0.5, **extra)),))
        m = Model(spec, torch.float32)
        raw = random_tensors(m.expected_tensors(), 9)
        m.load({k: _dev(v.float()) for k, v in raw.items()}, torch.device("cuda"))
        cache = CacheManager(page_size=16)
        m.bind_cache(cache)
        cache.allocate(8, 2, device=torch.device("cuda"), dtype=torch.float32)
        toks = [(7 * i + 3) % V for i in range(40)]
        runner = ModelRunner(m, cache, torch.device("cuda"))
        got = torch.cat([runner.step([StepEntry("r", toks[:33], list(range(33)))])] + [runner.step([StepEntry("r", [t], [0])]) for t in toks[33:]])
        p = {k: v.double() for k, v in raw.items()}
        x = p["embed"][torch.tensor(toks)] * 20.0
        q, k = (x @ p["l0.mix." + n].T for n in ("q", "k"))
        if "joint_norm_eps" in extra:
            q, k = (plain.rms(t, p[f"l0.mix.{n}.norm"], 1e-5) for t, n in ((q, "q"), (k, "k")))
        v = (x @ p["l0.mix.v"].T).view(40, G, VD).repeat_interleave(H // G, dim=1)
        talk = p.get("l0.mix.talk", torch.eye(H, dtype=torch.float64))
        w = plain.sigmoid_weights(plain.talking_scores(q.view(40, H, D), k.view(40, G, D), 0.5, talk), p.get("l0.mix.pb", torch.zeros(H, dtype=torch.float64)))
        o = torch.einsum("hij,jhd->ihd", w, v).reshape(40, -1)
        if "output_gate" in extra:
            o = o * torch.sigmoid(x @ p["l0.mix.g"].T)
        x = x + plain.rms(o @ p["l0.mix.o"].T, p["l0.norm1"], 1e-6)
        assert_logits(got, plain.rms(x, p["final.norm"], 1e-6) @ p["embed"].T, "float32", str(extra))


def test_the_stream_behind_every_layer(folders):
    """The residual stream after each layer, taken from the engine's blocks, against the plain implementation's."""
    for name in ("A", "C"):
        cfg, tensors = read_folder(folders[name])
        toks = tokens_for(cfg, 50, 3)
        ref = []
        plain.forward(cfg, tensors, toks, layers_out=ref)
        for dtype, tol in (("float32", 2e-5), ("bfloat16", 5e-2)):
            from openinfer_b200.engine.runner import StepEntry
            runner = runner_for(folders[name], dtype, graphs=False)
            runner.stream_probe = []
            runner.step([StepEntry("r", toks, [0])])
            assert len(runner.stream_probe) == len(ref)
            for i, (a, b) in enumerate(zip(runner.stream_probe, ref)):
                err = (a.double().cpu() - b).abs().max().item() / b.pow(2).mean().sqrt().item()
                assert err < tol * (i + 1), f"{name} {dtype}: layer {i}: {err:.2e}"


# ---------------------------------------------------------------------------------------------- whole models, every cutting
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_whole_prompts_and_decoding_match_plain(folders, name, dtype):
    cfg = CASES[name][0]
    requests = {f"r{n}": tokens_for(cfg, n, n) for n in (1, 2, 17, 64, 131)}
    runner = runner_for(folders[name], dtype, max_tokens=256)
    check_trace(runner, folders[name], requests, trace_whole(requests), dtype, name)
    check_trace(runner, folders[name], requests, trace_tail(requests, tail=24), dtype, name + "/decoded")
    runner.cuda_graph = False
    check_trace(runner, folders[name], requests, trace_tail(requests, tail=5), dtype, name + "/decoded, not recorded")
    assert runner.cache.slot_pool.used_count == 0


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_prefill_equals_token_by_token(folders, name):
    """From the very first token: every position once out of one prompt, once decoded alone."""
    cfg = CASES[name][0]
    toks = tokens_for(cfg, 90, 8)
    for dtype in DTYPES:
        runner = runner_for(folders[name], dtype, max_tokens=128)
        whole = replay_in_process(runner, trace_whole({"r": toks}))["r"]
        single = replay_in_process(runner, trace_tail({"r": toks}, tail=89))["r"]
        compare(single, folders[name], toks, dtype, f"{name}: token by token")
        assert_logits(single, whole, dtype, f"{name}: token by token against the prompt", noise=2 * float32_noise(folders[name], toks),
                      noise16=bfloat16_noise(folders[name], toks))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_down_to_two_tokens(folders, name, dtype):
    cfg = CASES[name][0]
    requests = {"a": tokens_for(cfg, 150, 1), "b": tokens_for(cfg, 61, 2)}
    runner = runner_for(folders[name], dtype, max_tokens=256)
    for sizes in ((2,), (2, 3, 2, 5), (7, 2, 13, 1, 2, 31, 3, 64, 2, 17), (16,), (33, 1)):
        check_trace(runner, folders[name], requests, trace_portions(requests, sizes=sizes), dtype, f"{name}/portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("A", 16), ("B", 8), ("C", 16), ("C", 32), ("D", 32), ("E", 16), ("F", 16)])
def test_mixed_batches_with_pages_and_slots_used_again(folders, name, page, dtype):
    """Unequal requests side by side, portions beside single tokens, in a pool that holds less than their sum: each matches
    what it gives alone (the oracle), although pages and slots go from one to the next."""
    cfg = CASES[name][0]
    requests = {f"m{i}": tokens_for(cfg, n, 50 + i) for i, n in enumerate([90, 3, 150, 44, 1, 70, 121, 64])}
    max_tokens = 384
    runner = runner_for(folders[name], dtype, max_tokens=max_tokens, max_requests=3, page_size=page)
    handed = count_page_handouts(runner.cache)
    steps = trace_mixed(requests, max_tokens, seed=3, max_live=3, tail=20)
    check_trace(runner, folders[name], requests, steps, dtype, f"{name}/mixed")
    if runner.cache.groups:
        assert max(handed.values()) >= 2, "no page was used a second time"


def test_a_slot_used_again_starts_from_zero(folders):
    """The same request twice through the one state slot, with another request's state left there in between."""
    name = "E"
    cfg = CASES[name][0]
    runner = runner_for(folders[name], "float32", max_requests=1)
    for seed in (1, 2, 1):
        toks = tokens_for(cfg, 50, seed)
        check_trace(runner, folders[name], {"r": toks}, trace_tail({"r": toks}, tail=10), "float32", f"slot/{seed}")


# ---------------------------------------------------------------------------------------------- single keys that decide
def _sharp_model(tmp_path, name, heads, dim, rot=None, seed=11):
    """One attention layer in which single keys decide rows: scores that spread over tens beside a bias of -12, so that a
    row's weights are close to one for the few keys that match and vanish for all others."""
    cfg = _one_layer(attn(heads[0], heads[1], dim, 4.5 / dim ** 0.5, rot=rot))
    path = make_folder(str(tmp_path / name), cfg, seed)
    tensors = dict(read_folder(path)[1])
    tensors["l0.mix.pb"] = torch.full_like(tensors["l0.mix.pb"], -12.0)
    save(path, tensors)
    return cfg, path


@pytest.mark.parametrize("heads,dim,rot", [((4, 2), 16, (4, 10000.0)), ((9, 3), 64, (8, 10000.0)), ((4, 1), 32, None)])
def test_far_keys_first_tokens_and_keys_at_borders(tmp_path, heads, dim, rot):
    """A row's result rests on the few keys that match it, wherever they are among 400: in prompts, in portions and decoded.
    The comparison is sharp: the plain implementation with one key taken away, the first, the ones at the edges of pages and of
    the kernels' key tiles, the row's own or the one in front of it, differs by far more than the engine does."""
    cfg, path = _sharp_model(tmp_path, "sharp", heads, dim, rot)
    raw, tensors = read_folder(path)
    T = 400
    toks = tokens_for(cfg, T, 5)
    ref = oracle(path, toks)
    size = ref.pow(2).mean().sqrt().item()
    runner = runner_for(path, "float32", max_tokens=512)
    got = replay_in_process(runner, trace_tail({"f": toks}, tail=60))["f"].double()
    err = (got - ref).abs().max().item() / size
    assert err < 3e-5
    causal = torch.ones((T, T), dtype=torch.bool).tril()

    def lost(change, rows):
        seen = causal.clone()
        change(seen)
        return (plain.forward(raw, tensors, toks, seen=seen)[rows] - ref[rows]).abs().max().item() / size

    everywhere, decoded = slice(0, 340), slice(340, T)
    for key in (0, 1, 15, 16, 17, 31, 32, 63, 64, 127, 128, 255, 256):
        for rows in (slice(key + 1, 340), decoded):
            assert lost(lambda s: s[key + 1:, key].fill_(False), rows) > 30 * err, f"a lost key {key} would not be noticed"
    for rows in (everywhere, decoded):
        assert lost(lambda s: s.fill_diagonal_(False), rows) > 100 * err
        assert lost(lambda s: s.logical_and_(torch.ones_like(s).triu(-200)), rows) > 100 * err or rows is everywhere
    for row in (0, 1, 2):
        assert lost(lambda s: s[row, 0].fill_(False), slice(row, row + 1)) > 30 * err
    for dtype in DTYPES:
        runner = runner_for(path, dtype, max_tokens=512)
        check_trace(runner, path, {"f": toks}, trace_portions({"f": toks}, sizes=(15, 1, 16, 17, 2, 31, 1, 64, 3)), dtype, "sharp/portions")
        check_trace(runner, path, {"f": toks}, trace_whole({"f": toks}), dtype, "sharp/whole")
        check_trace(runner, path, {"f": toks}, trace_tail({"f": toks}, tail=40), dtype, "sharp/decoded")


def test_old_state_is_carried(tmp_path):
    """Gates that hardly open keep a sequence's first token in the state over hundreds of rows: another first token shows in
    the decoded rows by far more than the engine's error."""
    cfg = _one_layer(gru(48))
    path = make_folder(str(tmp_path / "old"), cfg, 12)
    raw, tensors = read_folder(path)
    tensors = dict(tensors)
    tensors["l0.mix.z"] = tensors["l0.mix.z"] * 0.2
    tensors["l0.mix.z.b"] = tensors["l0.mix.z.b"] * 0 - 6.0
    save(path, tensors)
    toks = tokens_for(cfg, 400, 6)
    runner = runner_for(path, "float32", max_tokens=512)
    got = replay_in_process(runner, trace_tail({"f": toks}, tail=100))["f"].double()
    ref = plain.forward(raw, tensors, toks)
    size = ref.pow(2).mean().sqrt().item()
    err = (got - ref).abs().max().item() / size
    other = plain.forward(raw, tensors, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert err < 3e-5 and (ref[300:] - other[300:]).abs().max().item() / size > 30 * err


def test_long_decoding(folders):
    """600 single-token steps behind a short prompt."""
    for name, dtype in (("D", "float32"), ("C", "bfloat16")):
        cfg = CASES[name][0]
        toks = tokens_for(cfg, 620, 77)
        runner = runner_for(folders[name], dtype, max_tokens=704)
        got = replay_in_process(runner, trace_tail({"l": toks}, tail=600))["l"]
        compare(got, folders[name], toks, dtype, "long decoding")


def test_a_long_prompt_whose_tiles_are_cut_into_slices(tmp_path):
    """1,100 tokens in one step and the rest behind it, on the tensor-core kernels: tiles whose keys are cut into slices."""
    cfg = model(83, 64, [attn(16, 4, 32, 0.35, rot=(32, 10000.0)), attn(6, 3, 64, 0.25, rot=(16, 100.0))], scale=20.0)
    path = make_folder(str(tmp_path / "long"), cfg, 2)
    toks = tokens_for(cfg, 1150, 4)
    runner = runner_for(path, "bfloat16", max_tokens=1216)
    check_trace(runner, path, {"p": toks}, trace_tail({"p": toks}, tail=50), "bfloat16", "long prompt")


# ---------------------------------------------------------------------------------------------- through the front doors
@pytest.mark.parametrize("name", ["A", "E"])
def test_greedy_generation_through_the_scheduler(folders, name):
    from openinfer_b200 import LLM, SamplingParams
    cfg, tensors = read_folder(folders[name])
    prompts = [tokens_for(cfg, n, 70 + n) for n in (1, 9, 33, 70)]
    n_new = 20

    def greedy(prompt):
        toks = list(prompt)
        for _ in range(n_new):
            toks.append(int(plain.forward(cfg, tensors, toks)[-1].argmax()))
        return toks[len(prompt):]

    want = [greedy(p) for p in prompts]
    llm = LLM(folders[name], dtype="float32", max_cache_tokens=512, max_prefill_tokens=13, max_decode_batch=3)
    assert llm.generate(prompts, max_tokens=n_new) == want
    assert llm.runner.cache.min_free_pages() == llm.runner.cache.num_pages
    assert [llm.generate([p], max_tokens=n_new)[0] for p in prompts] == want
    llm16 = LLM(folders[name], dtype="bfloat16", max_cache_tokens=512, max_decode_batch=4)
    sp = SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=5)
    a = llm16.generate(prompts, sp, max_tokens=12)
    assert a == llm16.generate(prompts, sp, max_tokens=12) and all(len(t) == 12 for t in a)
    assert llm16.runner.cache.slot_pool.used_count == 0


def test_batch_invariant_mode_is_bitwise(folders):
    """In batch-invariant mode a request's bfloat16 logits are the same bit for bit alone and among others."""
    from openinfer_b200.engine.runner import StepEntry
    from openinfer_b200.kernels import policy
    cfg = CASES["F"][0]
    reqs = {f"b{i}": tokens_for(cfg, n, 90 + i) for i, n in enumerate([40, 65, 1, 33])}
    policy.set_batch_invariant(True)
    try:
        def run(ids):
            runner = runner_for(folders["F"], "bfloat16", max_tokens=512)
            rows = {r: [] for r in ids}
            for part in (slice(0, 20), slice(20, 33)):
                entries = [StepEntry(r, reqs[r][part], list(range(len(reqs[r][part])))) for r in ids if reqs[r][part]]
                out, at = runner.step(entries), 0
                for e in entries:
                    rows[e.request_id].append(out[at: at + len(e.tokens)].clone())
                    at += len(e.tokens)
            for i in range(33, 40):
                entries = [StepEntry(r, [reqs[r][i]], [0]) for r in ids if len(reqs[r]) > i]
                if entries:
                    out = runner.step(entries)
                    for j, e in enumerate(entries):
                        rows[e.request_id].append(out[j: j + 1].clone())
            return {r: torch.cat(v) for r, v in rows.items()}

        together = run(list(reqs))
        for r in reqs:
            assert torch.equal(run([r])[r], together[r]), r
    finally:
        policy.set_batch_invariant(False)


def test_command_line_and_trace_program(folders, tmp_path):
    name = "B"
    cfg, tensors = read_folder(folders[name])
    toks = [7, 8, 9]
    want = []
    for _ in range(5):
        want.append(int(plain.forward(cfg, tensors, toks + want)[-1].argmax()))
    out = subprocess.run([sys.executable, "-m", "openinfer_b200", "--model-path", folders[name], "--dtype", "float32",
                          "--prompt-ids", "7,8,9", "--max-tokens", "5", "--num-pages", "32"],
                         cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    line = json.loads(out.stdout.strip().splitlines()[-1])
    assert line["token_ids"] == want and line["finish_reason"] == "length"
    name = "A"
    cfg = CASES[name][0]
    requests = {f"t{i}": tokens_for(cfg, n, 30 + i) for i, n in enumerate([80, 5, 130, 41, 1])}
    max_tokens = round64(130) + round64(80) + 64
    steps = trace_mixed(requests, max_tokens, seed=1, max_live=4, tail=16)
    for dtype in DTYPES:
        got = replay_trace_run(folders[name], dtype, steps, str(tmp_path / dtype), max_tokens, cfg["vocab"])
        for rid, t in requests.items():
            compare(got[rid], folders[name], t, dtype, f"trace_run/{dtype}/{rid}")
