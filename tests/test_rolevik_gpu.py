"""Rolevik in the engine against the plain implementation: the design's kernels alone, every mechanism alone in a model of one
layer, the stream behind every layer, whole prompts, decoding through cache and state, portions, mixed batches, pages and slots
that are used again, keys just inside and outside of chunks and at page and tile borders, first tokens, old state, long decoding,
greedy generation through the scheduler, the command line and the trace program."""
import json
import random
import subprocess
import sys
import types

import pytest
import torch

import plain_rolevik as plain
from rolevik_cases import (CASES, SETTLED, SPREAD, assert_logits, attn, bfloat16_noise, delta, dense, first_close_call, float32_noise, lru, make_folder,
                           model, moe, oracle, par, read_folder, tokens_for)
from helpers import (ROOT, count_page_handouts, replay_in_process, replay_trace_run, round64, trace_mixed, trace_portions,
                     trace_tail, trace_whole)

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """Model folders by (case, dtype): routers whose choice the scores decide for 32-bit, settled ones for 16 bits."""
    return {(n, d): make_folder(str(tmp_path_factory.mktemp(f"rol{n}{d}")), cfg, seed, SPREAD if d == "float32" else SETTLED)
            for n, (cfg, seed) in CASES.items() for d in DTYPES}


def runner_for(path, dtype, max_tokens=2048, max_requests=4, page_size=16, graphs=True):
    from openinfer_b200.engine.runner import ModelRunner
    r = ModelRunner.from_folder(path, dtype=dtype, max_tokens=max_tokens, max_requests=max_requests, page_size=page_size)
    r.cuda_graph = graphs
    return r


def compare(got, path, toks, dtype, what):
    assert_logits(got, oracle(path, toks), dtype, what, noise=float32_noise(path, toks), noise16=bfloat16_noise(path, toks),
                  first_close=first_close_call(path, toks))


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


def _step(lens, slots, phases=None, padding=False):
    """The metadata of a step whose requests bring ``lens`` rows; with ``padding`` a last request that is nobody's."""
    all_lens = list(lens) + ([1] if padding else [])
    starts = [0]
    for n in all_lens:
        starts.append(starts[-1] + n)
    return types.SimpleNamespace(
        cu_seqlens=_i32(starts), token_req=_i32([b for b, n in enumerate(lens) for _ in range(n)] + ([-1] if padding else [])),
        state_slots=_i32(slots), state_phase=_i32(phases or [0] * len(all_lens)), num_requests=len(all_lens), decode_only=max(lens) == 1,
        q_lens_host=all_lens), starts


# ---------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,hd,qk,rot_half,bias,page", [(4, 2, 16, 16, 4, True, 16), (3, 1, 16, 10, 3, True, 4), (5, 5, 40, 40, 0, False, 8),
                                                             (9, 3, 64, 64, 32, True, 16), (1, 1, 8, 6, 1, True, 2), (20, 5, 128, 128, 16, True, 16),
                                                             (64, 8, 128, 128, 64, True, 16), (2, 1, 24, 24, 8, False, 16), (3, 3, 56, 50, 15, True, 16)])
def test_joint_norm_of_halves_kernel(dtype, nq, nkv, hd, qk, rot_half, bias, page):
    """Bias, q and k normed over all heads together, pairs (d, d + half) turned; q in place, k and v to their page; a padding
    row stores nothing."""
    from openinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(nq * 100 + hd)
    T, pages, td = 7, 9, TORCH[dtype]
    cols = (nq + 2 * nkv) * hd
    head = (torch.arange(hd) < qk).float().repeat(nq + 2 * nkv)
    proj = torch.zeros(T, cols + 8)
    proj[:, :cols] = torch.randn(T, cols, generator=g) * 2 * head
    proj = proj.to(td)
    b = torch.randn(cols, generator=g) * head if bias else torch.zeros(cols)
    qw, kw = ((1 + 0.2 * torch.randn(h * hd, generator=g)) * head[: h * hd] for h in (nq, nkv))
    pos, slots = [0, 3, 11, 12, 4, 30, 31], [1, 0, 2 * page + 1, -1, 8 * page + page - 1, 3 * page, 4 * page]
    base, n = 77.0, torch.arange(max(rot_half, 1), dtype=torch.float64)
    ang = torch.arange(32, dtype=torch.float64)[:, None] * base ** (-2.0 * n / max(2 * rot_half, 1))[None, :]
    cos, sin = (_dev(f(ang).float().contiguous()) if rot_half else None for f in (torch.cos, torch.sin))
    kc, vc = (torch.full((pages, page, nkv, hd), 9.0, dtype=td, device="cuda") for _ in range(2))
    x = _dev(proj.clone())
    ops.joint_norm_half_store(x, nq, nkv, hd, qk, bias=_dev(b) if bias else None, q_norm_w=_dev(qw), k_norm_w=_dev(kw), eps=1e-3, cos=cos,
                              sin=sin, positions=_i32(pos), slots=_i32(slots), k_cache=kc, v_cache=vc, page_stride=kc.stride(0), page_size=page)
    p64 = proj[:, :cols].double() + b.double()

    def ready(at, heads, w):
        z = p64[:, at: at + heads * hd].view(T, heads, hd)[..., :qk].reshape(T, -1)
        z = plain.rms(z, w.double().view(heads, hd)[:, :qk].reshape(-1), 1e-3).view(T, heads, qk)
        return plain.turn_halves(z, torch.tensor(pos), base, 2 * rot_half) if rot_half else z

    tol = 2e-6 if dtype == "float32" else 1e-2
    rq, rk = ready(0, nq, qw), ready(nq * hd, nkv, kw)
    rv = p64[:, (nq + nkv) * hd: cols].view(T, nkv, hd)
    gq = x[:, : nq * hd].double().cpu().view(T, nq, hd)
    assert (gq[..., :qk] - rq).abs().max().item() < tol * max(1.0, rq.abs().max().item()) and (gq[..., qk:] == 0).all()
    written = torch.zeros(pages, page, dtype=torch.bool)
    for t, s in enumerate(slots):
        if s < 0:
            continue
        written[s // page, s % page] = True
        assert (kc[s // page, s % page, :, :qk].double().cpu() - rk[t]).abs().max().item() < tol * max(1.0, rk.abs().max().item())
        assert (vc[s // page, s % page].double().cpu() - rv[t]).abs().max().item() < tol * max(1.0, rv.abs().max().item())
        assert (kc[s // page, s % page, :, qk:] == 0).all()
    assert (kc.cpu()[~written] == 9.0).all() and (vc.cpu()[~written] == 9.0).all()


def _paged_case(nq, nkv, hd, q_lens, kv_lens, page, td, seed):
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
    q = torch.randn(T, nq * hd, generator=g).to(td)
    starts = [0]
    for n in q_lens:
        starts.append(starts[-1] + n)
    ctx = types.SimpleNamespace(
        num_tokens=T, num_requests=B, cache=types.SimpleNamespace(page_size=page), scratch={}, q_lens_host=list(q_lens), kv_lens_host=list(kv_lens),
        token_req=_i32([b for b, n in enumerate(q_lens) for _ in range(n)]),
        positions=_i32([p for n, k in zip(q_lens, kv_lens) for p in range(k - n, k)]), cu_seqlens=_i32(starts))
    return q, kc, vc, table, starts, ctx, types.SimpleNamespace(block_table=_dev(table), kv_lens=_i32(kv_lens))


@pytest.mark.parametrize("chunk", [1, 5, 16, 64, 65, 100, 1000])
@pytest.mark.parametrize("nq,nkv,hd", [(4, 2, 128), (6, 2, 64), (3, 3, 32), (8, 1, 128), (5, 1, 40)])
def test_attention_kernels_under_chunks(nq, nkv, hd, chunk):
    """The tcgen05 tiles, the mma.sync tiles, the decode kernel and the general kernel, on shuffled pages: portions that begin and
    end inside chunks, behind cached keys, beside single tokens. What lies outside of a row's chunk is poisoned."""
    from openinfer_b200.kernels import attention as A
    scale = 3.0 * hd ** -0.5
    for td, tcgen in ((torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)):
        for page, q_lens, kv_lens in ((16, [1], [1]), (16, [5, 1], [37, 513]), (16, [1, 40, 1, 3], [16, 300, 66, 3]), (32, [150], [230])):
            q, kc, vc, table, starts, ctx, group = _paged_case(nq, nkv, hd, q_lens, kv_lens, page, td, nq + hd + page + chunk)
            refs, oldest = [], {}
            for b, (n, kv) in enumerate(zip(q_lens, kv_lens)):
                pages = table[b, : -(-kv // page)].long()
                k, v = (c[pages].reshape(-1, nkv, hd)[:kv].double() for c in (kc, vc))
                qq = torch.zeros(kv, nq, hd, dtype=torch.float64)
                qq[kv - n:] = q[starts[b]: starts[b] + n].double().view(n, nq, hd)
                refs.append(plain.softmax_attention(qq, k, v, scale, plain.chunk_mask(kv, chunk))[kv - n:])
                first = (kv - n) - (kv - n) % chunk           # keys in front of the first row's chunk: nobody may see them
                for pos in range(0, first):
                    kc[table[b, pos // page].long(), pos % page] = 60.0
                    vc[table[b, pos // page].long(), pos % page] = 1e4
            d = [_dev(t) for t in (q, kc, vc)]
            out = torch.zeros(sum(q_lens), nq * hd, dtype=td, device="cuda")
            old, A.USE_TCGEN05 = A.USE_TCGEN05, tcgen
            try:
                step = A.attention_step(ctx, group, d[0], out, d[1], d[1].stride(0), nq, nkv, hd, -chunk)
                layer = A.attention_layer(d[0], out, d[1], d[2], nq, nkv, hd, scale, -chunk, write_kv=False, rope_mode=0)
                A.run_attention(step, layer)
            finally:
                A.USE_TCGEN05 = old
            assert bool(step.tensor_core) == (td == torch.bfloat16 and hd in (32, 64, 128))
            for b, ref in enumerate(refs):
                err = (out[starts[b]: starts[b + 1]].double().cpu() - ref).abs().max().item()
                assert err < (2e-5 if td == torch.float32 else 3e-2), f"{td} tcgen05 {tcgen} page {page} request {b}: {err}"


@pytest.mark.parametrize("H,G,D,V", [(4, 2, 16, 24), (3, 1, 7, 5), (2, 2, 64, 40), (1, 1, 20, 3), (4, 1, 128, 64), (2, 1, 200, 8), (1, 1, 300, 16), (5, 5, 32, 17), (20, 5, 96, 128), (24, 24, 48, 130)])
def test_delta_rule_with_a_decay_per_head_kernel(H, G, D, V):
    """Portions over old state beside single tokens and a padding request: runs of four rows, what is left over, both copies of
    the state; strong and weak decays, queries and keys of any length."""
    from openinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(H * 1000 + D)
    for lens in ([7, 1, 130], [4, 2, 3], [1, 1], [65]):
        B = len(lens) + 1
        slots, phases = list(range(B, 0, -1)), [b % 2 for b in range(B)]
        ctx, starts = _step(lens, slots, phases, padding=True)
        T, cols = starts[-1], 2 * G * D + H * V
        qkv = torch.randn(T, cols + 4, generator=g)
        gates = torch.randn(T, 2 * H + 3, generator=g) * 2
        dt, A = torch.randn(H, generator=g) - 1.0, torch.randn(H, generator=g)
        state = torch.randn(B + 1, 2, H, D * V, generator=g)
        s_dev, out = _dev(state.clone()), torch.zeros(T, H * V, device="cuda")
        ops.recurrent_scan(ops.SCAN_DELTA_HEAD_DECAY, out, _dev(qkv), (0, G * D, 2 * G * D), _dev(gates), (1, H + 2), s_dev, ctx, H, G, D, V,
                           p0=_dev(dt), p1=_dev(A), q_scale=D ** -0.5)
        for b, n in enumerate(lens):
            x, z = qkv[starts[b]: starts[b] + n].double(), gates[starts[b]: starts[b] + n].double()
            q = (plain.unit(x[:, : G * D].view(n, G, D)) * D ** -0.5).repeat_interleave(H // G, dim=1)
            k = plain.unit(x[:, G * D: 2 * G * D].view(n, G, D)).repeat_interleave(H // G, dim=1)
            v = x[:, 2 * G * D: cols].view(n, H, V)
            decay = torch.exp(-torch.exp(A.double()) * plain.softplus(z[:, H + 2: 2 * H + 2] + dt.double()))
            S0 = state[slots[b], phases[b]].double().view(H, V, D).transpose(1, 2)
            ref = plain.delta_rule(q, k, v, torch.sigmoid(z[:, 1: H + 1]), decay, S=S0)
            tail = plain.delta_rule(torch.eye(D, dtype=torch.float64)[:, None].repeat(1, H, 1), k.new_zeros(D, H, D), k.new_zeros(D, H, V),
                                    k.new_zeros(D, H), k.new_ones(D, H), S=_last_state(q, k, v, z, decay, S0, H))
            err = (out[starts[b]: starts[b] + n].double().cpu().view(n, H, V) - ref).abs().max().item()
            assert err < 1e-5 * max(1.0, ref.abs().max().item()), (lens, b, err)
            got = s_dev[slots[b], 1 - phases[b]].double().cpu().view(H, V, D).permute(2, 0, 1)
            assert (got - tail).abs().max().item() < 1e-5 * max(1.0, tail.abs().max().item())
            assert torch.equal(s_dev[slots[b], phases[b]].cpu(), state[slots[b], phases[b]])
        assert torch.equal(s_dev[0].cpu(), state[0]) and torch.equal(s_dev[slots[-1]].cpu(), state[slots[-1]])


def _last_state(q, k, v, z, decay, S, H):
    for t in range(k.shape[0]):
        S = decay[t][:, None, None] * S
        u = torch.sigmoid(z[t, 1: H + 1])[:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
    return S


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("blocks,size", [(1, 1), (3, 11), (4, 16), (2, 64), (5, 40), (1, 200), (2, 72)])
def test_recurrent_unit_kernels(blocks, size, dtype):
    """The gates, the coefficients and the scan over old state: portions, single tokens, a padding request."""
    from openinfer_b200.kernels import ops
    C, td = blocks * size, TORCH[dtype]
    g = torch.Generator().manual_seed(C)
    w = (torch.randn(2, blocks, size, size, generator=g) * size ** -0.5).to(td)
    bias, y_bias = torch.randn(2, C, generator=g), torch.randn(C, generator=g)
    lam = torch.randn(C, generator=g) * 2 - 3.0
    rate = 8.0 * plain.softplus(lam.double())
    for lens in ([7, 1, 256, 130], [1, 70], [1, 1, 1], [2, 515, 5]):
        B = len(lens) + 1
        slots = list(range(B, 0, -1))
        ctx, starts = _step(lens, slots, padding=True)
        T = starts[-1]
        step = -(-C // 8) * 8
        u, y = torch.randn(T, step, generator=g), torch.randn(T, step + 8, generator=g)
        state = torch.randn(B + 1, C, generator=g)
        s_dev, out = _dev(state.clone()), torch.zeros(T, C, dtype=td, device="cuda")
        ops.rglru_scan(out, _dev(u)[:, :C], _dev(w), _dev(bias), _dev(rate.float()), _dev(y), _dev(y_bias), s_dev, ctx)
        for b, n in enumerate(lens):
            uu = u[starts[b]: starts[b] + n, :C].double()
            r, i = (plain.block_gates(uu, w[k].double(), bias[k].double().view(blocks, size)) for k in (0, 1))
            S = plain.rglru_states(uu, r, i, lam.double(), S=state[slots[b]].double())
            ref = S * plain.gelu_tanh(y[starts[b]: starts[b] + n, :C].double() + y_bias.double())
            # 16-bit matrices meet u as two bfloat16 halves: 16 bits of it; the results are rounded to their type
            err = (s_dev[slots[b]].double().cpu() - S[-1]).abs().max().item()
            assert err < (4e-6 if dtype == "float32" else 4e-5) * max(1.0, S.abs().max().item()), (lens, b, err)
            err = (out[starts[b]: starts[b] + n].double().cpu() - ref).abs().max().item()
            assert err < (4e-6 if dtype == "float32" else 6e-3) * max(1.0, ref.abs().max().item()), (lens, b, err)
        assert torch.equal(s_dev[0].cpu(), state[0]) and torch.equal(s_dev[slots[-1]].cpu(), state[slots[-1]])


def test_a_unit_that_hardly_forgets():
    """a close to one: sqrt(1 - a^2) formed from the logarithm keeps its digits (1 - a^2 in float32 would lose them)."""
    from openinfer_b200.kernels import ops
    C = 64
    g = torch.Generator().manual_seed(3)
    ctx, _ = _step([50], [0])
    lam = torch.full((C,), -13.0)
    rate = 8.0 * plain.softplus(lam.double())
    u, w, zero = torch.randn(50, C, generator=g), torch.zeros(2, 1, C, C), torch.zeros(C)
    s, out = torch.zeros(1, C, device="cuda"), torch.zeros(50, C, device="cuda")
    ops.rglru_scan(out, _dev(u), _dev(w), torch.zeros(2, C, device="cuda"), _dev(rate.float()), torch.ones(50, C, device="cuda"), _dev(zero), s, ctx)
    half = torch.full((50, C), 0.5, dtype=torch.float64)
    S = plain.rglru_states(u.double(), half, half, lam.double())
    assert ((s.double().cpu()[0] - S[-1]).abs().max() / S.abs().max()).item() < 2e-6
    a = torch.exp(-0.5 * rate.float())
    assert ((torch.sqrt(1.0 - a * a) - torch.sqrt(-torch.expm1(-rate)).float()).abs() / torch.sqrt(-torch.expm1(-rate)).float()).max() > 1e-3


@pytest.mark.parametrize("taps", [1, 2, 4, 5, 9])
@pytest.mark.parametrize("channels", [6, 40])
def test_filter_with_biases(taps, channels):
    """The bias in front of the filter enters the state with the inputs, and not what lies before a sequence's start."""
    from openinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(taps)
    x, w = torch.randn(30, channels, generator=g), torch.randn(channels, taps, generator=g)
    ib, ob = torch.randn(channels, generator=g), torch.randn(channels, generator=g)
    ref = plain.causal_filter(x + ib, w, ob)
    for sizes in ([30], [1] * 30, [2, 3, 25], [7, 1, 1, 21]):
        state = torch.zeros(2, 2, max(1, taps - 1), channels, device="cuda") if taps > 1 else None
        at, got = 0, []
        for k, n in enumerate(sizes):
            ctx, _ = _step([n], [1], [k % 2])
            out = torch.empty(n, channels, device="cuda")
            ops.short_conv_act(out, _dev(x[at: at + n].contiguous()), _dev(w), state, ctx.cu_seqlens, ctx.token_req, ctx.state_slots,
                               ctx.state_phase, in_bias=_dev(ib), out_bias=_dev(ob))
            got.append(out.cpu())
            at += n
        assert (torch.cat(got) - ref).abs().max().item() < 1e-5


@pytest.mark.parametrize("width", [1, 37, 64, 320, 1024, 2048, 4100, 8192])
def test_joining_a_branch_kernel(width):
    """Layer and rms norms on a branch, on the sum of a normed pair, and that sum alone; the stream's bfloat16 copy."""
    from openinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(width)
    a, b, h = (torch.randn(5, width, generator=g) * s + m for s, m in ((3.0, 40.0), (0.02, 0.0), (1.0, 0.0)))
    wa, wb, w = (1 + 0.3 * torch.randn(width, generator=g) for _ in range(3))
    pair = ops.NormedPair(_dev(a), _dev(b), _dev(wa), _dev(wb), 0.5, 0.25, 1e-4)
    summed = 0.5 * plain.rms(a.double(), wa.double(), 1e-4) + 0.25 * plain.rms(b.double(), wb.double(), 1e-4)
    for branch, v in ((_dev(a), a.double()), (pair, summed)):
        for center in (True, False):
            for low in (None, torch.zeros(5, width, dtype=torch.bfloat16, device="cuda")):
                hd = _dev(h.clone())
                ops.branch_join(hd, branch, weight=_dev(w), center=center, eps=1e-5, low=low)
                ref = h.double() + (plain.layer_norm if center else plain.rms)(v, w.double(), 1e-5)
                assert (hd.double().cpu() - ref).abs().max().item() < 2e-5 * max(1.0, ref.abs().max().item())
                assert low is None or torch.equal(low, hd.bfloat16())
    out = ops.branch_join(None, pair, out=torch.empty(5, width, device="cuda"))
    assert (out.double().cpu() - summed).abs().max().item() < 1e-5 * max(1.0, summed.abs().max().item())
    x = torch.empty(2, width, device="cuda")
    ops.rmsnorm_cast(x, _dev(a), _dev(w), 1e-5, row_idx=_i32([3, 0]), center=True)
    assert (x.double().cpu() - plain.layer_norm(a.double(), w.double(), 1e-5)[[3, 0]]).abs().max().item() < 2e-5 * max(1.0, width ** 0.5)


@pytest.mark.parametrize("rows", [1, 9, 200])
@pytest.mark.parametrize("experts,identity,top,groups,keep", [(8, 0, 3, 1, 1), (6, 2, 3, 2, 1), (5, 3, 8, 4, 4), (12, 4, 2, 8, 1), (40, 8, 6, 6, 3), (3, 3, 2, 3, 1)])
def test_router_with_softmax_scores_and_choices_without_an_expert(rows, experts, identity, top, groups, keep):
    """Choice, weights and the experts' sum. Choice scores are far apart and mostly negative; rows whose every choice stands for
    the input itself, and none."""
    from openinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(rows + experts + top)
    W, F, n = 48, 24, experts + identity
    if (n // groups) * keep < top:
        pytest.skip("the kept groups cannot give that many choices")
    x = torch.randn(rows, W, generator=g)
    router, corr = torch.randn(n, W, generator=g) * W ** -0.5 * 3, (torch.randperm(n, generator=g) - n) * 0.3
    wgu, wd = torch.randn(experts, 2 * F, W, generator=g) * W ** -0.5, torch.randn(experts, W, F, generator=g) * F ** -0.5
    add = torch.randn(rows, W, generator=g)
    for td in (torch.float32, torch.bfloat16):
        xx, ww, gu, dn = x.to(td), router.to(td), wgu.to(td), wd.to(td)
        z = xx.double() @ ww.double().T
        s, e = plain.choose(z, corr.double(), top, groups, keep)
        sure = plain.choice_margin(z, corr.double(), top, groups, keep) > 1e-4
        routing = ops.moe_route(_dev(xx), _dev(ww), top, scoring="softmax_groups", correction=_dev(corr), groups=groups, keep_groups=keep,
                                identity=identity, weight_scale=1.9)
        ids, wts = routing[0].cpu(), routing[1].double().cpu()
        assert sure.float().mean() > 0.8 and torch.equal(ids.sort(dim=1).values[sure], e.int().sort(dim=1).values[sure])
        assert (wts - 1.9 * s.gather(1, ids.long())).abs().max().item() < 1e-5
        out = ops.moe_experts(_dev(xx), _dev(gu), _dev(dn), routing, 0.0, act="silu", add=_dev(add)).double().cpu()
        ref = add.double()
        for t in range(rows):
            for j in range(top):
                i = int(ids[t, j])
                if i >= experts:
                    y = xx[t].double()
                else:
                    gate, up = (gu[i].double() @ xx[t].double()).chunk(2)
                    y = dn[i].double() @ (plain.silu(gate) * up)
                ref[t] += wts[t, j] * y
        assert (out - ref).abs().max().item() < (2e-5 if td == torch.float32 else 3e-2) * max(1.0, ref.abs().max().item())


# ---------------------------------------------------------------------------------------------- mechanisms alone
def _one_layer(layer, width=48, vocab=83, **kw):
    return model(vocab, width, [layer], **{"scale": 3.0, **kw})


PLAIN_DELTA = delta(2, 1, 8, 12, 3)
PLAIN_ATTN = attn(2, 1, 16, 16, 0.5, chunk=20, rot=(8, 100.0))
MECHANISMS = {
    "unit of one channel": _one_layer(lru(1, 1, 1)),
    "unit wider than the model": _one_layer(lru(200, 5, 4)),
    "unit with a part per channel": _one_layer(lru(24, 24, 2)),
    "unit without a filter": _one_layer(lru(40, 2, 1)),
    "unit behind a long filter": _one_layer(lru(40, 2, 9)),
    "one head, no mask, no rotation": _one_layer(par(attn(1, 1, 16, 16, 0.5), PLAIN_DELTA)),
    "chunks of one": _one_layer(par(attn(4, 1, 16, 16, 0.5, chunk=1), PLAIN_DELTA)),
    "chunks of a page": _one_layer(par(attn(4, 2, 16, 16, 0.5, chunk=16), PLAIN_DELTA)),
    "chunks longer than the sequence": _one_layer(par(attn(4, 4, 8, 24, 0.7, chunk=500), PLAIN_DELTA)),
    "rotation of the first two numbers": _one_layer(par(attn(2, 1, 16, 16, 0.5, chunk=30, rot=(2, 40.0)), PLAIN_DELTA)),
    "rotation of the whole head": _one_layer(par(attn(2, 2, 32, 8, 0.4, chunk=30, rot=(32, 10000.0)), PLAIN_DELTA)),
    "heads of 64, groups of three": _one_layer(par(attn(9, 3, 64, 64, 0.25, chunk=33, rot=(64, 10000.0)), PLAIN_DELTA)),
    "heads of 128, groups of eight": _one_layer(par(attn(16, 2, 128, 128, 0.15, chunk=48, rot=(32, 10000.0)), PLAIN_DELTA)),
    "heads of 264 numbers": _one_layer(par(attn(2, 1, 264, 40, 0.1, chunk=25, rot=(64, 10000.0)), PLAIN_DELTA)),
    "delta rule of one head": _one_layer(par(PLAIN_ATTN, delta(1, 1, 16, 16, 1))),
    "delta rule with shared keys": _one_layer(par(PLAIN_ATTN, delta(6, 2, 20, 4, 4))),
    "delta rule of 128 channels": _one_layer(par(PLAIN_ATTN, delta(2, 2, 128, 32, 4))),
    "dense feed-forward": _one_layer(lru(24, 3, 2, mlp=dense(70))),
    "experts": _one_layer(lru(24, 3, 2, mlp=moe(20, 6, 2)), vocab=60),
    "experts in groups with a shared one": _one_layer(lru(24, 3, 2, mlp=moe(20, 6, 2, groups=(3, 1), scale=2.2, shared=30))),
    "choices that stand for the input": _one_layer(lru(24, 3, 2, mlp=moe(20, 2, 2, identity=4, scale=1.5))),
    "every expert at once": _one_layer(lru(24, 3, 2, mlp=moe(20, 3, 4, identity=1))),
    "a large eps": _one_layer(par(PLAIN_ATTN, PLAIN_DELTA), eps=0.5),
    "embedding as it is, small logits": _one_layer(lru(24, 3, 2), scale=1.0, logit_scale=0.01),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MECHANISMS))
def test_each_mechanism_alone(tmp_path, name, dtype):
    """A model of one layer with one mechanism: a whole prompt, then portions of 2, 1, 5 and 3 tokens and decoding."""
    cfg = MECHANISMS[name]
    path = make_folder(str(tmp_path / "m"), cfg, 7, SPREAD if dtype == "float32" else SETTLED)
    requests = {"a": tokens_for(cfg, 75, 1), "b": tokens_for(cfg, 40, 2)}
    runner = runner_for(path, dtype, max_tokens=256)
    check_trace(runner, path, requests, trace_whole(requests), dtype, name)
    check_trace(runner, path, requests, trace_portions(requests, sizes=(2, 1, 5, 3, 30, 1, 1, 2)), dtype, name + "/portions")


def test_a_normed_pair_in_a_block_that_does_not_join_it():
    """A parallel mixer whose results are normed, inside a block that asks for one result."""
    from openinfer_b200.cache.manager import CacheManager
    from openinfer_b200.engine.runner import ModelRunner, StepEntry
    from openinfer_b200.parts.model import Model
    from openinfer_b200.parts.spec import BlockSpec, MinGruSpec, ModelSpec, NormSpec, ParallelMixerSpec, RgLruSpec
    from openinfer_b200.weights.random import random_tensors
    W, V = 40, 61
    norm = NormSpec(size=W, param_name="")
    spec = ModelSpec(vocab_size=V, hidden_size=W, order=(0,), final_norm=norm, embedding_name="embed", final_norm_name="final.norm",
                     head_name=None, residual_dtype="float32", embedding_scale=20.0, blocks=(BlockSpec(
                         kind="shared_norm", name="l0.", mixer_name="mix.", input_norm_name="norm1", input_norm=norm, mixer=ParallelMixerSpec(
                             left=RgLruSpec(hidden_size=W, channels=24, blocks=3, conv_taps=3), right=MinGruSpec(hidden_size=W, channels=10),
                             left_scale=0.3, right_scale=0.9, out_norm_eps=1e-4)),))
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
    h = plain.rms(x, p["l0.norm1"], 1e-6)
    left, q = plain.rglru(h, p, "l0.mix.left."), "l0.mix.right."
    z, u = torch.sigmoid(h @ p[q + "z"].T + p[q + "z.b"]), h @ p[q + "x"].T + p[q + "x.b"]
    S, rows = torch.zeros(10, dtype=torch.float64), []
    for t in range(40):
        S = (1 - z[t]) * S + z[t] * torch.where(u[t] >= 0, u[t] + 0.5, torch.sigmoid(u[t]))
        rows.append(S)
    right = (torch.stack(rows) * plain.silu(h @ p[q + "g"].T)) @ p[q + "o"].T
    x = x + 0.3 * plain.rms(left, p["l0.mix.left.out"], 1e-4) + 0.9 * plain.rms(right, p["l0.mix.right.out"], 1e-4)
    assert_logits(got, plain.rms(x, p["final.norm"], 1e-6) @ p["embed"].T, "float32", "normed pair")


def test_the_stream_behind_every_layer(folders):
    """The residual stream after each layer, taken from the engine's blocks, against the plain implementation's."""
    from openinfer_b200.engine.runner import StepEntry
    for name in ("A", "E", "F"):
        for dtype, tol in (("float32", 2e-5), ("bfloat16", 5e-2)):
            cfg, tensors = read_folder(folders[name, dtype])
            toks = tokens_for(cfg, 50, 3)
            ref = []
            plain.forward(cfg, tensors, toks, layers_out=ref)
            runner = runner_for(folders[name, dtype], dtype, graphs=False)
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
    runner = runner_for(folders[name, dtype], dtype, max_tokens=256)
    check_trace(runner, folders[name, dtype], requests, trace_whole(requests), dtype, name)
    check_trace(runner, folders[name, dtype], requests, trace_tail(requests, tail=24), dtype, name + "/decoded")
    runner.cuda_graph = False
    check_trace(runner, folders[name, dtype], requests, trace_tail(requests, tail=5), dtype, name + "/decoded, not recorded")
    assert runner.cache.slot_pool.used_count == 0


@pytest.mark.parametrize("name", ["B", "C", "D", "F"])
def test_prefill_equals_token_by_token(folders, name):
    """From the very first token: every position once out of one prompt, once decoded alone."""
    cfg = CASES[name][0]
    toks = tokens_for(cfg, 90, 8)
    for dtype in DTYPES:
        runner = runner_for(folders[name, dtype], dtype, max_tokens=128)
        whole = replay_in_process(runner, trace_whole({"r": toks}))["r"]
        single = replay_in_process(runner, trace_tail({"r": toks}, tail=89))["r"]
        compare(single, folders[name, dtype], toks, dtype, f"{name}: token by token")
        assert_logits(single, whole, dtype, f"{name}: token by token against the prompt", noise=2 * float32_noise(folders[name, dtype], toks),
                      noise16=bfloat16_noise(folders[name, dtype], toks), first_close=first_close_call(folders[name, dtype], toks))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_down_to_two_tokens(folders, name, dtype):
    cfg = CASES[name][0]
    requests = {"a": tokens_for(cfg, 150, 1), "b": tokens_for(cfg, 61, 2)}
    runner = runner_for(folders[name, dtype], dtype, max_tokens=256)
    for sizes in ((2,), (2, 3, 2, 5), (7, 2, 13, 1, 2, 31, 3, 64, 2, 17), (16,), (33, 1)):
        check_trace(runner, folders[name, dtype], requests, trace_portions(requests, sizes=sizes), dtype, f"{name}/portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("A", 16), ("B", 8), ("C", 16), ("C", 32), ("D", 32), ("E", 16), ("F", 16)])
def test_mixed_batches_with_pages_and_slots_used_again(folders, name, page, dtype):
    """Unequal requests side by side, portions beside single tokens, in a pool that holds less than their sum: each matches
    what it gives alone (the oracle), although pages and slots go from one to the next."""
    cfg = CASES[name][0]
    requests = {f"m{i}": tokens_for(cfg, n, 50 + i) for i, n in enumerate([90, 3, 150, 44, 1, 70, 121, 64])}
    max_tokens = 384
    runner = runner_for(folders[name, dtype], dtype, max_tokens=max_tokens, max_requests=3, page_size=page)
    handed = count_page_handouts(runner.cache)
    steps = trace_mixed(requests, max_tokens, seed=3, max_live=3, tail=20)
    check_trace(runner, folders[name, dtype], requests, steps, dtype, f"{name}/mixed")
    if runner.cache.groups:
        assert max(handed.values()) >= 2, "no page was used a second time"


def test_a_slot_used_again_starts_from_zero(folders):
    """The same request twice through the one state slot, with another request's state left there in between."""
    for name in ("E", "D"):
        cfg = CASES[name][0]
        runner = runner_for(folders[name, "float32"], "float32", max_requests=1)
        for seed in (1, 2, 1):
            toks = tokens_for(cfg, 50, seed)
            check_trace(runner, folders[name, "float32"], {"r": toks}, trace_tail({"r": toks}, tail=10), "float32", f"slot/{name}/{seed}")


# ---------------------------------------------------------------------------------------------- single keys that decide
@pytest.mark.parametrize("heads,dim,chunk,rot", [((4, 2), 16, 48, (4, 10000.0)), ((9, 3), 64, 70, (8, 10000.0)), ((2, 1), 128, 64, (32, 10000.0)),
                                                 ((4, 1), 32, 128, None)])
def test_keys_just_inside_and_outside_of_chunks(tmp_path, heads, dim, chunk, rot):
    """Scores that spread over tens: a row rests on the few keys that match it, wherever they are in its chunk. The comparison is
    sharp: the plain implementation with a key taken away (a chunk's first and last, the ones at page and tile edges, a row's
    own) or with chunks one position off differs by far more than the engine does, in prompts, in portions and decoded."""
    cfg = _one_layer(par(attn(heads[0], heads[1], dim, dim, 6.0 / dim ** 0.5, chunk=chunk, rot=rot), delta(1, 1, 4, 4, 1)))
    path = make_folder(str(tmp_path / "sharp"), cfg, 11)
    tensors = dict(read_folder(path)[1])
    tensors["l0.mix.right.out"] = tensors["l0.mix.right.out"] * 0.05          # the attention decides
    save(path, tensors)
    T = 4 * chunk + chunk // 2
    toks = tokens_for(cfg, T, 5)
    ref = oracle(path, toks)
    size = ref.pow(2).mean().sqrt().item()
    tail = chunk + chunk // 2 + 3                                             # decoding passes an edge
    runner = runner_for(path, "float32", max_tokens=1024)
    got = replay_in_process(runner, trace_tail({"f": toks}, tail=tail))["f"].double()
    err = (got - ref).abs().max().item() / size
    assert err < 3e-5
    own = plain.chunk_mask(T, chunk)

    def other(seen, rows):
        return (plain.forward(cfg, tensors, toks, seen=seen)[rows] - ref[rows]).abs().max().item() / size

    def lost(key):
        seen = own.clone()
        seen[key + 1:, key] = False
        return seen

    for key in (0, 1, 15, 16, chunk - 2, chunk, 2 * chunk, 2 * chunk + 1, 3 * chunk - 2):
        assert other(lost(key), slice(key + 1, T)) > 30 * err, f"a lost key {key} would not be noticed"
    edges = [e for e in range(chunk, T, chunk)]
    for e in edges:                                                            # in the prompt and among the decoded rows
        seen = own.clone()
        seen[e: e + 3, e - 1] = True
        assert other(seen, slice(e, e + 3)) > 100 * err, "a key of the chunk before would not be noticed"
    assert any(e >= T - tail for e in edges) and any(e < T - tail for e in edges)
    seen = own & ~torch.eye(T, dtype=torch.bool)
    seen[torch.arange(0, T, chunk), torch.arange(0, T, chunk)] = True          # (a chunk's first row has no other key)
    assert other(seen, slice(0, T)) > 100 * err
    for dtype in DTYPES:
        runner = runner_for(path, dtype, max_tokens=1024)
        check_trace(runner, path, {"f": toks}, trace_portions({"f": toks}, sizes=(15, 1, 16, 17, 2, 31, 1, 64, 3)), dtype, "sharp/portions")
        check_trace(runner, path, {"f": toks}, trace_whole({"f": toks}), dtype, "sharp/whole")
        check_trace(runner, path, {"f": toks}, trace_tail({"f": toks}, tail=tail), dtype, "sharp/decoded")


def test_far_keys_without_a_mask(tmp_path):
    """A mixer without chunks sees every key: the first key of 300 shows in the decoded rows."""
    cfg = _one_layer(par(attn(4, 2, 32, 32, 1.1, rot=(4, 10000.0)), delta(1, 1, 4, 4, 1)))
    path = make_folder(str(tmp_path / "far"), cfg, 11)
    raw, tensors = read_folder(path)
    toks = tokens_for(cfg, 300, 5)
    got = replay_in_process(runner_for(path, "float32", max_tokens=512), trace_tail({"f": toks}, tail=60))["f"].double()
    ref = oracle(path, toks)
    size = ref.pow(2).mean().sqrt().item()
    err = (got - ref).abs().max().item() / size
    seen = plain.chunk_mask(300, None)
    seen[200:, :40] = False
    assert err < 3e-5 and (plain.forward(raw, tensors, toks, seen=seen)[240:] - ref[240:]).abs().max().item() / size > 30 * err


@pytest.mark.parametrize("kind", ["unit", "delta"])
def test_old_state_is_carried(tmp_path, kind):
    """Decays near one keep a sequence's first token in the state over hundreds of rows: another first token shows in the decoded
    rows by far more than the engine's error."""
    cfg = _one_layer(lru(48, 3, 2)) if kind == "unit" else _one_layer(par(attn(1, 1, 8, 8, 0.3, chunk=1), delta(2, 1, 16, 16, 2)))
    path = make_folder(str(tmp_path / "old"), cfg, 12)
    raw, tensors = read_folder(path)
    tensors = dict(tensors)
    if kind == "unit":
        tensors["l0.mix.lam"] = tensors["l0.mix.lam"] * 0 - 9.0
    else:
        tensors["l0.mix.right.dt_bias"] = tensors["l0.mix.right.dt_bias"] * 0 - 9.0
        tensors["l0.mix.right.b"] = tensors["l0.mix.right.b"] * 0.0                  # every row corrects by half ...
        tensors["l0.mix.right.k"] = tensors["l0.mix.right.k"] * 0.0                  # ... along a key that is no direction at all,
        tensors["l0.mix.right.k"][0] = 3.0 * tensors["l0.mix.right.q"][0]            # but for one number of it
    save(path, tensors)
    toks = tokens_for(cfg, 400 if kind == "unit" else 60, 6)
    runner = runner_for(path, "float32", max_tokens=512)
    got = replay_in_process(runner, trace_tail({"f": toks}, tail=len(toks) // 4))["f"].double()
    ref = plain.forward(raw, tensors, toks)
    size = ref.pow(2).mean().sqrt().item()
    err = (got - ref).abs().max().item() / size
    other = plain.forward(raw, tensors, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    late = slice(3 * len(toks) // 4, None) if kind == "unit" else slice(2, None)
    assert err < 3e-5 and (ref[late] - other[late]).abs().max().item() / size > 30 * err


def test_long_decoding(folders):
    """600 single-token steps behind a short prompt, through many chunks."""
    for name, dtype in (("D", "float32"), ("F", "bfloat16"), ("E", "bfloat16")):
        cfg = CASES[name][0]
        toks = tokens_for(cfg, 620, 77)
        runner = runner_for(folders[name, dtype], dtype, max_tokens=704)
        got = replay_in_process(runner, trace_tail({"l": toks}, tail=600))["l"]
        compare(got, folders[name, dtype], toks, dtype, "long decoding")
        for gi, g in enumerate(runner.cache.groups):
            assert g.pool.used_count == 0


def test_a_long_prompt_in_one_step(tmp_path):
    """1,100 tokens in one step and the rest behind it, on the tensor-core kernels, with chunks of 300 and none, wide enough for
    the tcgen05 products and the experts' big tiles."""
    cfg = model(83, 256, [par(attn(4, 2, 128, 128, 0.1, chunk=300, rot=(64, 10000.0)), delta(4, 2, 64, 64, 4), mlp=moe(64, 4, 2, identity=1, shared=128)),
                          lru(384, 4, 4, mlp=dense(512)), par(attn(6, 3, 64, 64, 0.15, rot=(16, 100.0)), delta(2, 2, 128, 128, 2))], scale=3.0)
    path = make_folder(str(tmp_path / "long"), cfg, 2, SETTLED)
    toks = tokens_for(cfg, 1150, 4)
    runner = runner_for(path, "bfloat16", max_tokens=1216)
    check_trace(runner, path, {"p": toks}, trace_tail({"p": toks}, tail=50), "bfloat16", "long prompt")


# ---------------------------------------------------------------------------------------------- through the front doors
@pytest.mark.parametrize("name", ["A", "E"])
def test_greedy_generation_through_the_scheduler(folders, name):
    from openinfer_b200 import LLM, SamplingParams
    cfg, tensors = read_folder(folders[name, "float32"])
    prompts = [tokens_for(cfg, n, 70 + n) for n in (1, 9, 33, 70)]
    n_new = 20

    def greedy(prompt):
        toks = list(prompt)
        for _ in range(n_new):
            toks.append(int(plain.forward(cfg, tensors, toks)[-1].argmax()))
        return toks[len(prompt):]

    want = [greedy(p) for p in prompts]
    llm = LLM(folders[name, "float32"], dtype="float32", max_cache_tokens=512, max_prefill_tokens=13, max_decode_batch=3)
    assert llm.generate(prompts, max_tokens=n_new) == want
    assert llm.runner.cache.min_free_pages() == llm.runner.cache.num_pages
    assert [llm.generate([p], max_tokens=n_new)[0] for p in prompts] == want
    llm16 = LLM(folders[name, "bfloat16"], dtype="bfloat16", max_cache_tokens=512, max_decode_batch=4)
    sp = SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=5)
    a = llm16.generate(prompts, sp, max_tokens=12)
    assert a == llm16.generate(prompts, sp, max_tokens=12) and all(len(t) == 12 for t in a)
    assert llm16.runner.cache.slot_pool.used_count == 0


@pytest.mark.parametrize("name", ["C", "F"])
def test_batch_invariant_mode_is_bitwise(folders, name):
    """In batch-invariant mode a request's bfloat16 logits are the same bit for bit alone and among others."""
    from openinfer_b200.engine.runner import StepEntry
    from openinfer_b200.kernels import policy
    cfg = CASES[name][0]
    reqs = {f"b{i}": tokens_for(cfg, n, 90 + i) for i, n in enumerate([40, 65, 1, 33])}
    policy.set_batch_invariant(True)
    try:
        def run(ids):
            runner = runner_for(folders[name, "bfloat16"], "bfloat16", max_tokens=512)
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
    cfg, tensors = read_folder(folders[name, "float32"])
    want = []
    for _ in range(5):
        want.append(int(plain.forward(cfg, tensors, [7, 8, 9] + want)[-1].argmax()))
    out = subprocess.run([sys.executable, "-m", "openinfer_b200", "--model-path", folders[name, "float32"], "--dtype", "float32",
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
        got = replay_trace_run(folders[name, dtype], dtype, steps, str(tmp_path / dtype), max_tokens, cfg["vocab"])
        for rid, t in requests.items():
            compare(got[rid], folders[name, dtype], t, dtype, f"trace_run/{dtype}/{rid}")
