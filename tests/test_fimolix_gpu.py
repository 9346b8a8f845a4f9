"""The Fimolix decoder on the GPU against the plain implementation: every new kernel alone against float64, then whole models (tiny
configurations that differ in every size) replayed whole, with the last tokens one by one, in portions down to two tokens, and
mixed in a pool so small that pages and state slots are used again; window edges; mistakes planted in the plain model that have
to show; decoding from CUDA graphs; greedy generation through `Engine.generate`, the scheduler and the command line."""

import copy
import json
import subprocess
import sys
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from tests.gpu_helpers import BF16, F32, assert_close, i32, table_tensor
from tests.plain import fimolix_plain as plain_model
from tests.plain.fimolix_plain import PlainFimolix, greedy_generate, logits_of
from tests.test_replay_gpu import cuts_changing, cuts_last32, cuts_whole, replay, steps_alone, steps_decode_together, steps_mixed
from tests.tiny import random_tokens
from tests.tiny_fimolix import CONFIGS, PAGE_SIZE, write_tiny_fimolix

pytestmark = pytest.mark.gpu

DT = [torch.float32, torch.bfloat16]
F32_ATOL = 5e-5
BF16_REL = 0.05
LENGTHS = {"F1": [1, 5, 17, 70, 33, 130, 64], "F2": [7, 40, 64, 97, 2, 150]}
F64 = torch.float64


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def tol(adt):
    return F32 if adt == torch.float32 else BF16


def step_of(step, at, slot):
    """The step's tensors for [(request, tokens)], requests at positions `at` (advanced) in slots `slot`."""
    q_start, slots, starts = [0], [], []
    for rid, n in step:
        starts.append(at[rid])
        q_start.append(q_start[-1] + n)
        slots.append(slot[rid])
        at[rid] += n
    return SimpleNamespace(q_start=i32(q_start), slots=i32(slots), start_pos=i32(starts), B=len(step), T=q_start[-1],
                           max_q_len=max(n for _, n in step), h_q_start=q_start)


# ------------------------------------------------------------------------------------------ kernels alone
CONV_CASES = [  # nq, nkv, maps, dim, dv, d, taps, q/k norm
    (4, 2, 2, 16, 32, 32, 4, True),             # rows without padding
    (6, 2, 2, 8, 24, 32, 3, True),              # padding behind keys and values
    (2, 1, 2, 64, 72, 128, 2, True),
    (5, 5, 2, 32, 136, 144, 4, True),           # values wider than two maps
    (3, 1, 1, 24, 16, 32, 4, True),             # one map; 24 channels are no power of two
    (3, 3, 2, 5, 7, 16, 6, True),               # nothing is a multiple of eight; six taps
    (8, 4, 2, 128, 256, 256, 3, False),
    (2, 2, 2, 256, 8, 512, 1, True),            # one tap: a factor, no state
    (1, 1, 3, 16, 40, 64, 9, True),             # three maps, nine taps: more than the tokens of a chunk of the plain kernel
]


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("case", CONV_CASES, ids=["-".join(map(str, c)) for c in CONV_CASES])
def test_convolution_norms_and_rows_across_portions_slots_and_pages(adt, case):
    """Steps over three request slots: a portion's first tokens reach back into the rows the request left (not those of the request
    in front in the batch, nor what the slot's former owner left), a request may be left out of a step; every row lands in its page,
    zeros around it.  The bits of one whole pass whatever the cuts."""
    from tensorline_b200 import ops
    nq, nkv, maps, dim, dv, d, taps, normed = case
    C = (nq + nkv) * maps * dim + nkv * dv
    eps, ps = 1e-5, 4
    lens = {"a": 60, "b": 9, "c": 41, "d": 10}
    slot = {"a": 2, "b": 0, "c": 0, "d": 1}                  # c takes b's slot
    proj = {k: rnd(n, C, seed=i, dtype=adt) for i, (k, n) in enumerate(lens.items())}
    w = rnd(C, taps, seed=20, dtype=torch.bfloat16)
    wq, wk = (rnd(dim, seed=21) + 1, rnd(dim, seed=22) + 1) if normed else (None, None)
    max_pages = 20
    g = torch.Generator().manual_seed(5)
    perm = torch.randperm(60, generator=g).tolist()
    page_of = {k: perm[i * 15:(i + 1) * 15] for i, k in enumerate(lens)}

    def table(live):
        rows = [[] for _ in range(4)]
        for k in live:
            rows[slot[k]] = page_of[k]
        return table_tensor(rows, max_pages, 60)

    def want(k):
        y = plain_model.short_conv(proj[k].double(), w.double())
        n = lens[k]
        q, kk, v = y[:, :nq * maps * dim].view(n, nq, maps, dim), y[:, nq * maps * dim:(nq + nkv) * maps * dim].view(n, nkv, maps, dim), \
            y[:, (nq + nkv) * maps * dim:].view(n, nkv, dv)
        if normed:
            q, kk = plain_model.unit(q, eps) * wq.double(), plain_model.unit(kk, eps) * wk.double()
        Q, K, V = torch.zeros(n, nq, maps, d, dtype=F64), torch.zeros(n, nkv, d, dtype=F64), torch.zeros(n, nkv, d, dtype=F64)
        for m in range(maps):
            Q[:, :, m, m * dim:(m + 1) * dim] = q[:, :, m]
            K[:, :, m * dim:(m + 1) * dim] = kk[:, :, m]
        V[:, :, :dv] = v
        return Q.reshape(n, -1), K, V

    def run(steps):
        kp, vp = (torch.full((61, nkv, ps, d), float("nan"), dtype=adt, device="cuda") for _ in range(2))
        state = torch.full((4, taps - 1, C), 50.0, dtype=adt, device="cuda")
        at, got = {k: 0 for k in lens}, {k: [] for k in lens}
        for step in steps:
            for k, _ in step:
                if at[k] == 0:
                    state[slot[k]].zero_()                   # what the runner does at admission
            frm = dict(at)
            ctx = step_of(step, at, slot)
            p = torch.cat([proj[k][frm[k]:frm[k] + n] for k, n in step]).contiguous().cuda()
            q = torch.full((ctx.T, nq * maps * d), float("nan"), dtype=adt, device="cuda")
            ops.conv_heads(p, w.cuda(), state if taps > 1 else None, ctx, table([k for k, _ in step]), ps, q, kp, vp, nq=nq, nkv=nkv, maps=maps,
                           dim=dim, dv=dv, q_norm=wq.cuda() if normed else None, k_norm=wk.cuda() if normed else None, eps=eps)
            for (k, n), r in zip(step, ctx.h_q_start):
                got[k].append(q[r:r + n])
        assert at == lens and bool((state[3] == 50.0).all())
        rows = {k: [torch.stack([x[page_of[k][i // ps], :, i % ps] for i in range(lens[k])]) for x in (kp, vp)] for k in lens}
        return {k: torch.cat(v) for k, v in got.items()}, rows
    whole, whole_rows = run([[("a", 60), ("b", 9), ("d", 10)], [("c", 41)]])
    cut, cut_rows = run([[("a", 3), ("b", 4), ("d", 1)], [("b", 1), ("d", 2)], [("b", 4)], [("c", 2), ("a", 1), ("d", 1)], [("a", 1), ("c", 1), ("d", 1)],
                         [("d", 5), ("a", 40), ("c", 20)], [("a", 1), ("c", 1)], [("c", 17), ("a", 14)]])
    for k in lens:
        Q, K, V = want(k)
        for what, got, rows in (("whole", whole, whole_rows), ("cut", cut, cut_rows)):
            assert_close(got[k], Q, f"{what}: queries of {k}", **tol(adt))
            assert_close(rows[k][0], K, f"{what}: keys of {k}", **tol(adt))
            assert_close(rows[k][1], V, f"{what}: values of {k}", **tol(adt))
        assert torch.equal(whole[k], cut[k]) and all(torch.equal(a, b) for a, b in zip(whole_rows[k], cut_rows[k])), f"request {k}: the cuts show"
    if taps > 1:                                             # a state that is lost at a cut shows
        lost = plain_model.short_conv(proj["a"][3:].double(), w.double())[0]
        assert float((lost - plain_model.short_conv(proj["a"].double(), w.double())[3]).abs().max()) > 0.1


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("H,dv,d", [(4, 64, 64), (3, 24, 32), (5, 7, 16), (2, 256, 256), (16, 128, 256), (1, 320, 320)])
def test_difference_of_two_maps_and_its_norm(adt, H, dv, d):
    from tensorline_b200 import ops
    T, lam, eps, c = 37, 0.7, 1e-5, 0.4
    a = rnd(T, H, 2, d, seed=1, dtype=adt)
    a[5] *= 1e-3                                             # eps counts
    y = torch.full((T, H * dv), float("nan"), dtype=adt, device="cuda")
    ops.map_difference(a.reshape(T, -1).cuda(), y, H, dv, lam, eps, c)
    o = a[:, :, 0, :dv].double() - lam * a[:, :, 1, :dv].double()
    assert_close(y.view(T, H, dv), plain_model.unit(o, eps) * c, "difference", **tol(adt))


def _rows(q, k, v, pos_q, scale, cap, window, sink):
    """q [n, nq, d] at positions pos_q over k, v [len, nkv, d]."""
    n, nq, d = q.shape
    g = nq // k.shape[1]
    out = torch.empty(n, nq, v.shape[2], dtype=F64)
    for i, p in enumerate(pos_q):
        lo = max(0, p - window + 1) if window else 0
        for h in range(nq):
            s = (k[lo:p + 1, h // g] @ q[i, h]) * scale
            if cap is not None:
                s = plain_model.capped(s, cap)
            P = torch.softmax(s, 0) if sink is None else plain_model.softmax_with_sink(s, sink[h])
            out[i, h] = P @ v[lo:p + 1, h // g]
    return out


CAP_CASES = [  # nq, nkv, d, page, context lengths before the step, tokens in the step, cap, window, sink
    (4, 2, 16, 4, [0, 5, 31], [9, 1, 2], 1.5, None, False),
    (8, 2, 64, 16, [300, 0, 65, 129], [1, 1, 1, 1], 4.0, None, True),
    (8, 2, 64, 16, [300, 40], [1, 1], 30.0, None, False),             # far below the cap: the polynomial
    (6, 2, 48, 16, [63, 64, 1399], [1, 1, 1], 3.0, 100, True),
    (18, 1, 64, 16, [2200, 64], [1, 1], 6.0, None, False),            # more than sixteen rows a key/value head, ranges of keys
    (14, 2, 64, 64, [15, 0], [17, 200], 5.0, None, False),
    (8, 4, 128, 16, [0, 700, 41], [200, 37, 90], 2.0, None, False),
    (8, 2, 128, 16, [0, 1000], [600, 300], 25.0, None, False),
    (4, 2, 64, 16, [100, 0, 517], [900, 300, 140], 8.0, 130, True),
    (4, 1, 256, 32, [300, 0], [40, 150], 4.0, None, True),
    (4, 2, 192, 16, [100, 7], [1, 1], 4.0, 33, False),
    (2, 1, 80, 16, [0, 100], [150, 1], None, 70, True),               # no cap: a window and a sink
]


@pytest.mark.parametrize("case", CAP_CASES, ids=[f"q{c[0]}kv{c[1]}d{c[2]}p{c[3]}n{len(c[4])}cap{c[6]}w{c[7]}" for c in CAP_CASES])
@pytest.mark.parametrize("kernel", ["exact_f32", "exact_bf16", "tensor_core_bf16", "tma_bf16", "tcgen05_bf16", "pair_bf16", "step_bf16"])
def test_attention_with_capped_scores(case, kernel):
    """Decode and prefill attention over scattered pages, scores cap * tanh(score / cap), against the plain formula.  The last query
    of the first request meets a key whose raw score stands far above the cap and one just under it: without the cap the first
    would take all the weight."""
    from tensorline_b200 import ops, ops_attention, ops_gemm
    nq, nkv, d, ps, ctx_lens, step_lens, cap, window, sinks = case
    single = all(n == 1 for n in step_lens)
    if kernel == "tcgen05_bf16" and d % 64:
        pytest.skip("the tcgen05 kernels take head sizes that are multiples of 64")
    if kernel == "pair_bf16" and d not in (64, 128):
        pytest.skip("the pair kernel takes head sizes 64 and 128")
    if kernel == "tma_bf16" and (d % 64 or not single):
        pytest.skip("the TMA decode kernel takes single tokens and head sizes that are multiples of 64")
    adt = torch.float32 if kernel == "exact_f32" else torch.bfloat16
    scale = 1.4 * d ** -0.5
    sink = rnd(nq, seed=3) + 1 if sinks else None
    B = len(ctx_lens)
    max_pages, num_pages = 160, 320
    kps = torch.full((num_pages + 1, nkv, ps, d), 37.0, dtype=adt)
    vps = torch.full_like(kps, -53.0)
    rows, qs, want, pos_all, slot_all = [], [], [], [], []
    for b in range(B):
        n = ctx_lens[b] + step_lens[b]
        k, v = rnd(n, nkv, d, seed=20 + b, dtype=adt), rnd(n, nkv, d, seed=40 + b, dtype=adt)
        q = rnd(step_lens[b], nq, d, seed=60 + b, scale=2.0, dtype=adt)
        if b == 0 and n > 4:
            lo = max(0, n - window) if window else 0
            q[-1] = 0.0; q[-1, :, 0] = 8.0
            k[lo] = 0.0; k[lo, :, 0] = 3.0 * (cap or 4.0) / (8.0 * scale)
            k[lo + 1] = 0.0; k[lo + 1, :, 0] = 0.9 * (cap or 4.0) / (8.0 * scale)
        gen = torch.Generator().manual_seed(100 + b)
        mine = (torch.randperm(num_pages // B, generator=gen)[:-(-n // ps)] * B + b).tolist()
        for i in range(n):
            kps[mine[i // ps], :, i % ps] = k[i]
            vps[mine[i // ps], :, i % ps] = v[i]
        rows.append(mine)
        pq = list(range(ctx_lens[b], n))
        kd_, vd_, sd = k.double(), v.double(), None if sink is None else sink.double()
        want.append(_rows(q.double(), kd_, vd_, pq, scale, cap, window, sd))
        if b == 0 and cap is not None and cap <= 8:
            gap = _rows(q[-1:].double(), kd_, vd_, pq[-1:], scale, None, window, sd) - want[0][-1:]
            assert float(gap.abs().max()) > 0.05, "a cap that is left out must show"
        qs.append(q)
        pos_all += pq
        slot_all += [b] * step_lens[b]
    q_all = torch.cat(qs).reshape(-1, nq * d).cuda()
    T = q_all.shape[0]
    out = torch.full((T, nq * d), float("nan"), dtype=adt, device="cuda")
    table = table_tensor(rows, max_pages, num_pages)
    kd, vd = kps.cuda(), vps.cuda()
    sk = None if sink is None else sink.cuda()
    q_start = [0]
    for n in step_lens:
        q_start.append(q_start[-1] + n)
    W = torch.cat(want)
    args = (q_all, nq * d, out, kd, vd, table, ps, i32(q_start), i32(ctx_lens), i32(list(range(B))))

    def close(what):
        ops_gemm.check_status()
        assert_close(out.view(T, nq, d), W, what, **tol(adt))
        out.fill_(float("nan"))
    if kernel.startswith("exact"):
        ops.attn_tokenwise(q_all, nq * d, out, kd, vd, table, ps, i32(pos_all), i32(slot_all), nq, nkv, d, window, scale, sink=sk, cap=cap)
    elif kernel in ("tensor_core_bf16", "tma_bf16"):
        if single:
            span = max(c + 1 for c in ctx_lens)
            if window:
                span = min(span, window + 63)
            tiles = -(-span // 64)
            for splits_wanted in (1, 3, 6, 64):             # one range, ranges that merge in a cluster, more ranges than tiles
                rng = -(-tiles // min(splits_wanted, tiles)) * 64
                splits = -(-tiles * 64 // rng)
                po = torch.full((B, nq, splits, d), float("nan"), device="cuda")
                pml = torch.full((B, nq, splits, 2), float("nan"), device="cuda")
                for cluster in (False, True) if kernel == "tma_bf16" else (None,):
                    ops_attention.decode(*args, B, nq, nkv, d, window, scale, rng, splits, po, pml, tma=kernel == "tma_bf16", cluster=cluster,
                                         sink=sk, cap=cap)
                    if kernel == "tensor_core_bf16" or splits_wanted != 64:
                        close(f"decode, {splits} ranges, cluster {cluster}")
            if kernel == "tma_bf16":
                return
            out.fill_(float("nan"))
        ops_attention.prefill(*args, q_start, nq, nkv, d, window, scale, sink=sk, cap=cap)
    elif kernel == "tcgen05_bf16":                          # the one-tile kernel
        ops_attention.prefill_tc(*args, q_start, nq, nkv, d, window, scale, sink=sk, cap=cap)
    elif kernel == "pair_bf16":                             # two query tiles a block, in both forms, keys dealt out or not
        for form in (False, "64"):
            for ksplit in (1, 3) if not window else (1,):
                if ops_attention.prefill_tc_pair(*args, q_start, nq, nkv, d, window, scale, p_in_tmem=form, ksplit=ksplit, sink=sk, cap=cap):
                    close(f"pair kernel, form {form}, {ksplit} runs of keys")
                else:
                    assert ps < 8
        if cap is not None:
            assert not ops_attention.prefill_tc_pair(*args, q_start, nq, nkv, d, window, scale, p_in_tmem=True, sink=sk, cap=cap)
        return
    else:                                                   # the step's own choice of kernels
        ctx = SimpleNamespace(B=B, T=T, decode_only=single, page_size=ps, q_start=i32(q_start), start_pos=i32(ctx_lens),
                              slots=i32(list(range(B))), h_q_start=q_start, h_start_pos=list(ctx_lens), h_slots=list(range(B)),
                              graph_max_ctx=0, max_ctx=max(c + n for c, n in zip(ctx_lens, step_lens)), scratch={})
        ops_attention.attend_bf16(q_all, out, ctx, kd, vd, table, nq, nkv, d, window, scale, sink=sk, cap=cap)
    close(kernel)


def test_the_caps_of_one_launch_do_not_reach_the_next():
    """The libraries keep the cap between a launcher's calls: a launch without one behind a launch with one is uncapped."""
    from tensorline_b200 import ops_attention
    nq, nkv, d, ps, n = 4, 2, 64, 16, 200
    q, k, v = rnd(n, nq, d, seed=1, scale=2.0, dtype=torch.bfloat16), rnd(n, nkv, d, seed=2, dtype=torch.bfloat16), rnd(n, nkv, d, seed=3, dtype=torch.bfloat16)
    pages = -(-n // ps)
    kp, vp = (torch.zeros(pages + 1, nkv, ps, d, dtype=torch.bfloat16) for _ in range(2))
    for i in range(n):
        kp[i // ps, :, i % ps], vp[i // ps, :, i % ps] = k[i], v[i]
    table = table_tensor([list(range(pages))], pages, pages)
    out = torch.empty(n, nq * d, dtype=torch.bfloat16, device="cuda")
    args = (q.reshape(n, -1).cuda(), nq * d, out, kp.cuda(), vp.cuda(), table, ps, i32([0, n]), i32([0]), i32([0]), [0, n], nq, nkv, d, None, 0.2)
    for fn in (ops_attention.prefill, ops_attention.prefill_tc, ops_attention.prefill_tc_pair):
        for cap in (2.0, None):
            fn(*args, cap=cap)
            assert_close(out.view(n, nq, d), _rows(q.double(), k.double(), v.double(), range(n), 0.2, cap, None, None), f"{fn.__name__} cap {cap}", **BF16)


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("W", [48, 33, 2048, 5120, 20000])
def test_a_stream_that_takes_a_normed_addend_and_is_read_as_it_is(adt, W):
    from tensorline_b200.parts import Runtime
    from tensorline_b200.parts.linear import PostNormed
    from tensorline_b200.parts.norm import RMSNorm, read_stream
    rt, eps, T = Runtime(torch.device("cuda"), adt), 1e-5, 7
    x0, a, w = rnd(T, W, seed=1, scale=3.0), rnd(T, W, seed=2, scale=0.2, dtype=adt), rnd(W, seed=3, scale=0.3, dtype=torch.bfloat16)
    norm = RMSNorm(rt, W, eps, tensor="", one_plus=True, cast_first=False)
    norm.bind({"n": w.cuda()}, "n")
    want = x0.double() + plain_model.one_plus_norm(a.double(), w.double(), eps)
    x = x0.clone().cuda()
    h = read_stream(x, None, rt)
    assert torch.equal(h.cpu(), x0.to(adt))
    h = read_stream(x, PostNormed(a.cuda(), norm.weight, eps), rt)
    assert_close(x, want, "sum", rtol=1e-5, atol=2e-5)
    assert torch.equal(h, x.to(adt)) and h.dtype == adt
    x = x0.clone().cuda()                                    # the model's norm of picked rows: x stays as it is
    got = norm.add_norm(x, PostNormed(a.cuda(), norm.weight, eps), rows=i32([6, 0, 2]))
    assert torch.equal(x.cpu(), x0)
    assert_close(got, plain_model.one_plus_norm(want, w.double(), eps)[[6, 0, 2]], "final norm", **tol(adt))


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("nq,d", [(5, 24), (3, 7), (16, 128)])
def test_gate_of_a_head_from_columns_of_a_wider_product(adt, nq, d):
    from tensorline_b200 import ops
    T = 11
    o, wide = rnd(T, nq * d, seed=1, dtype=adt), rnd(T, nq + 13, seed=2, scale=2.0).cuda()
    got = o.clone().cuda()
    ops.head_gate(got, wide[:, 13:], nq, d)
    want = o.double().view(T, nq, d) * plain_model.sig(wide[:, 13:].double().cpu())[..., None]
    assert_close(got.view(T, nq, d), want, "gate", **tol(adt))


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("T,H,I", [(3, 40, 24), (5, 2048, 4096), (16, 4096, 2048), (48, 2048, 6016), (300, 256, 512), (1536, 2048, 4096)])
def test_feed_forward_with_gelu_and_no_gate(adt, T, H, I):
    from tensorline_b200.parts import FEED_FORWARDS, PartSpec, Runtime
    from tensorline_b200.parts.linear import resolve
    if adt == torch.float32 and T * H * I > 1 << 26:
        pytest.skip("the 32-bit product at these sizes is tested elsewhere")
    ff = FEED_FORWARDS.build(PartSpec("plain_mlp", {"hidden": H, "intermediate": I, "activation": "gelu_tanh", "names": {"up": "up", "down": "down"}}),
                             Runtime(torch.device("cuda"), adt))
    w = {"m.up": rnd(I, H, seed=1, scale=2 * H ** -0.5, dtype=torch.bfloat16).cuda(), "m.down": rnd(H, I, seed=2, scale=I ** -0.5, dtype=torch.bfloat16).cuda()}
    ff.bind(w, "m")
    h = rnd(T, H, seed=3, dtype=adt).cuda()
    got = resolve(ff.forward(h, None))
    want = plain_model.feed_forward(h.double(), {"up": w["m.up"].double(), "down": w["m.down"].double()})
    assert_close(got, want, "feed-forward", **(dict(rtol=1e-4, atol=1e-4) if adt == torch.float32 else dict(rtol=0.03, atol=0.05)))


# ------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module", params=["F1", "F2"])
def model(request, tmp_path_factory):
    name = request.param
    folder = write_tiny_fimolix(name, tmp_path_factory.mktemp(f"tiny_{name}"))
    plain = PlainFimolix(folder)
    V = CONFIGS[name]["vocab"]
    reqs = {f"r{i}": random_tokens(V, n, seed=100 + i) for i, n in enumerate(LENGTHS[name])}
    want = {rid: logits_of(plain, toks) for rid, toks in reqs.items()}
    return dict(name=name, folder=folder, reqs=reqs, want=want, page=PAGE_SIZE[name], vocab=V, plain=plain)


def check(model, dtype, got, what):
    """32-bit: every position within F32_ATOL (times the largest |logit| where that is above one).  bfloat16: the largest logit
    error of a position within BF16_REL of the request's largest |logit|."""
    assert got, "nothing was compared"
    for (rid, p), row in got.items():
        ref = model["want"][rid][p]
        err = float((row - ref).abs().max())
        bound = F32_ATOL * max(1.0, float(ref.abs().max())) if dtype == "float32" else BF16_REL * float(model["want"][rid].abs().max())
        assert err <= bound, f"{what}: request {rid} position {p}: max abs err {err:.3e} > {bound:.3e}"


def test_the_model_is_chosen_by_its_configuration_and_every_layer_matches(model):
    """The residual stream after every layer, with what still waits to be added, 32-bit engine against the plain model."""
    from tensorline_b200.replay import TraceSession, make_runner
    runner, cfg = make_runner(model["folder"], "float32", 256, page_size=model["page"], max_live=2)
    assert type(cfg).__name__ == "FimolixConfig" and cfg.to_json_dict() == CONFIGS[model["name"]]
    seen = []
    for blk in runner.model.blocks:
        def fwd(x, pending, ctx, cache, orig=blk.forward):
            out = orig(x, pending, ctx, cache)
            y = x.clone()
            out.add_into(y)
            seen.append(y.double().cpu())
            return out
        blk.forward = fwd
    toks = model["reqs"]["r2"]
    TraceSession(runner).run_step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": []}], "end": ["a"]})
    want = []
    logits_of(model["plain"], toks, want)
    assert len(seen) == len(want) == len(CONFIGS[model["name"]]["layers"])
    for i, (g, w) in enumerate(zip(seen, want)):
        assert_close(g, w, f"stream after layer {i}", rtol=5e-5, atol=F32_ATOL * max(1.0, float(w.abs().max())))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_all_schedules_agree_with_the_plain_model(model, dtype):
    results = {}
    for what, cuts in (("whole", cuts_whole), ("last 32 one by one", cuts_last32), ("changing portions", cuts_changing)):
        results[what] = replay(model, dtype, steps_alone(model, cuts), max_tokens=192)
        check(model, dtype, results[what], what)
        assert len(results[what]) == sum(len(t) for t in model["reqs"].values())
    for seed in (1, 2):
        steps, peak = steps_mixed(model, seed)
        assert max(len(s["entries"]) for s in steps) >= 3
        total = sum(-(-len(t) // model["page"]) * model["page"] for t in model["reqs"].values())
        assert peak < total, "the pool must be too small to hold all requests: pages and slots have to be used again"
        results[f"mixed {seed}"] = replay(model, dtype, steps, max_tokens=peak)
        check(model, dtype, results[f"mixed {seed}"], f"mixed {seed}")
        assert len(results[f"mixed {seed}"]) == len(results["whole"])
    if dtype == "float32":                                  # one order of additions per position
        for what, got in results.items():
            for key, row in got.items():
                assert torch.equal(row, results["whole"][key]), f"{what} differs from whole at {key}"


def test_the_forms_of_long_steps_agree_with_the_plain_model(model, monkeypatch):
    """The bfloat16 engine's form of the latent's products per head for long steps, taken from two tokens on."""
    from tensorline_b200.parts import latent
    monkeypatch.setattr(latent, "HEAD_PRODUCT_LIBRARY_MIN_TOKENS", 2)
    for what, steps, most in (("whole", steps_alone(model, cuts_whole), 192), ("changing portions", steps_alone(model, cuts_changing), 192),
                              ("mixed", *steps_mixed(model, 3))):
        check(model, "bfloat16", replay(model, "bfloat16", steps, max_tokens=most), f"long forms, {what}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(model, dtype):
    """A one-token prompt, then 150 tokens decoded one by one: the rows of the convolutions and the pages are carried through 150
    launches, and decoded tokens pass out of every window."""
    toks = random_tokens(model["vocab"], 151, seed=7)
    want = logits_of(model["plain"], toks)
    steps = [{"step": i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
    steps[-1]["end"] = ["x"]
    m2 = dict(model, reqs={"x": toks}, want={"x": want})
    got = replay(m2, dtype, steps, max_tokens=160)
    check(m2, dtype, got, "token by token")
    assert sorted(p for _, p in got) == list(range(151))


def _other_windows(raw, only, by):
    raw = copy.deepcopy(raw)
    raw["layers"][only]["mixer"]["mask"]["size"] += by
    return raw


def test_edges_of_windows_of_owners_and_readers(model):
    """The plain model with one layer's window a position longer or shorter gives other logits from the first position on that
    the window's edge cuts: a key that is wrongly seen (or not seen) shows, in an owner's window and in its readers'.  The engine
    follows the right one: whole, decoded one by one around every edge, and in portions that end on both sides of the edges."""
    toks = random_tokens(model["vocab"], 90, seed=11)
    right = logits_of(model["plain"], toks)
    windows = {i: l["mixer"]["mask"]["size"] for i, l in enumerate(CONFIGS[model["name"]]["layers"]) if "mask" in l["mixer"]}
    for i, size in windows.items():
        for by in (-1, 1):
            other = PlainFimolix(model["folder"])
            other.cfg = _other_windows(other.cfg, i, by)
            gap = (logits_of(other, toks) - right).abs().max(1).values
            first = min(size, size + by)                    # the first position that sees one key more, or one less
            assert float(gap[:first].max()) == 0.0
            assert float(gap[first:].max()) > 1.5 * BF16_REL * float(right.abs().max()), f"layer {i}: a window that is one position off ({by}) must show"
    m2 = dict(model, reqs={"w": toks}, want={"w": right})
    edges = sorted({s + j for s in windows.values() for j in (-1, 0, 1, 2) if 0 < s + j < 90})
    first = min(windows.values())
    cuts = [[90], [first - 1] + [1] * (91 - first), [b - a for a, b in zip([0] + edges, edges + [90]) if b > a]]
    for dtype in ("float32", "bfloat16"):
        for c in cuts:
            assert sum(c) == 90
            got = replay(m2, dtype, steps_alone(m2, lambda n, c=c: c), max_tokens=96)
            check(m2, dtype, got, f"window edges, portions {c[:4]}...")


def test_mistakes_planted_in_the_plain_model_show(model, monkeypatch):
    """What the comparisons above would not let pass: the plain model with a mechanism left out or turned around gives logits
    far beyond the bounds."""
    toks = model["reqs"]["r3"]
    right = model["want"]["r3"]

    def gap():
        return float((logits_of(model["plain"], toks) - right).abs().max()) / float(right.abs().max())
    assert gap() == 0.0
    plants = {
        "no convolution": ("short_conv", lambda x, w: x * w[:, -1]),
        "the convolution's taps turned around": ("short_conv", lambda x, w, f=plain_model.short_conv: f(x, w.flip(1))),
        "no cap": ("capped", lambda s, cap: s),
        "one map only": ("mix_weight", lambda w, diff: 0.0),
        "the maps' weights turned around": ("mix_weight", lambda w, diff, f=plain_model.mix_weight: 2 * diff - f(w, diff)),
        "no norm of the difference": ("head_norm", lambda o, eps: o),
        "no sink": ("softmax_with_sink", lambda s, sink: torch.softmax(s, -1)),
        "no gate": ("head_gates", lambda h, w: torch.ones(h.shape[0], w["g"].shape[0], dtype=F64)),
        "nothing turned": ("turn_pairs", lambda x, rot: x),
        "a plain weight in the norms": ("one_plus_norm", lambda v, w, eps: plain_model.unit(v, eps) * w),
        "no activation": ("gelu", lambda z: z),
        "every earlier key": ("window", lambda T, size: plain_model.causal(T)),
    }
    for what, (name, fn) in plants.items():
        with monkeypatch.context() as m:
            m.setattr(plain_model, name, fn)
            assert gap() > 2 * BF16_REL, f"{what} must show ({gap():.3f})"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decode_graphs_agree_with_eager_steps(model, dtype):
    """Steps of single tokens replayed from CUDA graphs (state slots are fixed addresses, padding rows use the spare slot): three
    live requests in the bucket of four, shrinking as they end; 32-bit: the bits of the eager steps."""
    rids = ["r3", "r5", "r2"]
    steps, decode_steps = steps_decode_together(model, rids, tail=12)
    eager = replay(model, dtype, steps, max_tokens=512)
    graphs = {}

    def after(runner):
        graphs["replays"] = runner.graph_replays
    got = replay(model, dtype, steps, max_tokens=512, graphs=True, after=after)
    assert graphs["replays"] == decode_steps
    check(model, dtype, got, "decode graphs")
    if dtype == "float32":
        for key, row in got.items():
            assert torch.equal(row, eager[key]), f"graph replay differs from the eager step at {key}"


def test_greedy_generation_through_the_engine_and_its_scheduler(model):
    """`Engine.generate`: five prompts through three slots and a small pool (queueing, slots and pages used again, portions of
    16 tokens), 32-bit, against greedy decoding with the plain model."""
    from tensorline_b200 import Engine, SamplingParams
    prompts = [random_tokens(model["vocab"], n, seed=50 + n) for n in (9, 2, 40, 5, 21)]
    want = [greedy_generate(model["plain"], p, 8) for p in prompts]
    for graphs in (False, True):
        eng = Engine(str(model["folder"]), dtype="float32", block_size=model["page"], num_blocks=160 // model["page"], max_num_seqs=3,
                     max_model_len=64, max_batched_tokens=16, cuda_graphs=graphs, overlap=graphs)
        got = [o.token_ids for o in eng.generate(prompts, SamplingParams(max_tokens=8, ignore_eos=True))]
        assert got == want, f"graphs {graphs}: {got} != {want}"
        st = eng.stats()
        assert st["free_pages"] == st["num_pages"] and st["max_running_seen"] == 3 and (st["graph_replays"] > 0) == graphs


@pytest.mark.parametrize("name", ["F3", "F4", "F5", "F6"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_further_shapes_of_the_design(name, dtype, tmp_path):
    """Odd head sizes and a width that is a multiple of nothing; sizes that the tensor-core kernels take, with prompts of hundreds
    of tokens; latents wider than those kernels take; no latent at all: whole requests, changing portions and a small pool against
    the plain model."""
    folder = write_tiny_fimolix(name, tmp_path / name)
    plain = PlainFimolix(folder)
    V = CONFIGS[name]["vocab"]
    lengths = [290, 3, 400, 130] if name == "F4" else [3, 50, 1, 81, 33]
    reqs = {f"r{i}": random_tokens(V, n, seed=300 + i) for i, n in enumerate(lengths)}
    m = dict(name=name, folder=folder, reqs=reqs, want={r: logits_of(plain, t) for r, t in reqs.items()}, page=PAGE_SIZE[name], vocab=V)
    most = max(128, -(-max(lengths) // 64) * 64)
    whole = replay(m, dtype, steps_alone(m, cuts_whole), max_tokens=most)
    check(m, dtype, whole, "whole")
    cut = replay(m, dtype, steps_alone(m, cuts_changing), max_tokens=most)
    check(m, dtype, cut, "changing portions")
    steps, peak = steps_mixed(m, 3, max_live=3)
    mixed = replay(m, dtype, steps, max_tokens=peak)
    check(m, dtype, mixed, "mixed")
    if dtype == "float32":
        assert all(torch.equal(cut[k], whole[k]) and torch.equal(mixed[k], whole[k]) for k in whole)


def test_generate_from_the_command_line(model, capsys):
    """The `tensorline` command with token ids, 32-bit, against greedy decoding with the plain model."""
    from tensorline_b200 import cli
    assert cli.main(["--model", str(model["folder"]), "--dtype", "float32", "--prompt-ids", "5,9,40,17", "--prompt-ids", "7",
                     "--max-tokens", "5", "--ignore-eos", "--block-size", str(model["page"]), "--num-blocks", "16",
                     "--max-num-seqs", "4", "--max-model-len", "64"]) == 0
    lines = [json.loads(l) for l in capsys.readouterr().out.splitlines() if l.startswith("{")]
    assert [l["token_ids"] for l in lines] == [greedy_generate(model["plain"], [5, 9, 40, 17], 5), greedy_generate(model["plain"], [7], 5)]


def test_the_replay_program_with_this_design(model, tmp_path):
    """`bin/trace_run` itself, 32-bit: JSON lines in, `done <step>` lines and <step>.f32 files out; a request that is left
    out of a step, one that starts in another's freed slot, portions of two tokens."""
    if model["name"] != "F1":
        pytest.skip("one configuration is enough for the command-line protocol")
    reqs = model["reqs"]
    a, b, c = reqs["r3"], reqs["r4"], reqs["r2"]
    lines = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:2], "want": [1]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [len(b) - 3]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[30:32], "want": []}, {"id": "c", "tokens": c, "want": [len(c) - 1]}], "end": ["c"]},
        {"step": 3, "entries": [{"id": "a", "tokens": a[32:], "want": [len(a) - 33]}], "end": ["a"]},
    ]
    out = tmp_path / "out"
    root = Path(__file__).resolve().parent.parent
    proc = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(model["folder"]), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "128", "--page-size", "8", "--max-live", "2"],
                          input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    V = model["vocab"]
    got = {n: torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, V).astype(np.float64)) for n in range(4)}
    assert [got[n].shape[0] for n in range(4)] == [3, 1, 1, 1]
    wa, wb, wc = model["want"]["r3"], model["want"]["r4"], model["want"]["r2"]
    for row, ref in ((got[0][0], wa[0]), (got[0][1], wa[29]), (got[0][2], wb[1]), (got[1][0], wb[-1]), (got[2][0], wc[-1]), (got[3][0], wa[-1])):
        assert float((row - ref).abs().max()) <= F32_ATOL * max(1.0, float(ref.abs().max()))
