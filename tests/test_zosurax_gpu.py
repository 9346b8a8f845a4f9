"""The Zosurax decoder on the GPU against the plain implementation: every new kernel alone against a float64 loop, then whole
models (tiny configurations that differ in every size) replayed whole, with the last tokens one by one, in portions down to two
tokens, and mixed in a pool so small that pages and state slots are used again; mistakes planted in the plain model that have to
show; decoding from CUDA graphs; greedy generation through `Engine.generate`, the scheduler and the command line."""

import json
import subprocess
import sys
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from tests.gpu_helpers import BF16, F32, assert_close, i32, table_tensor
from tests.plain import zosurax_plain as plain_model
from tests.plain.zosurax_plain import PlainZosurax, greedy_generate, logits_of
from tests.test_replay_gpu import cuts_changing, cuts_last32, cuts_whole, replay, steps_alone, steps_decode_together, steps_mixed
from tests.tiny import random_tokens
from tests.tiny_zosurax import CONFIGS, PAGE_SIZE, write_tiny_zosurax

pytestmark = pytest.mark.gpu

DT = [torch.float32, torch.bfloat16]
F32_ATOL = 5e-5
BF16_REL = 0.05
LENGTHS = {"Z1": [1, 5, 17, 70, 33, 130, 64], "Z2": [7, 40, 64, 97, 2, 150]}
F64 = torch.float64


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def tol(adt):
    return F32 if adt == torch.float32 else BF16


def step_of(step, at, slot):
    """The step's tensors for [(request, tokens)], requests at positions `at` (advanced) in slots `slot`."""
    pos, req, q_start, slots = [], [], [0], []
    for rid, n in step:
        pos += list(range(at[rid], at[rid] + n))
        req += [slot[rid]] * n
        q_start.append(q_start[-1] + n)
        slots.append(slot[rid])
        at[rid] += n
    return SimpleNamespace(pos=i32(pos), req_slot=i32(req), q_start=i32(q_start), slots=i32(slots), B=len(step), T=len(pos),
                           decode_only=all(n == 1 for _, n in step), h_q_start=q_start)


# ------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("W", [48, 33, 1024, 5120, 12288])
def test_sum_of_waiting_addends_and_its_norm(adt, W):
    from tensorline_b200 import ops
    T, eps = 9, 1e-5
    x0, base, row = rnd(T, W, seed=1, scale=3.0), rnd(T, W, seed=2), rnd(W, seed=3)
    adds = [(rnd(T, W, seed=10 + i, dtype=adt), rnd(W, seed=20 + i)) for i in range(3)]
    w = rnd(W, seed=4, dtype=adt)

    def total(n, with_base, with_row, scaled=True):
        v = x0.double() + (base.double() if with_base else 0.0) + (row.double() if with_row else 0.0)
        for a, s in adds[:n]:
            v = v + a.double() * (s.double() if scaled else 1.0)
        return v
    for n, b, r in ((0, False, False), (1, False, True), (2, True, True), (3, True, False)):
        x = x0.clone().cuda()
        h = torch.empty(T, W, dtype=adt, device="cuda")
        kw = dict(base=base.cuda() if b else None, row=row.cuda() if r else None, w=w.cuda(), eps=eps)
        dev = [(a.cuda(), s.cuda()) for a, s in adds[:n]]
        ops.sum_norm(x, dev, h=h, **kw)
        want = total(n, b, r)
        assert_close(x, want, f"sum of {n}", rtol=1e-5, atol=2e-5)
        assert_close(h, plain_model.normed(want, w.double(), eps), f"norm of {n}", **tol(adt))
        rows = [7, 0, 3]                                     # picked rows: x stays as it is
        x = x0.clone().cuda()
        h = torch.empty(3, W, dtype=adt, device="cuda")
        ops.sum_norm(x, dev, h=h, rows=i32(rows), **kw)
        assert torch.equal(x.cpu(), x0)
        assert_close(h, plain_model.normed(want, w.double(), eps)[rows], "picked rows", **tol(adt))
    x = x0.clone().cuda()                                    # the sum alone, addends without a scale
    ops.sum_norm(x, [(a.cuda(), None) for a, _ in adds[:2]])
    assert_close(x, total(2, False, False, scaled=False), "sum alone", rtol=1e-5, atol=2e-5)


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("W", [48, 33, 2048, 5120])
def test_token_shift_across_portions_and_slots(adt, W):
    """Steps over three request slots: the row in front of a portion's first row is the request's last row of the step before
    (not the row in front in the batch, which is another request's, nor what the slot's former owner left), a request's first
    token sees zeros, a request may be left out of a step; long steps take several rows a block.  32-bit: the bits of one
    whole pass, whatever the cuts."""
    from tensorline_b200 import ops
    eps = 1e-6
    lens = {"a": 12 + 700, "b": 5, "c": 330, "d": 9}
    slot = {"a": 2, "b": 0, "c": 0, "d": 1}                  # c takes b's slot
    x = {k: rnd(n, W, seed=i, scale=2.0) for i, (k, n) in enumerate(lens.items())}
    add = {k: rnd(n, W, seed=10 + i, dtype=adt) for i, (k, n) in enumerate(lens.items())}
    scale, mu, w = rnd(W, seed=30), torch.rand(W, generator=torch.Generator().manual_seed(31)), rnd(W, seed=32, dtype=adt)
    want = {k: plain_model.shifted(plain_model.normed(x[k].double() + scale.double() * add[k].double(), w.double(), eps), mu.double())
            for k in lens}
    steps = [[("a", 3), ("b", 4), ("d", 1)], [("b", 1), ("d", 2)], [("c", 2), ("a", 1), ("d", 1)], [("a", 1), ("c", 1), ("d", 1)],
             [("d", 4), ("a", 700), ("c", 320)], [("c", 7), ("a", 7)]]
    prev = torch.full((4, W), 77.0, device="cuda")
    at = {k: 0 for k in lens}
    got = {k: [] for k in lens}
    for step in steps:
        frm = dict(at)
        ctx = step_of(step, at, slot)
        xs = torch.cat([x[k][frm[k]:frm[k] + n] for k, n in step]).cuda()
        ad = torch.cat([add[k][frm[k]:frm[k] + n] for k, n in step]).contiguous().cuda()
        keep = xs.clone()
        h = torch.full((ctx.T, W), float("nan"), dtype=adt, device="cuda")
        ops.sum_norm(xs, [(ad, scale.cuda())], w=w.cuda(), eps=eps, h=h, shift=mu.cuda(), prev=prev, ctx=ctx)
        assert torch.equal(xs, keep)
        for (k, n), r in zip(step, ctx.h_q_start):
            got[k].append(h[r:r + n])
    assert at == lens and torch.equal(prev[3].cpu(), torch.full((W,), 77.0))
    for k in lens:
        g = torch.cat(got[k])
        assert_close(g, want[k], f"request {k}", **(dict(rtol=2e-5, atol=4e-5) if adt == torch.float32 else BF16))
        ctx = step_of([(k, lens[k])], {k: 0}, slot)
        h = torch.empty(lens[k], W, dtype=adt, device="cuda")
        ops.sum_norm(x[k].cuda(), [(add[k].cuda(), scale.cuda())], w=w.cuda(), eps=eps, h=h, shift=mu.cuda(), prev=torch.zeros(4, W, device="cuda"),
                     ctx=ctx)
        assert torch.equal(h, g), f"request {k}: the cuts show"
    wrong = plain_model.normed(x["a"].double() + scale.double() * add["a"].double(), w.double(), eps)
    assert float((wrong - want["a"]).abs().max()) > 0.1, "a shift that is left out must show"


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("H,d,dv", [(3, 7, 5), (2, 32, 16), (1, 40, 33), (2, 128, 64), (1, 200, 24), (4, 64, 256), (2, 256, 70), (3, 128, 200)])
def test_memory_with_channel_gates(H, d, dv, chunked):
    """The recurrence of HGRN2 over portions, single tokens and slots that change their owner; the state starts at zero.  In order
    (single tokens by the step kernel): the bits of one whole pass whatever the cuts.  `chunked`: portions as chunks side by
    side, in turns with the step kernel for single tokens."""
    from tensorline_b200 import ops
    lens = {"a": 150 + 400, "b": 20, "c": 61 + 128}
    slot = {"a": 1, "b": 0, "c": 0}
    g = torch.Generator().manual_seed(5)
    lower, bias = torch.rand(H * d, generator=g) * 0.95, torch.rand(H * d, generator=g) * 4 - 1
    proj = {k: rnd(n, H * (2 * d + dv), seed=i, scale=1.5) for i, (k, n) in enumerate(lens.items())}

    def plain(p):
        T = p.shape[0]
        p = p.double()
        q = plain_model.silu(p[:, :H * d]).view(T, H, d)
        f = (lower.double() + (1.0 - lower.double()) * plain_model.sig(p[:, H * d:2 * H * d] + bias.double())).view(T, H, d)
        return plain_model.decayed_memory(q, f, p[:, 2 * H * d:].view(T, H, dv)).reshape(T, -1)
    want = {k: plain(p) for k, p in proj.items()}
    per = H * -(-dv // ops.scan_columns()) * ops.scan_state_floats(d, False)
    state = torch.zeros(3, per, device="cuda")
    at = {k: 0 for k in lens}
    got = {k: [] for k in lens}
    steps = [[("a", 17), ("b", 2)], [("b", 1), ("a", 1)], [("b", 17)], [("c", 33), ("a", 2)], [("a", 1), ("c", 1)], [("c", 27), ("a", 129)], [("a", 400), ("c", 128)]]
    for step in steps:
        if step[0][0] == "c" and at["c"] == 0:
            state[slot["c"]].zero_()                          # what the runner does at admission
        frm = dict(at)
        ctx = step_of(step, at, slot)
        p = torch.cat([proj[k][frm[k]:frm[k] + n] for k, n in step]).cuda()
        o = torch.full((ctx.T, H * dv), float("nan"), device="cuda")
        if chunked and not ctx.decode_only:
            ctx.scratch = {}
            ops.channel_scan(p, 0, H * d, 2 * H * d, H, d, dv, state, ctx, o, lower.cuda(), bias.cuda())
        else:
            ops.linear_scan(p, 0, H * d, 2 * H * d, H, d, dv, state, ctx.q_start, ctx.slots, ctx.pos, o, B=ctx.B, lower=lower.cuda(),
                            bias=bias.cuda(), single_tokens=ctx.decode_only)
        for (k, n), r in zip(step, ctx.h_q_start):
            got[k].append(o[r:r + n])
    assert at == lens
    for k in lens:
        top = float(want[k].abs().max())
        assert_close(torch.cat(got[k]), want[k], f"request {k}", rtol=2e-5, atol=3e-5 * max(1.0, top))
        ctx = step_of([(k, lens[k])], {k: 0}, slot)
        o = torch.empty(lens[k], H * dv, device="cuda")
        ops.linear_scan(proj[k].cuda(), 0, H * d, 2 * H * d, H, d, dv, torch.zeros(3, per, device="cuda"), ctx.q_start, ctx.slots, ctx.pos, o,
                        B=1, lower=lower.cuda(), bias=bias.cuda())
        assert chunked or torch.equal(o, torch.cat(got[k])), f"request {k}: the cuts show"
    lost = plain(proj["a"][17:])                              # a state that is lost at a cut shows long after it
    assert float((lost[5] - want["a"][22]).abs().max()) > 1e-3


def _mixed_rows(q, k, v, pos_q, scale, mix):
    """q [n, nq, d] at positions pos_q over k, v [len, nkv, d]."""
    n, nq, d = q.shape
    g = nq // k.shape[1]
    out = torch.empty(n, nq, v.shape[2], dtype=F64)
    for i, p in enumerate(pos_q):
        P = torch.stack([torch.softmax((k[:p + 1, h // g] @ q[i, h]) * scale, 0) for h in range(nq)])
        M = mix @ P
        for h in range(nq):
            out[i, h] = M[h] @ v[:p + 1, h // g]
    return out


MIX_CASES = [  # nq, nkv, d, page, context lengths before the step, tokens in the step
    (4, 2, 64, 4, [0, 5, 31], [9, 1, 2]),
    (6, 6, 64, 16, [0, 130], [70, 3]),
    (17, 1, 64, 8, [300, 0, 63, 64], [1, 1, 1, 1]),            # single tokens; at a tile's last key and at the next one's first
    (16, 4, 128, 32, [511, 512, 1399], [1, 1, 1]),             # ranges of keys that end at a block's edge and one behind it
    (20, 4, 128, 16, [100, 0, 517], [200, 129, 128]),          # portions of more than one row tile, of exactly one
    (3, 1, 192, 64, [15, 0], [17, 140]),
    (5, 1, 256, 16, [257, 40], [1, 66]),
    (33, 3, 64, 16, [90, 2], [5, 1]),                          # eleven heads a group, three groups of sixteen in the mix
    (1, 1, 64, 16, [0, 700], [1, 40]),
    (64, 8, 64, 16, [200, 0], [1, 33]),
    (12, 4, 64, 2, [70], [3]),
    (32, 32, 128, 16, [2300, 64], [1, 1]),
]


@pytest.mark.parametrize("case", MIX_CASES, ids=[f"q{c[0]}kv{c[1]}d{c[2]}p{c[3]}n{len(c[4])}x{max(c[5])}" for c in MIX_CASES])
@pytest.mark.parametrize("kernel", ["exact_f32", "exact_bf16", "prompt_bf16", "decode_bf16", "step_bf16"])
def test_attention_with_mixed_weights(case, kernel):
    """Attention whose heads' weights are mixed, over scattered pages, against the plain formula.  The first key of the first
    request carries a score that stands out for one head only, so that the others see it through the mix alone."""
    from tensorline_b200 import ops, ops_attention_mix as om, ops_gemm
    nq, nkv, d, ps, ctx_lens, step_lens = case
    if kernel == "decode_bf16" and max(step_lens) > 1:
        pytest.skip("the decode kernels take single tokens")
    adt = torch.float32 if kernel == "exact_f32" else torch.bfloat16
    scale = 1.3 * d ** -0.5
    B = len(ctx_lens)
    max_pages = max(-(-(c + n) // ps) for c, n in zip(ctx_lens, step_lens)) + 3
    num_pages = max(300, B * max_pages)
    kps = torch.full((num_pages + 1, nkv, ps, d), 37.0, dtype=adt)
    vps = torch.full_like(kps, -53.0)
    mix = (torch.eye(nq) + rnd(nq, nq, seed=9, scale=1.2 * nq ** -0.5)).to(torch.bfloat16)
    rows, qs, want, pos_all, slot_all = [], [], [], [], []
    for b in range(B):
        n = ctx_lens[b] + step_lens[b]
        k, v = rnd(n, nkv, d, seed=20 + b, dtype=adt), rnd(n, nkv, d, seed=40 + b, dtype=adt)
        q = rnd(step_lens[b], nq, d, seed=60 + b, scale=1.5, dtype=adt)
        if b == 0:                                           # the last query's head 0 finds the first key, no other head does
            q[-1] *= 0.2
            q[-1, 0] = 0.0; q[-1, 0, 0] = 8.0
            k[0, 0] = 0.0; k[0, 0, 0] = 9.0
        gen = torch.Generator().manual_seed(100 + b)
        mine = (torch.randperm(num_pages // B, generator=gen)[:-(-n // ps)] * B + b).tolist()
        for i in range(n):
            kps[mine[i // ps], :, i % ps] = k[i]
            vps[mine[i // ps], :, i % ps] = v[i]
        rows.append(mine)
        pq = list(range(ctx_lens[b], n))
        want.append(_mixed_rows(q.double(), k.double(), v.double(), pq, scale, mix.double()))
        if b == 0:
            alone = _mixed_rows(q[-1:].double(), k.double(), v.double(), pq[-1:], scale, torch.eye(nq, dtype=F64))
            assert nq == 1 or float((alone - want[0][-1:]).abs().max()) > 0.05, "a mix that is left out must show"
        qs.append(q)
        pos_all += pq
        slot_all += [b] * step_lens[b]
    q_all = torch.cat(qs).reshape(-1, nq * d)
    T = q_all.shape[0]
    qkv = torch.zeros(T, (nq + 2 * nkv) * d, dtype=adt)
    qkv[:, :nq * d] = q_all
    qkv = qkv.cuda()
    out = torch.full((T, nq * d), float("nan"), dtype=adt, device="cuda")
    table = table_tensor(rows, max_pages, num_pages)
    kd, vd = kps.cuda(), vps.cuda()
    q_start = [0]
    for n in step_lens:
        q_start.append(q_start[-1] + n)
    pad = om.pad_mix(mix.cuda())
    where = (i32(q_start), i32(ctx_lens), i32(list(range(B))))
    W = torch.cat(want)
    if kernel.startswith("exact"):
        ops.attn_mixed_tokenwise(qkv, qkv.shape[1], out, kd, vd, table, ps, i32(pos_all), i32(slot_all), nq, nkv, d, scale, mix.float().cuda())
    elif kernel == "prompt_bf16":                              # everything through the prompt kernels, single tokens too
        for units in (1000, 3):
            launches = [tuple(torch.from_numpy(a).cuda() for a in l) for l in om.row_tiles(q_start, ctx_lens, range(B), units)]
            out.fill_(float("nan"))
            om.prefill(qkv, out, kd, vd, table, ps, *where, launches, nq, nkv, d, scale, pad)
            assert_close(out.view(T, nq, d), W, f"{kernel}, {units} tiles a launch", **BF16)
    elif kernel == "decode_bf16":
        span = max(c + 1 for c in ctx_lens)
        for rng in (64, 192, 512):
            out.fill_(float("nan"))
            om.decode(qkv, out, kd, vd, table, ps, *where, B, nq, nkv, d, scale, pad, rng, -(-span // rng))
            assert_close(out.view(T, nq, d), W, f"{kernel}, ranges of {rng}", **BF16)
        for clusters in (1, 3, 8, 16):                         # one launch; contexts shorter than a block's run leave blocks without keys
            out.fill_(float("nan"))
            if om.decode_cluster(qkv, out, kd, vd, table, ps, *where, B, nq, nkv, d, scale, pad, clusters, span + 70):
                assert_close(out.view(T, nq, d), W, f"{kernel}, clusters of {clusters}", **BF16)
            else:
                assert nq * span > 8192 * clusters
    else:                                                      # the step's own choice of kernels
        ctx = SimpleNamespace(B=B, T=T, decode_only=all(n == 1 for n in step_lens), page_size=ps, q_start=where[0], start_pos=where[1],
                              slots=where[2], h_q_start=q_start, h_start_pos=list(ctx_lens), h_slots=list(range(B)), graph_max_ctx=0,
                              max_ctx=max(c + n for c, n in zip(ctx_lens, step_lens)), scratch={})
        om.attend(qkv, out, ctx, kd, vd, table, nq, nkv, d, scale, pad)
    ops_gemm.check_status()
    assert_close(out.view(T, nq, d), W, kernel, **tol(adt))


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("pairing", ["half", "interleaved"])
@pytest.mark.parametrize("weighted", [True, False])
@pytest.mark.parametrize("dk,d,rot", [(24, 32, 12), (128, 128, 64), (64, 64, 64), (16, 64, 0), (7, 8, 6)])
def test_normed_heads_rotated_in_part_and_written_to_their_pages(adt, pairing, weighted, dk, d, rot):
    """q and k heads of `dk` dimensions padded to `d`, normed without a rounding in front of the weight, the first `rot` turned;
    v passes.  Without weights the norm behind the rotation is the same thing."""
    from tensorline_b200 import ops
    if adt == torch.bfloat16 and d % 16:
        pytest.skip("the bfloat16 engine's heads are multiples of 16")
    nq, nkv, ps, eps = 3, 2, 4, 1e-5
    pos, slot = [0, 1, 2, 9, 10, 3, 40], [0, 0, 0, 1, 1, 0, 2]
    T = len(pos)
    raw = torch.zeros(T, nq + 2 * nkv, d)
    raw[..., :dk] = rnd(T, nq + 2 * nkv, dk, seed=1, scale=2.0)
    raw = raw.to(adt)
    wq, wk = rnd(d, seed=2), rnd(d, seed=3)
    if not weighted:
        wq = wk = torch.ones(d)
    base = 700.0
    inv = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
    table = table_tensor([[3, 5], [1, 1, 7], [2] * 11], 12, 8)
    kp, vp = torch.zeros(9, nkv, ps, d, dtype=adt, device="cuda"), torch.zeros(9, nkv, ps, d, dtype=adt, device="cuda")
    qkv = raw.reshape(T, -1).clone().cuda()
    ops.rope_kv_write(qkv, None, i32(pos), i32(slot), table, ps, inv.cuda(), rot, nq, nkv, d, kp, vp, pairing=pairing, q_norm=wq.cuda(),
                      k_norm=wk.cuda(), norm_eps=eps, norm_dim=dk, norm_cast=False)
    for t in range(T):
        def turned(x):
            return x if rot == 0 else plain_model.turn(torch.cat([torch.zeros(pos[t], *x.shape, dtype=F64), x[None]]), {"base": base, "dims": rot},
                                                       "half" if pairing == "half" else "pairs")[-1]
        r = raw[t].double()[:, :dk]
        if weighted:
            q, k = turned(plain_model.normed(r[:nq], wq.double()[:dk], eps)), turned(plain_model.normed(r[nq:nq + nkv], wk.double()[:dk], eps))
        else:
            q, k = plain_model.unit(turned(r[:nq]), eps), plain_model.unit(turned(r[nq:nq + nkv]), eps)
        pg, off = int(table[slot[t], pos[t] // ps]), pos[t] % ps
        assert_close(qkv[t].view(-1, d)[:nq, :dk], q, f"q of token {t}", **tol(adt))
        assert_close(kp[pg, :, off, :dk], k, f"k of token {t}", **tol(adt))
        assert_close(vp[pg, :, off, :dk], r[nq + nkv:], f"v of token {t}", **tol(adt))
        assert float(kp[pg, :, off, dk:].abs().sum()) == 0.0 and float(qkv[t].view(-1, d)[:nq, dk:].abs().sum()) == 0.0


@pytest.mark.parametrize("adt", DT)
@pytest.mark.parametrize("T,H,I", [(3, 40, 24), (5, 2048, 4096), (16, 4096, 2048), (48, 2048, 6016), (300, 256, 512), (1536, 2048, 4096)])
def test_feed_forward_with_the_square_of_relu(adt, T, H, I):
    from tensorline_b200.parts import FEED_FORWARDS, PartSpec, Runtime
    from tensorline_b200.parts.linear import resolve
    if adt == torch.float32 and T * H * I > 1 << 26:
        pytest.skip("the 32-bit product at these sizes is tested elsewhere")
    ff = FEED_FORWARDS.build(PartSpec("plain_mlp", {"hidden": H, "intermediate": I, "names": {"up": "up", "down": "down"}}),
                             Runtime(torch.device("cuda"), adt))
    w = {"m.up": rnd(I, H, seed=1, scale=H ** -0.5, dtype=torch.bfloat16).cuda(), "m.down": rnd(H, I, seed=2, scale=I ** -0.5, dtype=torch.bfloat16).cuda()}
    ff.bind(w, "m")
    h = rnd(T, H, seed=3, dtype=adt).cuda()
    got = resolve(ff.forward(h, None))
    want = torch.clamp(h.double() @ w["m.up"].double().T, min=0.0) ** 2 @ w["m.down"].double().T
    assert_close(got, want, "feed-forward", **(dict(rtol=1e-4, atol=1e-4) if adt == torch.float32 else dict(rtol=0.03, atol=0.05)))


# ------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module", params=["Z1", "Z2"])
def model(request, tmp_path_factory):
    name = request.param
    folder = write_tiny_zosurax(name, tmp_path_factory.mktemp(f"tiny_{name}"))
    plain = PlainZosurax(folder)
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


def test_the_model_is_chosen_by_its_configuration_and_every_layer_run_matches(model):
    """The residual stream after every layer run, with what still waits to be added, 32-bit engine against the plain model."""
    from tensorline_b200.parts.linear import StreamSum
    from tensorline_b200.replay import TraceSession, make_runner
    runner, cfg = make_runner(model["folder"], "float32", 256, page_size=model["page"], max_live=2)
    assert type(cfg).__name__ == "ZosuraxConfig" and cfg.to_json_dict() == CONFIGS[model["name"]]
    seen = []
    for blk in runner.model.blocks:
        def fwd(x, pending, ctx, cache, orig=blk.forward):
            out = orig(x, pending, ctx, cache)
            y = x.clone()
            StreamSum.of(out).write_into(y)
            seen.append(y.double().cpu())
            return out
        blk.forward = fwd
    toks = model["reqs"]["r2"]
    TraceSession(runner).run_step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": []}], "end": ["a"]})
    want = []
    logits_of(model["plain"], toks, want)
    assert len(seen) == len(want) == len(plain_model.order(CONFIGS[model["name"]]))
    for i, (g, w) in enumerate(zip(seen, want)):
        assert_close(g, w, f"stream after layer run {i}", rtol=5e-5, atol=F32_ATOL * max(1.0, float(w.abs().max())))


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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(model, dtype):
    """A one-token prompt, then 150 tokens decoded one by one: the memories, the shifted rows and the pages are carried through
    150 launches of every pass."""
    toks = random_tokens(model["vocab"], 151, seed=7)
    want = logits_of(model["plain"], toks)
    steps = [{"step": i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
    steps[-1]["end"] = ["x"]
    m2 = dict(model, reqs={"x": toks}, want={"x": want})
    got = replay(m2, dtype, steps, max_tokens=160)
    check(m2, dtype, got, "token by token")
    assert sorted(p for _, p in got) == list(range(151))


def test_mistakes_planted_in_the_plain_model_show(model, monkeypatch):
    """What the comparisons above would not let pass: the plain model with a mechanism left out or turned around gives logits
    far beyond the bounds."""
    toks = model["reqs"]["r3"]
    right = model["want"]["r3"]

    def gap():
        return float((logits_of(model["plain"], toks) - right).abs().max()) / float(right.abs().max())
    assert gap() == 0.0
    order = plain_model.order
    plants = {
        "no token shift": ("shifted", lambda h, mu: h),
        "a shift towards the next token": ("shifted", lambda h, mu: h + (torch.cat([h[1:], torch.zeros_like(h[:1])]) - h) * mu),
        "weights not mixed": ("mixed_weights", lambda P, talk: P),
        "the mix transposed": ("mixed_weights", lambda P, talk: torch.einsum("ba,btj->atj", talk, P)),
        "no lower bound": ("forget_gates", lambda h, w, c: plain_model.sig(h @ w["f"].T + w["f.b"]).view(h.shape[0], c["heads"], c["dim"])),
        "the embedding not added again": ("order", lambda c: [(i, r if not r else 0) for i, r in order(c)]),
        "relu not squared": ("relu_squared_ff", lambda h, w: torch.clamp(h @ w["up"].T, min=0.0) @ w["down"].T),
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


@pytest.mark.parametrize("name", ["Z3", "Z4", "Z5", "Z6"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_further_shapes_of_the_design(name, dtype, tmp_path):
    """No loop and nothing rotated with single heads; a loop over layers without a feed-forward, odd head sizes and a width that
    is a multiple of nothing; seventeen mixed heads and a loop of one pass; sizes that the tensor-core kernels take, with prompts
    of hundreds of tokens: whole requests, changing portions and a small pool against the plain model."""
    folder = write_tiny_zosurax(name, tmp_path / name)
    plain = PlainZosurax(folder)
    V = CONFIGS[name]["vocab"]
    lengths = [290, 3, 400, 130] if name == "Z6" else [3, 50, 1, 81, 33]
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
    if model["name"] != "Z1":
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
    assert sorted(p.name for p in out.iterdir()) == ["0.f32", "1.f32", "2.f32", "3.f32"]
    V = model["vocab"]
    got = {n: torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, V).astype(np.float64)) for n in range(4)}
    assert [got[n].shape[0] for n in range(4)] == [3, 1, 1, 1]
    wa, wb, wc = model["want"]["r3"], model["want"]["r4"], model["want"]["r2"]
    for row, ref in ((got[0][0], wa[0]), (got[0][1], wa[29]), (got[0][2], wb[1]), (got[1][0], wb[-1]), (got[2][0], wc[-1]), (got[3][0], wa[-1])):
        assert float((row - ref).abs().max()) <= F32_ATOL * max(1.0, float(ref.abs().max()))
