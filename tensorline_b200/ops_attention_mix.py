"""Launchers of the attention kernels whose heads' softmax weights are mixed (`csrc/attn_mix.cu`, bfloat16), built per head size.

A step's single tokens go to the decode kernels (scores, mix and values, sum over the ranges of keys), its prompt portions to
the prompt kernels (scores, mix, values over a scratch of score tiles).  What these kernels do not take (`takes`) runs in the
exact-order kernel."""
from __future__ import annotations

import ctypes
import os

import numpy as np
import torch

from .csrc.build import load_library
from . import ops
from .ops import KernelError, _check, _ptr, _stream

_P, _I, _F = ctypes.c_void_p, ctypes.c_int, ctypes.c_float
_libs: dict = {}

HEAD_MULTIPLE = 64                  # head sizes the kernels are compiled for: multiples of this up to 256
MAX_HEADS = 64
ROW_TILE, KEY_TILE = 128, 64
SCRATCH_BYTES = int(os.environ.get("TENSORLINE_B200_MIX_SCRATCH_MB", 512)) << 20      # score and weight tiles of one launch, at most
DECODE_MAX_RANGE = 256              # keys a block of the kernels over ranges, at most (they take up to 512; longer was slower)


def lib(head_dim: int):
    l = _libs.get(head_dim)
    if l is None:
        if head_dim % HEAD_MULTIPLE or not HEAD_MULTIPLE <= head_dim <= 256:
            raise KernelError(f"head_dim {head_dim}: the mixed-head attention kernels take multiples of {HEAD_MULTIPLE} up to 256")
        l = load_library(f"tl_attn_mix_hd{head_dim}", ["attn_mix.cu"], {"HEAD_DIM": head_dim})
        l.tl_mix_prefill.argtypes = [_P, _I, _P, _P, _P, _P, _I, _I, _P, _P, _P, _I, _I, _F, _P, _I, _P, _I, _P, _I, _P, _P, _P, _P, _P, _I,
                                     _P, _I, _I, _P, _P]
        l.tl_mix_prefill.restype = ctypes.c_int
        l.tl_mix_decode.argtypes = [_P, _I, _P, _P, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _F, _I, _I, _P, _P, _P, _P, _I, _I, _I, _P, _P]
        l.tl_mix_decode.restype = ctypes.c_int
        l.tl_mix_decode_cluster.argtypes = [_P, _I, _P, _P, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _F, _I, _I, _P, _I, _I, _I, _P, _P]
        l.tl_mix_decode_cluster.restype = ctypes.c_int
        if l.tl_mix_max_parts() != MAX_PARTS or any(l.tl_mix_parts(n) != parts_of(n) for n in (1, 8, 9, 128, 129, 1000, 5000)):
            raise KernelError("the mixed-head attention library cuts key tiles into other runs than its launcher")
        _libs[head_dim] = l
    return l


MAX_PARTS = 16


def parts_of(n_kt: int) -> int:
    """Runs a row tile of n_kt key tiles is cut into for the scores kernel: of eight key tiles, or sixteen runs of more."""
    size = -(-n_kt // MAX_PARTS) if n_kt > 8 * MAX_PARTS else 8
    return -(-n_kt // size)


def takes(nq: int, d: int, page_size: int, mix_dtype) -> bool:
    """Whether the bfloat16 kernels take these sizes; the mix has to be exact in bfloat16."""
    return (d % HEAD_MULTIPLE == 0 and d <= 256 and nq <= MAX_HEADS and 2 <= page_size <= KEY_TILE and page_size & (page_size - 1) == 0
            and mix_dtype == torch.bfloat16)


def pad_mix(mix: torch.Tensor) -> torch.Tensor:
    """[H, H] -> bfloat16 [hp, hp], H padded with zeros to a multiple of 16: what the kernels read."""
    H = mix.shape[0]
    hp = -(-H // 16) * 16
    out = torch.zeros((hp, hp), dtype=torch.bfloat16, device=mix.device)
    out[:H, :H] = mix
    return out


def row_tiles(h_q_start, h_start_pos, requests, max_units: int):
    """Row tiles of 128 tokens of the given requests, the one that reads the most keys first, cut into launches of at most
    `max_units` (row tile x key tile) pairs (a single row tile may exceed it): [(tiles int32 [n, 4] rows (request, tile, first
    unit, key tiles), parts int32 [m, 2] (row tile, run of its key tiles), unit -> row tile int32)], numpy."""
    tiles = []
    for b in requests:
        n = h_q_start[b + 1] - h_q_start[b]
        for t in range(-(-n // ROW_TILE)):
            last = h_start_pos[b] + min(n, (t + 1) * ROW_TILE) - 1
            tiles.append((last // KEY_TILE + 1, b, t))
    tiles.sort(key=lambda x: (-x[0], x[1], x[2]))
    out, cur, units = [], [], 0

    def close():
        nonlocal cur, units
        if cur:
            parts = [(i, p) for i, c in enumerate(cur) for p in range(parts_of(c[3]))]
            out.append((np.array(cur, dtype=np.int32), np.array(parts, dtype=np.int32),
                        np.repeat(np.arange(len(cur), dtype=np.int32), [c[3] for c in cur])))
        cur, units = [], 0

    for kt, b, t in tiles:
        if cur and units + kt > max_units:
            close()
        cur.append((b, t, units, kt))
        units += kt
    close()
    return out


def prefill(q, out, k_pages, v_pages, table, page_size, q_start, start_pos, slots, launches, nq, nkv, d, scale, mix, lse=None) -> None:
    """The prompt kernels over `launches` ([(tiles, parts, unit -> tile)] device tensors, see `row_tiles`)."""
    from .ops_gemm import status_word
    T = out.shape[0]
    most = max(u.numel() for _, _, u in launches)
    scores = torch.empty(most * nq * ROW_TILE * KEY_TILE, dtype=torch.float32, device=q.device)
    mixed = torch.empty(most * nq * ROW_TILE * KEY_TILE, dtype=torch.bfloat16, device=q.device)
    lse = torch.empty((T, nq), dtype=torch.float32, device=q.device) if lse is None else lse
    part_ml = torch.empty((T, nq, MAX_PARTS, 2), dtype=torch.float32, device=q.device)
    for tiles, parts, unit_tile in launches:
        _check(lib(d).tl_mix_prefill(_ptr(q), q.shape[1], _ptr(out), _ptr(k_pages), _ptr(v_pages), _ptr(table), table.shape[1], page_size,
                                     _ptr(q_start), _ptr(start_pos), _ptr(slots), nq, nkv, float(scale), _ptr(tiles), tiles.shape[0],
                                     _ptr(parts), parts.shape[0], _ptr(unit_tile), unit_tile.numel(), _ptr(scores), _ptr(part_ml), _ptr(lse),
                                     _ptr(mixed), _ptr(mix), mix.shape[0], _ptr(status_word(q.device)), table.shape[0], k_pages.shape[0],
                                     ops.fault_words(q.device), _stream()), "mix_prefill", launches=4)


def plan_ranges(n: int, nkv: int, group: int, d: int, span: int, sms: int | None = None) -> tuple:
    """(keys a range, ranges) of a decode step of n requests that read at most `span` keys: enough ranges that the blocks of
    the second kernel fill the GPU once, none under 64 keys."""
    sms = sms or ops.num_sms()
    blocks = n * -(-nkv * d // 8 // 64) * -(-group // 8)
    tiles = max(1, -(-span // 64))
    splits = min(tiles, max(1, sms // max(1, blocks)))
    rng = min(DECODE_MAX_RANGE, -(-tiles // splits) * 64)
    return rng, -(-tiles * 64 // rng)


def decode(q, out, k_pages, v_pages, table, page_size, rows, start_pos, slots, n, nq, nkv, d, scale, mix, rng, splits) -> None:
    """The decode kernels: request i's query is row rows[i] of q (its result row of out), at position start_pos[i]."""
    dev = q.device
    scores = torch.empty((n, nq, splits * rng), dtype=torch.float32, device=dev)
    ml = torch.empty((n, splits, nq, 2), dtype=torch.float32, device=dev)
    part = torch.empty((n, splits, nq, d), dtype=torch.float32, device=dev) if splits > 1 else None
    _check(lib(d).tl_mix_decode(_ptr(q), q.shape[1], _ptr(out), _ptr(k_pages), _ptr(v_pages), _ptr(table), table.shape[1], page_size,
                                _ptr(rows), _ptr(start_pos), _ptr(slots), n, nq, nkv, float(scale), rng, splits, _ptr(scores), _ptr(ml),
                                _ptr(part), _ptr(mix), mix.shape[0], table.shape[0], k_pages.shape[0], ops.fault_words(dev), _stream()),
           "mix_decode", launches=3 if splits > 1 else 2)


def plan_cluster(n: int, nq: int, nkv: int, d: int, span: int, sms: int | None = None) -> int:
    """Blocks a request of the one-launch decode kernel, or 0 where the kernels over ranges serve better: long contexts and many KV
    heads, which want every SM.  The two estimates (microseconds) are fits of measurements at 148 SMs: the cluster kernel 12 and
    0.04 a key a block of 512 values (a third more where every head has keys of its own), the others 24 and the cache's bytes at
    4.5 TB/s; n = 8, 4 KV heads of 128, 2,304 keys: 23 against 30; 64 requests: 61 against 107; 8 requests of 16 KV heads of 64 at
    4,096 keys: 62 against 43."""
    sms = sms or ops.num_sms()
    # as many blocks as run at once, one an SM: six clusters of sixteen fit this GPU, twelve of eight (measured, 148 SMs)
    clusters = next((c for c, most in ((16, sms // 24), (8, sms // 12), (4, sms // 4), (2, sms // 2)) if n <= most), 1)
    keys = -(-span // clusters)
    one = 12.0 + 0.04 * keys * nkv * d / 512 * (1.3 if nkv == nq else 1.0)
    three = 24.0 + 4.0 * n * span * nkv * d / 4.5e6
    return clusters if keys * nq <= 36 * 1024 and one <= 1.2 * three else 0


def decode_cluster(q, out, k_pages, v_pages, table, page_size, rows, start_pos, slots, n, nq, nkv, d, scale, mix, clusters, span) -> bool:
    """`decode` in one launch, `clusters` blocks a request; `span`: the most keys a request reads.  False: nothing launched (the
    keys' weights do not fit the shared memory)."""
    most = -(-(-(-span // clusters)) // 32) * 32
    rc = lib(d).tl_mix_decode_cluster(_ptr(q), q.shape[1], _ptr(out), _ptr(k_pages), _ptr(v_pages), _ptr(table), table.shape[1], page_size,
                                      _ptr(rows), _ptr(start_pos), _ptr(slots), n, nq, nkv, float(scale), clusters, most, _ptr(mix),
                                      mix.shape[0], table.shape[0], k_pages.shape[0], ops.fault_words(q.device), _stream())
    if rc == 2:
        return False
    _check(rc, "mix_decode+cluster")
    return True


def _decode(q, out, k_pages, v_pages, table, page_size, rows, start_pos, slots, n, nq, nkv, d, scale, mix, span) -> None:
    args = (q, out, k_pages, v_pages, table, page_size, rows, start_pos, slots, n, nq, nkv, d, scale, mix)
    clusters = plan_cluster(n, nq, nkv, d, span)
    if not (CLUSTER and clusters and decode_cluster(*args, clusters, span)):
        decode(*args, *plan_ranges(n, nkv, nq // nkv, d, span))


CLUSTER = os.environ.get("TENSORLINE_B200_MIX_CLUSTER", "1") != "0"      # 0: the kernels over ranges only (A/B timing)


def attend(qkv, o, ctx, k_pages, v_pages, table, nq, nkv, d, scale, mix) -> None:
    """A step's attention: single tokens through the decode kernels, portions through the prompt kernels."""
    if qkv.dtype != torch.bfloat16 or k_pages.dtype != torch.bfloat16 or mix.dtype != torch.bfloat16:
        raise KernelError("mixed-head attention: bfloat16 tensors only")
    args = (k_pages, v_pages, table, ctx.page_size)
    if ctx.decode_only:
        _decode(qkv, o, *args, ctx.q_start, ctx.start_pos, ctx.slots, ctx.B, nq, nkv, d, scale, mix, ctx.graph_max_ctx or ctx.max_ctx)
        return
    units = max(1, SCRATCH_BYTES // (nq * ROW_TILE * KEY_TILE * 6))
    key = ("mix_tiles", units)
    if key not in ctx.scratch:                           # one description a step, for every layer
        ones = [b for b in range(ctx.B) if ctx.h_q_start[b + 1] - ctx.h_q_start[b] == 1]
        rest = [b for b in range(ctx.B) if ctx.h_q_start[b + 1] - ctx.h_q_start[b] > 1]
        launches = [tuple(torch.from_numpy(a).to(qkv.device, non_blocking=True) for a in l)
                    for l in row_tiles(ctx.h_q_start, ctx.h_start_pos, rest, units)]
        singles = None
        if ones:
            packed = torch.tensor([[ctx.h_q_start[b] for b in ones], [ctx.h_start_pos[b] for b in ones], [ctx.h_slots[b] for b in ones]],
                                  dtype=torch.int32).to(qkv.device, non_blocking=True)
            singles = (packed, len(ones), max(ctx.h_start_pos[b] for b in ones) + 1)
        ctx.scratch[key] = (launches, singles)
    launches, singles = ctx.scratch[key]
    if singles:
        packed, n, span = singles
        _decode(qkv, o, *args, packed[0], packed[1], packed[2], n, nq, nkv, d, scale, mix, span)
    if launches:
        prefill(qkv, o, *args, ctx.q_start, ctx.start_pos, ctx.slots, launches, nq, nkv, d, scale, mix)
