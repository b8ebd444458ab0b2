"""Attention over a cached latent ("multi-head latent attention") for layer-listed models: the cache holds one row per token, a normed
latent and a rotated key part that all heads share; keys and values are linear in the latent.  Any head count and widths, a sliding
window, a learned sink per head.

Two forms.  *Latent space* (decode, short pieces of prompts, the fp32 form): a query goes through its head's key projection once, is
scored against whole cached rows (``csrc/latent_rows.cuh``, ``csrc/talking_attn.cu``), and the weighted latent goes through the value
projection.  *Expanded* (longer pieces, bf16): cached rows of the visible pages are multiplied out to keys and values of all heads,
page by page, and the prompt kernel of plain heads runs on those (``csrc/gqa_prefill.cu``).

Layouts: query heads [rotated | rest], cache rows [latent | rotated], every part padded with zero channels to a multiple of 8.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from . import _ext, gemm, talking
from .conv import rotate_ref
from .residual import _DT, _i


@dataclass
class LatentParams:
    heads: int
    dim_p: int                               # unrotated query / key channels of a head, as stored
    rot_dim: int
    rot_p: int
    rank: int                                # latent width
    rank_p: int
    vdim_p: int
    q_rank: int                              # width of the latent that queries go through
    scale: float
    eps: float
    window: int                              # the last so many positions are seen, the query's own among them; 0 = all
    sinks: torch.Tensor                      # [heads] fp32
    q_norm: torch.Tensor                     # [q_rank rounded up to 8] fp32 gain
    c_norm: Optional[torch.Tensor]           # [rank_p] fp32 gain; None: the latents are another layer's
    w_uq: torch.Tensor                       # [heads * (rot_p + dim_p), operand width] query projection
    w_uk: torch.Tensor                       # [heads, rank_p, dim_p rounded up to the operand's step] key projection, transposed per head
    w_uv: torch.Tensor                       # [heads, vdim_p, rank_p rounded up] value projection
    w_up: Optional[torch.Tensor] = None      # [heads * (rot_p + dim_p) + heads * vdim_p, row rounded up]: cached row -> keys, values

    @property
    def row(self) -> int:
        return self.rank_p + self.rot_p

    @property
    def expanded(self) -> talking.TalkParams:
        """Plain heads over expanded keys and values."""
        return talking.TalkParams(self.heads, self.heads, self.rot_p + self.dim_p, self.vdim_p, self.scale, window=self.window, sinks=self.sinks)

    def shared(self, h0: int, n: int) -> talking.TalkParams:
        """Heads h0 .. h0 + n over whole cached rows."""
        return talking.TalkParams(n, 1, self.row, self.rank_p, self.scale, window=self.window, sinks=self.sinks[h0:h0 + n], shared_row=True)


def prepare(z: torch.Tensor, cols: Tuple[int, Optional[int], Optional[int]], slots: torch.Tensor, cache: torch.Tensor, p: LatentParams,
            rope: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """z [T, *] fp32 projections; ``cols``: first columns of the query latent, the latent and the rotated key part (None: nothing is
    cached).  Writes cache[slot] (slots [T] int64, < 0: nowhere) and returns the operand [T, w_uq's width] of the query projection."""
    T, n = z.shape[0], p.w_uq.shape[1]
    q0, c0, r0 = cols
    if not z.is_cuda:
        def normed(x, w, d):
            return x / torch.sqrt((x * x).sum(-1, keepdim=True) / d + p.eps) * w[:d]
        out = torch.zeros(T, n, dtype=dtype)
        out[:, :p.q_rank] = normed(z[:, q0:q0 + p.q_rank], p.q_norm, p.q_rank).to(dtype)
        if c0 is not None:
            row = torch.zeros(T, p.row)
            row[:, :p.rank] = normed(z[:, c0:c0 + p.rank], p.c_norm, p.rank)
            row[:, p.rank_p:p.rank_p + p.rot_dim] = rotate_ref(z[:, None, r0:r0 + p.rot_dim], rope)[:, 0]
            talking.kv_write(row, slots, cache)
        return out
    own = c0 is not None
    assert z.dtype == torch.float32 and z.stride(1) == 1 and slots.dtype == torch.int64 and slots.shape[0] == T
    assert p.q_norm.shape[0] >= -(-p.q_rank // 4) * 4 and cache.stride(1) == cache.shape[2] == p.row and cache.dtype == dtype
    assert z.shape[1] >= q0 + p.q_rank and (not own or (z.shape[1] >= max(c0 + p.rank, r0 + p.rot_dim) and p.c_norm.shape[0] >= p.rank_p))
    assert rope.is_contiguous() and rope.shape == (T, p.rot_dim)
    out = torch.empty(T, n, dtype=dtype, device=z.device)
    at = lambda c: ctypes.c_void_p(0 if c is None else z.data_ptr() + 4 * c)      # noqa: E731
    rc = _ext.lib().bg_latent_prep(
        _i(_DT[dtype]), at(q0), at(c0), at(r0), _i(z.stride(0)), _ext.ptr(p.q_norm), _ext.ptr(p.c_norm), _i(p.q_rank), _i(p.rank),
        _i(p.rot_dim // 2), _i(n), _i(p.rank_p), _i(p.rot_p), _ext.ptr(rope), _ext.ptr(out), _ext.ptr(slots), _ext.ptr(cache),
        ctypes.c_longlong(cache.stride(0)), _i(cache.shape[1]), _i(p.row), ctypes.c_float(p.eps), _i(T), _ext.stream())
    _ext.check(rc, "bg_latent_prep")
    return out


def head_product(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """out[:, h] = a[:, h] @ w[h]^T: a [T, H, K] contiguous, w [H, N, K rounded up: zero columns], out [T, H, N] with unit inner stride.
    bf16 (``csrc/head_gemm.cu``: a head's last step may run on into the next head's numbers, which meet the zeros) or fp32."""
    T, H, K = a.shape
    N, Kp = w.shape[1:]
    if not a.is_cuda:
        out.copy_(torch.einsum("thk,hnk->thn", a.float(), w[..., :K].float()).to(out.dtype))
        return
    assert a.is_contiguous() and w.is_contiguous() and a.dtype == w.dtype == out.dtype and out.stride(2) == 1 and w.shape[0] == H
    L = _ext.lib()
    if a.dtype == torch.float32:
        rc = L.bg_head_gemm_f32(_ext.ptr(a), _i(H * K), _i(K), _ext.ptr(w), _i(Kp), _ext.ptr(out), _i(out.stride(0)), _i(out.stride(1)), _i(T),
                                _i(H), _i(N), _i(K), _ext.stream())
        _ext.check(rc, "bg_head_gemm_f32")
        return
    rc = L.bg_head_gemm(_ext.ptr(a), ctypes.c_longlong(H * K), _i(K), ctypes.c_longlong(H * K), _ext.ptr(w), _ext.ptr(out),
                        ctypes.c_longlong(out.stride(0)), ctypes.c_longlong(out.stride(1)), _i(T), _i(H), _i(N), _i(Kp),
                        _ext.ptr(_ext.status_word(a.device)), _ext.stream())
    _ext.check(rc, "bg_head_gemm")


def queries(q: torch.Tensor, p: LatentParams, rope: torch.Tensor, rows: Optional[torch.Tensor] = None,
            dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """q [T, heads * (rot_p + dim_p)] fp32 -> queries in latent space [R, heads, row] of ``dtype`` (``rows`` [R] int32: those alone)."""
    H, hw = p.heads, p.rot_p + p.dim_p
    R = q.shape[0] if rows is None else rows.shape[0]
    qa = torch.empty(R, H, p.row, dtype=dtype, device=q.device)
    rest = torch.empty(R, H, p.dim_p, dtype=dtype, device=q.device)
    if not q.is_cuda:
        x = q[:, :H * hw].view(-1, H, hw)
        x, cs = (x, rope) if rows is None else (x[rows.long()], rope[rows.long()])
        qa[..., p.rank_p:] = rotate_ref(x[..., :p.rot_p], cs).to(dtype)
        rest.copy_(x[..., p.rot_p:])
    else:
        assert q.dtype == torch.float32 and q.stride(1) == 1 and q.shape[1] >= H * hw and rope.is_contiguous() and rope.shape[1] == p.rot_dim
        assert rows is None or rows.dtype == torch.int32
        rc = _ext.lib().bg_latent_query(_i(_DT[dtype]), _ext.ptr(q), _i(q.stride(0)), _ext.ptr(rows), _ext.ptr(rope), _i(p.rot_dim // 2),
                                        _ext.ptr(rest), _ext.ptr(qa), _i(R), _i(H), _i(p.rot_p), _i(p.dim_p), _i(p.rank_p), _ext.stream())
        _ext.check(rc, "bg_latent_query")
    head_product(rest, p.w_uk, qa[..., :p.rank_p])
    return qa


def _key_ranges(ctas: int, keys: int, sms: int) -> int:
    """Key ranges per row: rounds of CTAs over the SMs (one fits an SM), of which each takes as long as its keys and some 128 more to
    start and end, and a little more for every range that is merged."""
    return min(range(1, max(1, min(16, keys // 64)) + 1), key=lambda s: math.ceil(ctas * s / sms) * (keys / s + 128) + 4 * s)


def on_tensor_cores(p: LatentParams, dtype: torch.dtype, page: int) -> bool:
    return dtype == torch.bfloat16 and p.row <= 640 and p.rank_p <= 512 and page >= 16


def _heads_at_a_time(p: LatentParams, esize: int) -> int:
    """Heads one CTA of the CUDA-core row kernel takes: items of 4 heads x 4 value columns, queries and one buffer of keys in shared memory."""
    n = p.heads
    while n > 1 and (-(-n // 4) * (p.rank_p // 4) > 2048 or 4 * n * (p.row + 72) + 32 * (p.row * esize + 16) > 200 * 1024):
        n = -(-n // 2)
    return n


def attend(qa: torch.Tensor, p: LatentParams, cache: torch.Tensor, block_table: torch.Tensor, lens: torch.Tensor,
           row_seq: Optional[torch.Tensor] = None, num_splits: int = 0) -> torch.Tensor:
    """Queries in latent space [R, heads, row] -> weighted latents [R, heads, rank_p].  ``lens`` [R] int32 = position + 1 (0: zero output),
    ``row_seq`` [R] int32 block-table row (None: row i).  The keys are in the cache already."""
    R, H, row = qa.shape
    out = torch.empty(R, H, p.rank_p, dtype=qa.dtype, device=qa.device)
    flat = out.view(R, H * p.rank_p)
    if qa.is_cuda and on_tensor_cores(p, qa.dtype, cache.shape[1]):
        assert qa.is_contiguous() and row == p.row == cache.shape[2] == cache.stride(1) and cache.dtype == qa.dtype
        assert lens.dtype == torch.int32 and lens.shape[0] == R and block_table.dtype == torch.int32
        assert row_seq is None or (row_seq.dtype == torch.int32 and row_seq.shape[0] == R)
        if num_splits <= 0:
            keys = block_table.shape[1] * cache.shape[1]
            num_splits = _key_ranges(R * -(-H // 32), min(keys, p.window) if p.window else keys, _ext.num_sms(qa.device))
        po = pml = None
        if num_splits > 1:
            po = torch.empty(R * num_splits * H * p.rank_p, dtype=torch.float32, device=qa.device)
            pml = torch.empty(R * num_splits * H * 2, dtype=torch.float32, device=qa.device)
        rc = _ext.lib().bg_latent_rows(
            _ext.ptr(qa), _ext.ptr(cache), ctypes.c_longlong(cache.stride(0)), _i(cache.shape[0]), _i(cache.shape[1]), _i(row),
            _ext.ptr(block_table), _i(block_table.stride(0)), _ext.ptr(row_seq), _ext.ptr(lens), _ext.ptr(out), _i(flat.stride(0)), _ext.ptr(po), _ext.ptr(pml),
            _i(R), _i(H), _i(p.rank_p), _i(p.window), _ext.ptr(p.sinks), ctypes.c_float(p.scale), _i(num_splits),
            _ext.ptr(_ext.status_word(qa.device)), _ext.stream())
        _ext.check(rc, "bg_latent_rows", kernels=2 if num_splits > 1 else 1)
        return out
    q = qa.view(R, H * row).float()
    n = _heads_at_a_time(p, qa.element_size()) if qa.is_cuda else H
    for h0 in range(0, H, n):
        m = min(n, H - h0)
        talking.attend_rows(q[:, h0 * row:(h0 + m) * row], p.shared(h0, m), cache, block_table, lens, flat[:, h0 * p.rank_p:(h0 + m) * p.rank_p],
                            row_seq, num_splits=num_splits)
    return out


# ---------------------------------------------------------------- expanded form
def prompt_supported(p: LatentParams, dtype: torch.dtype, page: int) -> bool:
    return p.w_up is not None and talking.prefill_supported(p.expanded, dtype, page)


@dataclass
class Expansion:
    """Which cached pages a group of prompt pieces sees, and where their expanded rows lie."""
    pages: torch.Tensor                      # [n, 2] int32: block-table row, page of the sequence
    table: torch.Tensor                      # [sequences, most pages] int32: page of the expanded rows
    blocks: List                             # ``talking.work_blocks``, positions counted from a sequence's first expanded page


EXPAND_TOKENS = 65536      # expanded rows held at a time, unless one piece sees more


def expansions(cu: List[int], ctx: List[int], window: int, page: int, device) -> List[Expansion]:
    """Groups of the pieces cu[i] .. cu[i + 1] (positions from ctx[i] on) that the expanded form takes, those of at least
    ``talking.PREFILL_MIN_TOKENS`` tokens."""
    out, group, held = [], [], 0

    def close():
        nonlocal group, held
        if not group:
            return
        pages, rows, work = [], {}, []
        for i, lo, hi in group:
            rows[i] = list(range(len(pages), len(pages) + hi - lo))
            pages += [(i, k) for k in range(lo, hi)]
            at = talking.prefill_work([cu[i], cu[i + 1]], [ctx[i] - lo * page], 0, 1, window)
            work += [(w[0], w[1], i, w[3]) for w in at]
        work.sort(key=lambda w: -(w[3] + w[1] - max(0, w[3] + 1 - window if window else 0)))
        table = torch.zeros(len(cu) - 1, max(map(len, rows.values())), dtype=torch.int32)
        for i, r in rows.items():
            table[i, :len(r)] = torch.tensor(r, dtype=torch.int32)
            table[i, len(r):] = r[-1]
        out.append(Expansion(torch.tensor(pages, dtype=torch.int32, device=device), table.to(device),
                             talking.work_blocks(work, cu[-1], device)))
        group, held = [], 0
    for i in range(len(cu) - 1):
        n = cu[i + 1] - cu[i]
        if n < talking.PREFILL_MIN_TOKENS:
            continue
        lo = max(0, ctx[i] + 1 - window if window else 0) // page
        hi = -(-(ctx[i] + n) // page)
        if group and held + (hi - lo) * page > EXPAND_TOKENS:
            close()
        group.append((i, lo, hi))
        held += (hi - lo) * page
    close()
    return out


def attend_prompt(q: torch.Tensor, p: LatentParams, cache: torch.Tensor, block_table: torch.Tensor, rope: torch.Tensor, out: torch.Tensor,
                  groups: List[Expansion]) -> None:
    """CUDA, bf16: q [T, heads * (rot_p + dim_p)] fp32 (not turned yet) -> out [T, >= heads * vdim_p] for the rows the groups cover."""
    page, cols = cache.shape[1], p.w_up.shape[1]
    t = p.expanded
    assert cache.dtype == torch.bfloat16 and cache.stride(1) == cache.shape[2] == p.row and block_table.dtype == torch.int32
    for g in groups:
        n = g.pages.shape[0]
        rows = torch.empty(n * page, cols, dtype=cache.dtype, device=cache.device)
        rc = _ext.lib().bg_latent_gather(_ext.ptr(cache), ctypes.c_longlong(cache.stride(0)), _ext.ptr(block_table), _i(block_table.stride(0)),
                                         _ext.ptr(g.pages), _i(n), _ext.ptr(rows), _i(page), _i(p.row), _i(cols), _ext.stream())
        _ext.check(rc, "bg_latent_gather")
        up = gemm.bf16_gemm(rows, p.w_up).view(n, page, t.kv_row)
        talking.attend_prefill(q, t, up, g.table, out, g.blocks, rope=rope)
