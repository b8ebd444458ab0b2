"""Paged grouped-query attention for layer-listed models.  Optional parts: heads' scores mixed before the softmax, chunked
visibility, a sliding window that keeps a sequence's first keys, a sink (score zero, or a learned one per head), rotary positions on
queries and keys, a sigmoid gate per head or per element on the output; biases and norms of query and key heads (each head alone, or
all at once; ``prepare_heads``, ``csrc/head_prep.cu``).

Cache rows, and one query row per CTA for decode and short pieces: ``csrc/talking_attn.cu`` (plain bf16 heads on the tensor
cores, ``csrc/gqa_rows.cuh``); tensor-core flash attention for long pieces of prompts, over mixed queries
(``csrc/talking_prefill.cu``) or plain heads (``csrc/gqa_prefill.cu``).
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import torch

from . import _ext
from .conv import rotate_ref
from .residual import _DT, _i


@dataclass
class TalkParams:
    """One layer's attention.  Head widths are padded to multiples of 8 with zero channels (dim_p, vdim_p)."""
    heads: int
    kv_heads: int
    dim_p: int
    vdim_p: int
    scale: float
    chunk: int = 0                           # keys are seen from the query's own chunk on; 0 = every earlier key
    sink: bool = False                       # one added to the softmax denominator
    talk: Optional[torch.Tensor] = None      # [heads, heads] fp32: score_h <- sum_g talk[h, g] score_g; None = no mixing
    window: int = 0                          # the last so many positions are seen, the query's own among them; 0 = all
    keep: int = 0                            # with a window: so many first positions stay visible
    out_scale: float = 1.0                   # factor of the output
    sinks: Optional[torch.Tensor] = None     # [heads] fp32: exp of it added to the softmax denominator (``sink`` is set then)
    gate_all: bool = False                   # the output gate has a column per element, not per head
    shared_row: bool = False                 # one key head whose first vdim_p channels are the values too (a cached latent)

    def __post_init__(self):
        if self.sinks is not None:
            self.sink = True

    @property
    def kv_row(self) -> int:
        return self.dim_p if self.shared_row else self.kv_heads * (self.dim_p + self.vdim_p)

    @property
    def v_col0(self) -> int:
        """First value column of a cached row."""
        return 0 if self.shared_row else self.kv_heads * self.dim_p

    @property
    def gate_cols(self) -> int:
        return self.vdim_p if self.gate_all else 1

    def first(self, pos: int) -> int:
        """First position that a query at ``pos`` sees, kept first ones aside."""
        first = pos - pos % self.chunk if self.chunk else 0
        return max(first, pos + 1 - self.window) if self.window else first

    def most_keys(self, keys: int) -> int:
        """An upper bound of the keys a query sees out of ``keys``."""
        for n in (self.chunk, self.window + self.keep if self.window else 0):
            keys = min(keys, n) if n else keys
        return keys


def kv_write(kv: torch.Tensor, slots: torch.Tensor, cache: torch.Tensor, p: Optional[TalkParams] = None,
             rope: Optional[torch.Tensor] = None) -> None:
    """cache[slot] = kv (fp32 columns: keys of all heads, values of all heads); cache [pages, page, row] (strided pages);
    slots [T] int64, < 0 writes nothing.  ``rope`` [T, dims] (``conv.Rotary.table``) turns the keys of ``p``'s heads."""
    P, page, row = cache.shape
    if not kv.is_cuda:
        if rope is not None:
            n = p.kv_heads * p.dim_p
            k = rotate_ref(kv[:, :n].view(-1, p.kv_heads, p.dim_p), rope).reshape(-1, n)
            kv = torch.cat([k, kv[:, n:row]], 1)
        live = slots >= 0
        s = slots[live]
        cache[s // page, s % page] = kv[live, :row].to(cache.dtype)
        return
    assert kv.dtype == torch.float32 and kv.stride(1) == 1 and cache.stride(1) == row and cache.stride(2) == 1
    assert slots.dtype == torch.int64
    rc = _ext.lib().bg_talk_kv_write(_i(_DT[cache.dtype]), _ext.ptr(kv), _i(kv.stride(0)), _ext.ptr(slots), _ext.ptr(cache),
                                     ctypes.c_longlong(cache.stride(0)), _i(page), _i(row), _i(kv.shape[0]), _ext.ptr(rope),
                                     _i(rope.shape[1] // 2 if rope is not None else 0), _i(p.kv_heads if p else 1),
                                     _i(p.dim_p if p else 0), _ext.stream())
    _ext.check(rc, "bg_talk_kv_write")


@dataclass
class HeadPrep:
    """What happens to a layer's heads between their projections and the scores, rotary positions aside.  Vectors are fp32, padded
    like the heads with zeros."""
    dim: int                                 # real width of query and key heads
    eps: float = 1e-6
    bias: Optional[torch.Tensor] = None      # [heads * dim_p + kv_row], columns as projected: queries, keys, values
    q_norm: Optional[torch.Tensor] = None    # [dim_p] gains of the RMS norms of query and key heads, or with ``whole`` [heads * dim_p]
    k_norm: Optional[torch.Tensor] = None
    interleaved: bool = False                # rotary pairs (2 i, 2 i + 1), else (i, i + dims / 2)
    whole: bool = False                      # one norm over all query heads of a token, one over all key heads


def prepare_heads(z: torch.Tensor, slots: torch.Tensor, cache: torch.Tensor, p: TalkParams, h: HeadPrep,
                  rope: Optional[torch.Tensor] = None, write_q: bool = True, operand: bool = False) -> Optional[torch.Tensor]:
    """z [T, >= heads * dim_p + kv_row] fp32 columns of queries, keys and values: bias, norms and rotary positions; keys and values
    go to cache[slot] (slots [T] int64, < 0: nowhere), queries back to z (``write_q``) and, with ``operand``, into the prompt
    kernel's bf16 queries, which are returned."""
    H, G, dp = p.heads, p.kv_heads, p.dim_p
    P, page, row = cache.shape
    if not z.is_cuda:
        n = H * dp
        x = z[:, :n + row] if h.bias is None else z[:, :n + row] + h.bias

        def turn(t, heads, w):
            if w is not None and h.whole:
                t = t / torch.sqrt((t * t).sum(-1, keepdim=True) / (heads * h.dim) + h.eps) * w
            t = t.reshape(-1, heads, dp)
            if w is not None and not h.whole:
                t = t / torch.sqrt((t * t).sum(-1, keepdim=True) / h.dim + h.eps) * w
            return rotate_ref(t, rope, h.interleaved).reshape(-1, heads * dp)
        kv_write(torch.cat([turn(x[:, n:n + G * dp], G, h.k_norm), x[:, n + G * dp:]], 1), slots, cache)
        z[:, :n] = turn(x[:, :n], H, h.q_norm)
        return None
    T = z.shape[0]
    assert z.dtype == torch.float32 and z.stride(1) == 1 and z.shape[1] >= H * dp + row and row == p.kv_row
    assert cache.stride(1) == row and cache.stride(2) == 1 and slots.dtype == torch.int64 and slots.shape[0] == T
    assert rope is None or (rope.is_contiguous() and rope.shape[0] == T)
    assert h.bias is None or h.bias.shape[0] == H * dp + row
    assert all(w is None or w.shape[0] == (n * dp if h.whole else dp) for w, n in ((h.q_norm, H), (h.k_norm, G)))
    kc = -(-dp // 64) * 64
    qf = torch.empty(T, H, kc, dtype=torch.bfloat16, device=z.device) if operand else None
    rc = _ext.lib().bg_head_prep(
        _i(_DT[cache.dtype]), _ext.ptr(z), _i(z.stride(0)), _ext.ptr(h.bias), _ext.ptr(h.q_norm), _ext.ptr(h.k_norm),
        _i(h.whole), ctypes.c_float(h.eps), _i(h.dim), _ext.ptr(rope), _i(rope.shape[1] // 2 if rope is not None else 0), _i(h.interleaved),
        _ext.ptr(slots), _ext.ptr(cache), ctypes.c_longlong(cache.stride(0)), _i(page), _i(row), _i(write_q), _ext.ptr(qf), _i(kc),
        ctypes.c_float(p.scale), _i(T), _i(H), _i(G), _i(dp), _i(p.vdim_p), _ext.stream())
    if rc == -3:
        raise _ext.KernelError(f"prepare_heads: {H} + {G} heads of {dp} are more than one norm takes (a token's row in shared memory)")
    _ext.check(rc, "bg_head_prep")
    return qf


def _rows_ref(q, p: TalkParams, cache, block_table, lens, out, row_seq, rope, gate):
    H, G, d, dv = p.heads, p.kv_heads, p.dim_p, p.vdim_p
    q = rotate_ref(q[:, : H * d].float().view(-1, H, d), rope).reshape(-1, H * d)
    rep = H // G
    page = cache.shape[1]
    for t in range(q.shape[0]):
        L = int(lens[t])
        out[t, : H * dv] = 0
        if L <= 0:
            continue
        pos = torch.arange(L)
        pos = pos[(pos >= p.first(L - 1)) | (pos < p.keep)]
        bt = block_table[int(row_seq[t]) if row_seq is not None else t].long()
        rows = cache[bt[pos // page], pos % page].float()
        k = rows[:, : G * d].view(-1, G, d).repeat_interleave(rep, 1)
        v = rows[:, p.v_col0:p.v_col0 + G * dv].view(-1, G, dv).repeat_interleave(rep, 1)
        s = torch.einsum("hd,jhd->hj", q[t, : H * d].view(H, d).float(), k) * p.scale
        if p.talk is not None:
            s = p.talk @ s
        m = s.amax(-1, keepdim=True)
        sink = None if not p.sink else torch.zeros(H, 1) if p.sinks is None else p.sinks.view(H, 1)
        if p.sink:
            m = torch.maximum(m, sink)
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True) + (torch.exp(sink - m) if p.sink else 0)
        o = torch.einsum("hj,jhv->hv", e / den, v) * p.out_scale
        if gate is not None:
            o = o * torch.sigmoid(gate[t, :H * p.gate_cols].float()).view(H, p.gate_cols)
        out[t, : H * dv] = o.reshape(-1).to(out.dtype)


def rows_on_tensor_cores(p: TalkParams, dtype: torch.dtype) -> bool:
    """The row kernel of plain bf16 heads up to 128 wide (``csrc/gqa_rows.cuh``)."""
    return dtype == torch.bfloat16 and p.talk is None and not p.shared_row and p.dim_p <= 128 and p.vdim_p <= 128


def _ranges(ctas: int, keys: int, sms: int) -> int:
    """Key ranges per row for ``gqa_rows.cuh``: rounds of CTAs over the SMs (two fit an SM), of which each takes as long as its
    keys and some 256 more to start and end."""
    return min(range(1, max(1, min(16, keys // 64)) + 1), key=lambda s: math.ceil(ctas * s / (2 * sms)) * (keys / s + 256))


def _splits(rows: int, keys: int, sms: int) -> int:
    """Key ranges per row: whole rounds of CTAs over the SMs (two fit an SM), each range a few 32-key tiles long."""
    slots, tiles = 2 * sms, max(1, -(-keys // 32))
    best, score = 1, -1.0
    for s in range(1, max(1, min(16, tiles // 4)) + 1):
        rounds = rows * s / slots
        v = rounds / math.ceil(rounds) - 0.004 * s             # share of the slots that work, less the merge
        if v > score:
            best, score = s, v
    return best


def attend_rows(q: torch.Tensor, p: TalkParams, cache: torch.Tensor, block_table: torch.Tensor, lens: torch.Tensor,
                out: torch.Tensor, row_seq: Optional[torch.Tensor] = None, row_ids: Optional[torch.Tensor] = None,
                num_splits: int = 0, rope: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None) -> None:
    """q [T, >= H * dim_p] fp32 -> out [T, >= H * vdim_p] (operand dtype, a column view is fine).  ``lens`` [T] int32 =
    position + 1 of each row (0: no query, zero output); ``row_seq`` [R] block-table row of each query row (None: row i);
    ``row_ids`` [R] the rows of q to compute (None: all).  ``rope`` [T, dims] turns the queries, ``gate`` [T, >= H (* vdim_p)] fp32 scales
    each head's output, or with ``gate_all`` each element, by its sigmoid.  The keys are in the cache already."""
    if not q.is_cuda:
        if row_ids is not None:
            raise NotImplementedError("row subsets are a device path")
        return _rows_ref(q, p, cache, block_table, lens, out, row_seq, rope, gate)
    P, page, row = cache.shape
    R = q.shape[0] if row_ids is None else row_ids.shape[0]
    assert q.dtype == torch.float32 and q.stride(1) == 1 and out.stride(1) == 1 and out.dtype == cache.dtype
    assert lens.dtype == torch.int32 and block_table.dtype == torch.int32 and row == p.kv_row and cache.stride(1) == row
    assert gate is None or (gate.dtype == torch.float32 and gate.stride(1) == 1 and gate.shape[1] >= p.heads * p.gate_cols)
    assert p.sinks is None or (p.sinks.dtype == torch.float32 and p.sinks.shape[0] == p.heads)
    for t in (row_seq, row_ids):
        assert t is None or t.dtype == torch.int32
    H = p.heads
    if num_splits <= 0:
        keys = block_table.shape[1] * page
        if rows_on_tensor_cores(p, cache.dtype):
            heads = p.kv_heads * -(-(H // p.kv_heads) // 16)              # CTAs of a row and key range
            num_splits = _ranges(R * heads, p.most_keys(keys), _ext.num_sms(q.device))
        else:
            num_splits = _splits(R, p.most_keys(keys), _ext.num_sms(q.device))
    po = pml = None
    if num_splits > 1:
        po = torch.empty(R * num_splits * H * p.vdim_p, dtype=torch.float32, device=q.device)
        pml = torch.empty(R * num_splits * H * 2, dtype=torch.float32, device=q.device)
    rc = _ext.lib().bg_talk_rows(
        _i(_DT[cache.dtype]), _ext.ptr(q), _i(q.stride(0)), _ext.ptr(p.talk), _ext.ptr(cache),
        ctypes.c_longlong(cache.stride(0)), _i(page), _i(row), _ext.ptr(block_table), _i(block_table.stride(0)),
        _ext.ptr(row_seq), _ext.ptr(row_ids), _ext.ptr(lens), _ext.ptr(out), _i(out.stride(0)), _ext.ptr(po),
        _ext.ptr(pml), _i(R), _i(H), _i(p.kv_heads), _i(p.dim_p), _i(p.vdim_p), _i(p.chunk), _i(p.window),
        _i(p.keep), _i(p.sink), ctypes.c_float(p.scale), ctypes.c_float(p.out_scale), _i(num_splits), _ext.ptr(rope), _i(rope.shape[1] // 2 if rope is not None else 0),
        _ext.ptr(gate), _i(gate.stride(0) if gate is not None else 0), _i(p.gate_cols), _ext.ptr(p.sinks), _i(p.v_col0),
        _ext.stream())
    if rc in (-1, -3):
        raise _ext.KernelError(f"attend_rows: heads {H}/{p.kv_heads}, widths {p.dim_p}/{p.vdim_p} are outside the kernel's "
                               "contract (shared memory of one CTA, 2,048 head-column items)")
    _ext.check(rc, "bg_talk_rows", kernels=2 if num_splits > 1 else 1)


PREFILL_MIN_TOKENS = 32      # pieces at least this long go to the tensor-core kernel
_TILE = 128                  # queries of one CTA
_FOLD_ROWS = 8192            # rows whose mixed queries are held at a time


def prefill_supported(p: TalkParams, dtype: torch.dtype, page: int) -> bool:
    """The tensor-core kernels read bf16 pages and keep one head's value columns in TMEM (plain heads: its queries in shared
    memory)."""
    return dtype == torch.bfloat16 and not p.shared_row and p.vdim_p <= 256 and page >= 16 and (p.talk is not None or p.dim_p <= 256)


def prefill_work(cu: Sequence[int], ctx: Sequence[int], chunk: int, min_tokens: int = 1,
                 window: int = 0) -> List[Tuple[int, int, int, int]]:
    """Tiles (first query row, queries, sequence, position of the first query) of every piece of at least ``min_tokens``
    tokens, the tiles with the most visible keys first."""
    out = []
    for i in range(len(cu) - 1):
        a, b = int(cu[i]), int(cu[i + 1])
        if b - a < min_tokens:
            continue
        for q0 in range(a, b, _TILE):
            out.append((q0, min(_TILE, b - q0), i, int(ctx[i]) + q0 - a))
    def first(pos):
        return max(pos // chunk * chunk if chunk else 0, pos + 1 - window if window else 0)
    out.sort(key=lambda w: -(w[3] + w[1] - first(w[3])))
    return out


def work_blocks(work: List[Tuple[int, int, int, int]], rows: int, device) -> List[Tuple[int, int, torch.Tensor]]:
    """Tiles grouped by ranges of query rows: (first row, rows, [n, 4] int32 tiles).  Bounds the mixed queries' memory."""
    blocks: dict = {}
    for w in work:
        blocks.setdefault(w[0] // _FOLD_ROWS, []).append(w)
    out = []
    for b in sorted(blocks):
        lo = b * _FOLD_ROWS
        hi = min(rows, max(w[0] + w[1] for w in blocks[b]))
        out.append((lo, hi - lo, torch.tensor(blocks[b], dtype=torch.int32, device=device)))
    return out


def attend_prefill(q: torch.Tensor, p: TalkParams, cache: torch.Tensor, block_table: torch.Tensor, out: torch.Tensor,
                   blocks: List[Tuple[int, int, torch.Tensor]], rope: Optional[torch.Tensor] = None,
                   gate: Optional[torch.Tensor] = None, operand: Optional[torch.Tensor] = None) -> None:
    """CUDA, bf16 cache: q [T, >= H * dim_p] fp32 -> out [T, >= H * vdim_p] for the rows covered by ``blocks``
    (``work_blocks``); ``rope`` and ``gate`` as for ``attend_rows``.  The keys of every query are in the cache already.
    ``operand``: the queries as ``prepare_heads`` returns them, instead of q and ``rope``.

    Mixed heads contract over a token's whole key block, plain heads over their own key head's columns."""
    P, page, row = cache.shape
    H, G = p.heads, p.kv_heads
    plain = p.talk is None
    assert plain or (rope is None and gate is None and not p.window and p.out_scale == 1.0 and p.sinks is None), \
        "mixed heads with rotary queries, windows, output gates, scales or learned sinks are not covered"
    assert gate is None or (gate.dtype == torch.float32 and gate.stride(1) == 1 and gate.shape[1] >= H * p.gate_cols)
    kc = -(-(p.dim_p if plain else G * p.dim_p) // 64) * 64
    assert q.dtype == torch.float32 and q.stride(1) == 1 and out.stride(1) == 1 and out.dtype == cache.dtype == torch.bfloat16
    assert row == p.kv_row and cache.stride(1) == row and block_table.dtype == torch.int32
    assert operand is None or (plain and rope is None and operand.is_contiguous() and operand.shape == (q.shape[0], H, kc))
    L = _ext.lib()
    for lo, n, work in blocks:
        qf = torch.empty(n, H, kc, dtype=torch.bfloat16, device=q.device) if operand is None else operand[lo:lo + n]
        if operand is not None:
            rc = 0
        elif plain:
            rc = L.bg_gqa_prompt_queries(_ext.ptr(q[lo:]), _i(q.stride(0)), _ext.ptr(rope[lo:] if rope is not None else None),
                                _i(rope.shape[1] // 2 if rope is not None else 0), _ext.ptr(qf), _i(n), _i(H), _i(p.dim_p),
                                _i(kc), ctypes.c_float(p.scale), _ext.stream())
        else:
            rc = L.bg_talk_fold(_ext.ptr(q[lo:]), _i(q.stride(0)), _ext.ptr(p.talk), _ext.ptr(qf), _i(n), _i(H), _i(G),
                                _i(p.dim_p), _i(kc), ctypes.c_float(p.scale), _ext.stream())
        if operand is None:
            _ext.check(rc, "bg_gqa_prompt_queries" if plain else "bg_talk_fold")
        where = (_ext.ptr(qf), _ext.ptr(cache), ctypes.c_longlong(cache.stride(0)), _i(P), _i(page), _i(row),
                 _ext.ptr(block_table), _i(block_table.stride(0)), _i(block_table.shape[1]), _ext.ptr(work), _i(work.shape[0]),
                 _i(n), _i(lo), _ext.ptr(out), _i(out.stride(0)), _i(H), _i(G), _i(p.dim_p), _i(p.vdim_p), _i(kc), _i(p.chunk),
                 _i(p.sink))
        status = _ext.ptr(_ext.status_word(q.device))
        if plain:
            rc = L.bg_gqa_prompt(*where, _i(p.window), _i(p.keep), ctypes.c_float(p.out_scale), _ext.ptr(gate),
                                 _i(gate.stride(0) if gate is not None else 0), _i(p.gate_cols), _ext.ptr(p.sinks), status,
                                 _ext.stream())
        else:
            rc = L.bg_talk_prefill(*where, status, _ext.stream())
        _ext.check(rc, "bg_gqa_prompt" if plain else "bg_talk_prefill")
