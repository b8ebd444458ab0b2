"""Causal depthwise convolution over time with per-sequence history, and rotary tables (``csrc/causal_conv.cu``)."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import torch

from . import _ext
from .residual import _DT, _i

CONV_KINDS = {"residual": 0, "silu": 1}


def causal_conv(x: torch.Tensor, w: torch.Tensor, hist: torch.Tensor, slots: torch.Tensor, out: torch.Tensor, kind: str,
                cu: Optional[torch.Tensor] = None, cu_host: Optional[Sequence[int]] = None,
                row_seq: Optional[torch.Tensor] = None, has_initial: Optional[torch.Tensor] = None) -> torch.Tensor:
    """y_t = sum_j w[j] x_(t - taps + 1 + j) per channel; inputs before a piece come from ``hist``, zeros before a sequence.

    x [T, >= C] fp32; w [taps, C] fp32 (C a multiple of 4); hist [slots, (taps - 1) * C] fp32 (a strided view of the state
    pool): the last inputs of a sequence, oldest first, updated here.  ``kind``: "residual" out = x + y, "silu" out = silu(y).
    ``out`` [T, >= C]: columns past C become zero.  Without ``cu`` every row is the next token of sequence ``slots[row]``
    (slot < 0: no history, none kept); with it, rows cu[s] .. cu[s + 1] are a piece of sequence s and ``row_seq`` [T] int32
    maps rows to sequences."""
    taps, C = w.shape
    if not x.is_cuda:
        return _conv_ref(x, w, hist, slots, out, kind, cu_host, has_initial)
    assert x.dtype == w.dtype == hist.dtype == torch.float32 and x.stride(1) == out.stride(1) == hist.stride(1) == 1
    assert x.shape[1] >= C and out.shape[0] == x.shape[0] and out.shape[1] >= C and hist.shape[1] == (taps - 1) * C
    assert (row_seq is None or row_seq.shape[0] == x.shape[0]) and (cu is None or cu.shape[0] == slots.shape[0] + 1)
    assert w.is_contiguous() and slots.dtype == torch.int32 and (row_seq is None or row_seq.dtype == torch.int32)
    rc = _ext.lib().bg_causal_conv(
        _i(_DT[out.dtype]), _i(CONV_KINDS[kind]), _ext.ptr(x), _i(x.stride(0)), _ext.ptr(w), _ext.ptr(hist),
        ctypes.c_longlong(hist.stride(0)), _ext.ptr(slots), _ext.ptr(cu), _ext.ptr(row_seq), _ext.ptr(has_initial),
        _ext.ptr(out), _i(out.stride(0)), _i(x.shape[0]), _i(slots.shape[0]), _i(C), _i(out.shape[1]), _i(taps), _ext.stream())
    _ext.check(rc, "bg_causal_conv", kernels=2 if cu is not None and taps > 1 else 1)
    return out


def _conv_ref(x, w, hist, slots, out, kind, cu_host, has_initial):
    taps, C = w.shape
    nseq = len(slots)
    bounds = list(range(nseq + 1)) if cu_host is None else list(cu_host)
    out.zero_()
    for s in range(nseq):
        a, b, slot = bounds[s], bounds[s + 1], int(slots[s])
        if b <= a:
            continue
        old = torch.zeros(taps - 1, C)
        if slot >= 0 and (has_initial is None or int(has_initial[s])):
            old = hist[slot].reshape(taps - 1, C).clone()
        full = torch.cat([old, x[a:b, :C].float()], 0)
        y = sum(full[j:j + b - a] * w[j] for j in range(taps))
        y = x[a:b, :C] + y if kind == "residual" else torch.nn.functional.silu(y)
        out[a:b, :C] = y.to(out.dtype)
        if slot >= 0 and taps > 1:
            hist[slot] = full[full.shape[0] - (taps - 1):].reshape(-1)
    return out


@dataclass
class Rotary:
    """Rotary positions of the leading ``dims`` dimensions, angle position * base^(-2 i / dims) of pair i: dimensions
    (i, i + dims / 2), or (2 i, 2 i + 1) when ``interleaved``.  ``yarn`` (factor, original positions, fast, slow): frequencies of
    pairs that turn fewer than ``slow`` times within the original positions are divided by ``factor``, those of pairs that turn
    more than ``fast`` times stay, with a ramp between them, and cosines and sines grow by 0.1 ln(factor) + 1."""
    dims: int
    base: float
    turns: torch.Tensor = None             # [dims / 2] float64: turns per position
    interleaved: bool = False
    yarn: Tuple[float, ...] = ()
    mult: float = 1.0                      # of cosines and sines

    @classmethod
    def make(cls, dims: int, base: float, device, interleaved: bool = False, yarn: Tuple[float, ...] = ()) -> Optional["Rotary"]:
        if not dims:
            return None
        i = torch.arange(dims // 2, dtype=torch.float64)
        f, mult = torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / dims), 1.0
        if yarn:
            factor, original, fast, slow = yarn

            def pair_of(turns):            # the pair that makes this many turns within the original positions
                return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
            lo, hi = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
            ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
            f, mult = f / factor * ramp + f * (1 - ramp), 0.1 * math.log(factor) + 1.0
        return cls(dims, base, (f / (2 * math.pi)).to(device), interleaved, tuple(yarn), mult)

    @property
    def key(self) -> Tuple:
        """Rotaries with equal keys have equal tables."""
        return self.dims, self.base, self.yarn

    def table(self, lens: torch.Tensor) -> torch.Tensor:
        """[T, dims] fp32 of the positions ``lens`` - 1: cosines, then sines.  The turn is reduced before it is rounded to
        32 bits, so far positions keep exact angles."""
        if not lens.is_cuda:
            a = (lens.double() - 1).unsqueeze(1) * self.turns * (2 * math.pi)
            return (torch.cat([a.cos(), a.sin()], 1) * self.mult).float()
        out = torch.empty(lens.shape[0], self.dims, dtype=torch.float32, device=lens.device)
        rc = _ext.lib().bg_rope_table(_ext.ptr(lens), _ext.ptr(self.turns), _ext.ptr(out), _i(lens.shape[0]),
                                      _i(self.dims // 2), ctypes.c_float(self.mult), _ext.stream())
        _ext.check(rc, "bg_rope_table")
        return out


def rotate_ref(x: torch.Tensor, rope: Optional[torch.Tensor], interleaved: bool = False) -> torch.Tensor:
    """x [T, heads, d] turned by ``rope`` (``Rotary.table``)."""
    if rope is None:
        return x
    half = rope.shape[1] // 2
    c, s = rope[:, None, :half], rope[:, None, half:]
    if interleaved:
        u, v = x[..., 0:2 * half:2], x[..., 1:2 * half:2]
        return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., 2 * half:]], -1)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)
