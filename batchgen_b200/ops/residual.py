"""Row operators of models with an fp32 residual stream: residual sum + RMS norm (with the embedding or the sublayers'
outputs folded in), the same step of blocks with a norm before and after each sublayer and of hyper-connected residual streams,
gated activations, operand casts, expert-row gather.

CUDA tensors go to ``csrc/residual.cu``; CPU tensors to plain fp32 torch.  Operand dtype (norm output, activations) is
bf16, or fp32 for the 32-bit form of a model.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _ext

_DT = {torch.bfloat16: 0, torch.float32: 1}
GLU_KINDS = {"gelu_tanh": 0, "swiglu_oai": 1, "silu": 2, "relu2": 3}        # relu2: no gate
CAST_KINDS = {"none": 0, "tanh": 1, "relu2": 2}


def _i(v) -> ctypes.c_int:
    return ctypes.c_int(int(v))


def pad_to(n: int, m: int) -> int:
    return -(-n // m) * m


def residual_norm(x: torch.Tensor, w: torch.Tensor, eps: float, width: int, out_cols: int, dtype: torch.dtype,
                  add: Optional[torch.Tensor] = None, routed: Optional[torch.Tensor] = None,
                  pos: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None,
                  embed: Optional[torch.Tensor] = None, embed_scale: float = 1.0, rows: Optional[torch.Tensor] = None,
                  keep: bool = True) -> torch.Tensor:
    """x [T, >= width] fp32 (+= ``add`` [T, width] fp32, += sum_k routed[pos[t, k]]; or = embed[ids] * embed_scale), then
    y = rmsnorm(x) * w as [R, out_cols] of ``dtype`` with zero columns past ``width``.  ``rows`` (int64) picks rows of x;
    ``keep=False`` leaves x as it was (the last norm of a step)."""
    R = x.shape[0] if rows is None else rows.shape[0]
    if not x.is_cuda:
        r = rows.long() if rows is not None else torch.arange(x.shape[0])
        cur = x[r, :width].clone()
        if ids is not None:
            cur = embed[ids[r].long()].float() * embed_scale
        if add is not None:
            cur = cur + add[r, :width]
        if routed is not None:
            p = pos[r].long()
            g = routed[p.clamp_min(0), :width] * (p >= 0).unsqueeze(-1)
            cur = cur + g.sum(1)
        if keep:
            x[r, :width] = cur
        y = torch.zeros(R, out_cols, dtype=dtype)
        y[:, :width] = (cur / torch.sqrt((cur * cur).mean(-1, keepdim=True) + eps) * w).to(dtype)
        return y
    y = torch.empty(R, out_cols, dtype=dtype, device=x.device)
    for t in (add, routed):
        assert t is None or (t.dtype == torch.float32 and t.stride(1) == 1)
    assert x.dtype == torch.float32 and w.dtype == torch.float32 and (embed is None or embed.dtype == dtype)
    assert (ids is None or ids.dtype == torch.int32) and (pos is None or (pos.dtype == torch.int32 and pos.is_contiguous()))
    assert rows is None or rows.dtype == torch.int64
    rc = _ext.lib().bg_residual_norm(
        _i(_DT[dtype]), _ext.ptr(x), _i(x.stride(0)), _ext.ptr(rows), _ext.ptr(ids), _ext.ptr(embed),
        _i(embed.stride(0) if embed is not None else 0), ctypes.c_float(embed_scale),
        _i(embed.shape[0] if embed is not None else 0), _ext.ptr(add), _i(add.stride(0) if add is not None else 0),
        _ext.ptr(routed), _i(routed.stride(0) if routed is not None else 0), _ext.ptr(pos),
        _i(pos.shape[1] if pos is not None else 0), _ext.ptr(w), _ext.ptr(y), _i(out_cols), _i(R), _i(width),
        ctypes.c_float(eps), _i(keep), _ext.stream())
    _ext.check(rc, "bg_residual_norm")
    return y


def _glu_ref(g: torch.Tensor, u: torch.Tensor, kind: str, limit: float) -> torch.Tensor:
    if kind == "gelu_tanh":
        return 0.5 * g * (1 + torch.tanh(math.sqrt(2 / math.pi) * (g + 0.044715 * g ** 3))) * u
    if kind == "silu":
        return g * torch.sigmoid(g) * u
    if kind == "relu2":
        return g.clamp_min(0) ** 2
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def glu(z: torch.Tensor, F: int, kind: str, limit: float = 0.0, row_scale: Optional[torch.Tensor] = None,
        gate: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None, total_rows: Optional[torch.Tensor] = None,
        dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """act(s * z[:, :F], s * z[:, F:2F]) * sigmoid(gate): ``kind`` gelu_tanh (tanh-GELU(g) * u), silu (SiLU(g) * u), swiglu_oai (g clamped from
    above, u on both sides, g * sigmoid(1.702 g) * (u + 1)) or relu2 (the square of g's positive part, no u).  z fp32 (a column view is fine), ``row_scale`` [R] = s,
    ``gate`` [R, 1] (a view is fine).  ``out``: [R, >= F] view, columns past F become zero."""
    R = z.shape[0]
    if not z.is_cuda:
        g, u = z[:, :F].float(), z[:, :F].float() if kind == "relu2" else z[:, F:2 * F].float()
        if row_scale is not None:
            g, u = g * row_scale.unsqueeze(-1), u * row_scale.unsqueeze(-1)
        y = _glu_ref(g, u, kind, limit)
        if gate is not None:
            y = y * torch.sigmoid(gate.float())
        if out is None:
            return y.to(dtype or torch.float32)
        out.zero_()
        out[:, :F] = y.to(out.dtype)
        return out
    if out is None:
        out = torch.empty(R, F, dtype=dtype, device=z.device)
    assert z.dtype == torch.float32 and z.stride(1) == 1 and out.stride(1) == 1
    rc = _ext.lib().bg_glu(_i(_DT[out.dtype]), _i(GLU_KINDS[kind]), _ext.ptr(z), _i(z.stride(0)), _i(F), _ext.ptr(out),
                           _i(out.stride(0)), _i(R), _i(F), _i(out.shape[1]), ctypes.c_float(limit), _ext.ptr(row_scale),
                           _ext.ptr(gate), _i(gate.stride(0) if gate is not None else 0), _ext.ptr(total_rows),
                           _ext.stream())
    _ext.check(rc, "bg_glu")
    return out


def cast_act(x: torch.Tensor, cols: int, dtype: torch.dtype, act: str = "none") -> torch.Tensor:
    """fp32 columns (a view is fine) -> [T, cols] of ``dtype``, zero past x's width; ``act`` none, tanh or relu2 (the square
    of the positive part)."""
    if not x.is_cuda:
        y = torch.zeros(x.shape[0], cols, dtype=dtype)
        y[:, : x.shape[1]] = (torch.tanh(x) if act == "tanh" else x.clamp_min(0) ** 2 if act == "relu2" else x).to(dtype)
        return y
    assert x.dtype == torch.float32 and x.stride(1) == 1
    out = torch.empty(x.shape[0], cols, dtype=dtype, device=x.device)
    rc = _ext.lib().bg_cast_act(_i(_DT[dtype]), _i(CAST_KINDS[act]), _ext.ptr(x), _i(x.stride(0)), _ext.ptr(out), _i(cols),
                                _i(x.shape[0]), _i(x.shape[1]), _ext.stream())
    _ext.check(rc, "bg_cast_act")
    return out


@dataclass
class Norm:
    """A norm over the model width: (x - mean) / sqrt(variance + eps) * w + b when ``center``, else x / sqrt(mean square +
    eps) * w (+ b).  Vectors are fp32, padded with zeros to a multiple of 4."""
    w: torch.Tensor
    b: Optional[torch.Tensor] = None
    center: bool = False

    def ref(self, x: torch.Tensor, eps: float, width: int) -> torch.Tensor:
        if self.center:
            x = x - x.mean(-1, keepdim=True)
        y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * self.w[:width]
        return y if self.b is None else y + self.b[:width]


@dataclass
class Canon:
    """Input convolution of a decode step, folded into the norm: y = h + conv(h) over this token and the stored inputs."""
    w: torch.Tensor                 # [taps, width rounded up to 4] fp32
    hist: torch.Tensor              # [slots, (taps - 1) * same] fp32 (strided view of the state pool), updated
    slots: torch.Tensor             # [T] int32, < 0: no history, none kept


def sandwich_norm(x: torch.Tensor, norm: Optional[Norm], eps: float, width: int, out_cols: int, dtype: torch.dtype,
                  add: Optional[torch.Tensor] = None, add2: Optional[torch.Tensor] = None,
                  branch_w: Optional[Tuple[torch.Tensor, torch.Tensor]] = None, post: Optional[Norm] = None,
                  ids: Optional[torch.Tensor] = None, embed: Optional[torch.Tensor] = None, embed_scale: float = 1.0,
                  rows: Optional[torch.Tensor] = None, keep: bool = True, raw: bool = False,
                  canon: Optional[Canon] = None, routed: Optional[torch.Tensor] = None, pos: Optional[torch.Tensor] = None,
                  route_w: Optional[torch.Tensor] = None, emit: bool = True) -> Optional[torch.Tensor]:
    """x [T, >= width] fp32 += post(sublayer output), then norm(x) (None: x itself) as [R, out_cols] of ``dtype`` with zero columns
    past ``width``, or with ``raw`` as fp32 [R, width rounded up to 4], or with ``emit=False`` nothing.  The sublayer's output is
    ``add`` [T, width] fp32, or with ``add2`` half the sum of both, each RMS-normed with its weight of ``branch_w``, or
    sum_k route_w[t, k] * routed[pos[t, k]]; ``ids``: x = embed[ids] * embed_scale instead.  ``canon`` (one token per sequence) applies the input convolution to the result.  ``rows`` (int64) picks rows of
    x; ``keep=False`` leaves x as it was."""
    R = x.shape[0] if rows is None else rows.shape[0]
    W4 = pad_to(width, 4)
    if not x.is_cuda:
        r = rows.long() if rows is not None else torch.arange(x.shape[0])
        cur = x[r, :width].clone()
        if ids is not None:
            cur = embed[ids[r].long()].float() * embed_scale
        if routed is not None:
            at = pos[r].long()
            cur = cur + post.ref((routed[at.clamp_min(0), :width] * (route_w[r] * (at >= 0)).unsqueeze(-1)).sum(1), eps, width)
        elif add is not None:
            s = add[r, :width]
            if add2 is not None:
                s = 0.5 * sum(t / torch.sqrt((t * t).mean(-1, keepdim=True) + eps) * g[:width]
                              for t, g in zip((s, add2[r, :width]), branch_w))
            cur = cur + post.ref(s, eps, width)
        if keep:
            x[r, :width] = cur
            x[r, width:W4] = 0                    # (an input convolution reads whole vectors of 4)
        if not emit:
            return None
        h = torch.nn.functional.pad(cur if norm is None else norm.ref(cur, eps, width), (0, W4 - width))
        if raw:
            return h
        if canon is not None:
            from .conv import causal_conv
            return causal_conv(h, canon.w, canon.hist, canon.slots, torch.zeros(R, out_cols, dtype=dtype), "residual")
        y = torch.zeros(R, out_cols, dtype=dtype)
        y[:, :width] = h[:, :width].to(dtype)
        return y
    y = torch.empty(R, W4 if raw else out_cols, dtype=torch.float32 if raw else dtype, device=x.device) if emit else None
    for t in (add, add2, routed):
        assert t is None or (t.dtype == torch.float32 and t.stride(1) == 1)
    assert x.dtype == torch.float32 and (embed is None or embed.dtype == dtype)
    assert (add is None and routed is None) == (post is None) and (add is None or routed is None) and (emit or keep)
    if routed is not None:
        assert pos.dtype == torch.int32 and pos.is_contiguous() and route_w.is_contiguous() and route_w.dtype == torch.float32
        assert pos.shape == route_w.shape and pos.shape[0] == x.shape[0] and routed.stride(0) >= W4
    assert (ids is None or ids.dtype == torch.int32) and (rows is None or rows.dtype == torch.int64)
    assert x.shape[1] >= W4 and all(n is None or n.w.shape[0] == W4 for n in (norm, post))
    for t in (add, add2):
        assert t is None or (t.shape[0] == x.shape[0] and t.stride(0) >= W4)
    if canon is not None:
        taps = canon.w.shape[0]
        assert canon.w.shape[1] == W4 and canon.hist.shape[1] == (taps - 1) * W4 and canon.slots.shape[0] == R
    assert canon is None or (rows is None and not raw and canon.slots.dtype == torch.int32 and canon.hist.stride(1) == 1)
    P = lambda n: (_ext.ptr(n.w if n is not None else None), _ext.ptr(n.b if n is not None else None))   # noqa: E731
    rc = _ext.lib().bg_sandwich_norm(
        _i(_DT[dtype]), _ext.ptr(x), _i(x.stride(0)), _ext.ptr(rows), _ext.ptr(ids), _ext.ptr(embed),
        _i(embed.stride(0) if embed is not None else 0), ctypes.c_float(embed_scale),
        _i(embed.shape[0] if embed is not None else 0), _ext.ptr(add), _i(add.stride(0) if add is not None else 0),
        _ext.ptr(add2), _i(add2.stride(0) if add2 is not None else 0), _ext.ptr(branch_w[0] if add2 is not None else None),
        _ext.ptr(branch_w[1] if add2 is not None else None), _ext.ptr(routed), _i(routed.stride(0) if routed is not None else 0),
        _ext.ptr(pos), _ext.ptr(route_w), _i(pos.shape[1] if pos is not None else 0), *P(post), _i(post is not None and post.center),
        *P(norm), _i(norm is not None and norm.center), _ext.ptr(y), _i(y.shape[1] if emit else W4), _i(raw), _ext.ptr(canon.w if canon else None),
        _ext.ptr(canon.hist if canon else None), ctypes.c_longlong(canon.hist.stride(0) if canon else 0),
        _ext.ptr(canon.slots if canon else None), _i(canon.w.shape[0] if canon else 0), _i(R), _i(width), ctypes.c_float(eps),
        _i(keep), _ext.stream())
    _ext.check(rc, "bg_sandwich_norm")
    return y


def token_side(z: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, out_cols: int, dtype: torch.dtype) -> torch.Tensor:
    """tanh-GELU(z) * table[ids] as [T, out_cols] of ``dtype``, zero past the table's width: z [T, >= n] fp32 (a column view is
    fine), table [vocab, n] (a column view is fine), ids [T] int32 (clamped to the table)."""
    n = table.shape[1]
    if not z.is_cuda:
        g = z[:, :n].float()
        y = torch.zeros(z.shape[0], out_cols, dtype=dtype)
        y[:, :n] = (_glu_ref(g, table[ids.long().clamp(0, table.shape[0] - 1)].float(), "gelu_tanh", 0.0)).to(dtype)
        return y
    assert z.dtype == torch.float32 and z.stride(1) == 1 and table.stride(1) == 1 and table.dtype == dtype
    assert ids.dtype == torch.int32 and ids.shape[0] == z.shape[0] and z.shape[1] >= n and out_cols >= n
    out = torch.empty(z.shape[0], out_cols, dtype=dtype, device=z.device)
    rc = _ext.lib().bg_token_side(_i(_DT[dtype]), _ext.ptr(z), _i(z.stride(0)), _ext.ptr(table), ctypes.c_longlong(table.stride(0)),
                                  _ext.ptr(ids), _i(table.shape[0]), _ext.ptr(out), _i(out_cols), _i(z.shape[0]), _i(n), _ext.stream())
    _ext.check(rc, "bg_token_side")
    return out


@dataclass
class Hyper:
    """Fixed hyper-connections of one sublayer over s residual streams (fp32): it reads sum_s read[s] x_s, then stream t becomes
    sum_s mix[s, t] x_s + share[t] * output."""
    read: torch.Tensor              # [s]
    mix: torch.Tensor               # [s, s]
    share: torch.Tensor             # [s]


def hyper_norm(x: torch.Tensor, w: torch.Tensor, eps: float, width: int, out_cols: int, dtype: torch.dtype,
               read: Optional[torch.Tensor] = None, hc: Optional[Hyper] = None, add: Optional[torch.Tensor] = None,
               bias: Optional[torch.Tensor] = None, routed: Optional[torch.Tensor] = None, pos: Optional[torch.Tensor] = None,
               route_w: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None, embed: Optional[torch.Tensor] = None,
               embed_scale: float = 1.0, rows: Optional[torch.Tensor] = None, keep: bool = True) -> torch.Tensor:
    """x [T, s, width rounded up to 4] fp32 residual streams.  With ``hc`` the previous sublayer's output joins them: ``add``
    [T, width] fp32, plus ``bias``, plus sum_k route_w[t, k] * routed[pos[t, k]] (each optional).  ``ids``: every stream =
    embed[ids] * embed_scale instead.  Then rmsnorm(sum_s read[s] x_s) * w as [R, out_cols] of ``dtype``, zero past ``width``
    (``read`` None: the plain sum).  Vectors of the width are padded with zeros to a multiple of 4.  ``rows`` (int64) picks rows
    of x; ``keep=False`` leaves x as it was."""
    T, S, W4 = x.shape
    R = T if rows is None else rows.shape[0]
    if not x.is_cuda:
        r = rows.long() if rows is not None else torch.arange(T)
        cur = x[r, :, :width].clone()
        if ids is not None:
            cur = (embed[ids[r].long()].float() * embed_scale).unsqueeze(1).repeat(1, S, 1)
        if hc is not None:
            o = torch.zeros(R, width) if add is None else add[r, :width]
            if bias is not None:
                o = o + bias[:width]
            if routed is not None:
                at = pos[r].long()
                o = o + (routed[at.clamp_min(0), :width] * (route_w[r] * (at >= 0)).unsqueeze(-1)).sum(1)
            cur = torch.einsum("st,rsd->rtd", hc.mix, cur) + hc.share.view(1, S, 1) * o.unsqueeze(1)
        if keep:
            x[r, :, :width] = cur
        u = cur.sum(1) if read is None else torch.einsum("s,rsd->rd", read, cur)
        y = torch.zeros(R, out_cols, dtype=dtype)
        y[:, :width] = (u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps) * w[:width]).to(dtype)
        return y
    y = torch.empty(R, out_cols, dtype=dtype, device=x.device)
    f32 = [t for t in (add, routed) if t is not None]
    assert all(t.dtype == torch.float32 and t.stride(1) == 1 and t.stride(0) >= W4 for t in f32)
    assert x.dtype == torch.float32 and x.is_contiguous() and W4 == pad_to(width, 4) and w.shape[0] == W4
    assert (embed is None or embed.dtype == dtype) and (ids is None or (ids.dtype == torch.int32 and ids.shape[0] == T))
    assert (rows is None or rows.dtype == torch.int64) and (add is None or add.shape[0] == T) and (bias is None or bias.shape[0] == W4)
    assert hc is None or (hc.mix.shape == (S, S) and hc.share.shape[0] == S and hc.mix.is_contiguous())
    assert read is None or read.shape[0] == S
    if routed is not None:
        assert pos.dtype == torch.int32 and pos.is_contiguous() and route_w.is_contiguous() and route_w.dtype == torch.float32
        assert pos.shape == route_w.shape and pos.shape[0] == T
    rc = _ext.lib().bg_hyper_norm(
        _i(_DT[dtype]), _ext.ptr(x), _ext.ptr(rows), _ext.ptr(ids), _ext.ptr(embed), _i(embed.stride(0) if embed is not None else 0),
        ctypes.c_float(embed_scale), _i(embed.shape[0] if embed is not None else 0), _ext.ptr(hc.mix if hc else None),
        _ext.ptr(hc.share if hc else None), _ext.ptr(add), _i(add.stride(0) if add is not None else 0), _ext.ptr(bias),
        _ext.ptr(routed), _i(routed.stride(0) if routed is not None else 0), _ext.ptr(pos), _ext.ptr(route_w),
        _i(pos.shape[1] if pos is not None else 0), _ext.ptr(read), _ext.ptr(w), _ext.ptr(y), _i(out_cols), _i(R), _i(width), _i(S),
        ctypes.c_float(eps), _i(keep), _ext.stream())
    _ext.check(rc, "bg_hyper_norm")
    return y


def moe_gather(x: torch.Tensor, pos: torch.Tensor, w: torch.Tensor, rows: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """CUDA: (xs [rows, cols], ws [rows]) with xs[pos[t, k]] = x[t], ws[pos[t, k]] = w[t, k]; other rows stay undefined."""
    assert x.is_contiguous() and pos.dtype == torch.int32 and w.dtype == torch.float32
    xs = torch.empty(rows, x.shape[1], dtype=x.dtype, device=x.device)
    ws = torch.empty(rows, dtype=torch.float32, device=x.device)
    rc = _ext.lib().bg_moe_gather(_i(_DT[x.dtype]), _ext.ptr(x), _i(x.shape[1]), _ext.ptr(pos), _ext.ptr(w), _ext.ptr(xs),
                                  _ext.ptr(ws), _i(pos.shape[0]), _i(pos.shape[1]), _ext.stream())
    _ext.check(rc, "bg_moe_gather")
    return xs, ws
