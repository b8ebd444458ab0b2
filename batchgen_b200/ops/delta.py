"""Generalised delta rule (``csrc/delta_rule.cu``): a matrix state per head with per-channel decay and removal rates,
its gated output norm included.  See ``DeltaParams`` for the shapes; the state of a sequence lives in a slot pool.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import torch

from . import _ext
from .residual import _DT, _i


@dataclass
class DeltaParams:
    """Per-layer vectors, fp32, [heads * Dp] (Dp: head width padded to a multiple of 8; zero in the padding)."""
    w0: torch.Tensor             # decay offset
    ab: torch.Tensor             # removal-rate offset
    norm_w: torch.Tensor         # gain of the output norm
    heads: int
    dim: int                     # real head width: channels of the output norm's mean
    dim_p: int
    decay_scale: float           # c of decay = exp(-c * sigmoid(.))
    unit_eps: float = 1e-6       # inside the root of the unit key
    eps: float = 1e-6            # of the output norm


def _delta_ref(z, offs, wl, p: DeltaParams, state, cu, slots, has_initial, out):
    H, D = p.heads, p.dim_p
    n = H * D
    r, k, v, g, a = (z[:, o:o + n].float().view(-1, H, D) for o in offs)
    w = torch.exp(-p.decay_scale * torch.sigmoid(wl.float().view(-1, H, D) + p.w0.view(H, D)))
    a = torch.sigmoid(a + p.ab.view(H, D))
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + p.unit_eps)
    for s, slot in enumerate(slots):
        lo, hi = cu[s], cu[s + 1]
        if slot < 0:
            out[lo:hi].zero_()
            continue
        if hi <= lo:
            continue
        S = state[slot].view(H, D, D).clone()
        if has_initial is not None and not has_initial[s]:
            S.zero_()
        for t in range(lo, hi):
            y = torch.einsum("hk,hkv->hv", u[t], S)
            S = w[t].unsqueeze(-1) * S - (a[t] * u[t]).unsqueeze(-1) * y.unsqueeze(1) + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
            o = torch.einsum("hkv,hk->hv", S, r[t])
            o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / p.dim + p.eps) * p.norm_w.view(H, D) * torch.sigmoid(g[t])
            out[t] = o.reshape(-1).to(out.dtype)
        state[slot] = S.reshape(state[slot].shape)
    return out


def delta_forward(z: torch.Tensor, offs: Tuple[int, int, int, int, int], wl: torch.Tensor, p: DeltaParams,
                  state: torch.Tensor, slots: torch.Tensor, out: torch.Tensor, cu: Optional[torch.Tensor] = None,
                  cu_host: Optional[Sequence[int]] = None, has_initial: Optional[torch.Tensor] = None) -> torch.Tensor:
    """z [T, *] fp32: stacked projections, ``offs`` the first columns of r, k, v, g (output gate) and a (removal rate);
    wl [T, heads * Dp] fp32 decay pre-activation; state [slots, heads * Dp * Dp] fp32 (a strided column view of the pool);
    slots [nseq] int32 (< 0: skipped, zero output); ``cu`` [nseq + 1] int32 token ranges, None = one token per sequence;
    ``has_initial`` [nseq] int32, None = continue from the slot.  ``out``: [T, >= heads * Dp] view in the operand dtype."""
    if not z.is_cuda:
        nseq = len(slots)
        bounds = list(range(nseq + 1)) if cu is None and cu_host is None else list(cu_host if cu_host is not None else cu.tolist())
        return _delta_ref(z, offs, wl, p, state, bounds, [int(x) for x in slots],
                          None if has_initial is None else [int(x) for x in has_initial], out)
    assert z.dtype == wl.dtype == state.dtype == torch.float32 and z.stride(1) == 1 and wl.stride(1) == 1
    assert out.stride(1) == 1 and state.stride(1) == 1 and slots.dtype == torch.int32
    arr = (ctypes.c_int * 5)(*offs)
    T = z.shape[0]
    scratch = None
    if cu is not None or p.dim_p > 128:
        per = p.heads * (6 * p.dim_p + 4)                      # a token's record and its scan output
        scratch = torch.empty(T * per, dtype=torch.float32, device=z.device)
    rc = _ext.lib().bg_delta_forward(
        _i(_DT[out.dtype]), _ext.ptr(z), _i(z.stride(0)), arr, _ext.ptr(wl), _i(wl.stride(0)), _ext.ptr(p.w0),
        _ext.ptr(p.ab), _ext.ptr(p.norm_w), _ext.ptr(state), ctypes.c_longlong(state.stride(0)), _ext.ptr(cu),
        _ext.ptr(slots), _ext.ptr(has_initial), _ext.ptr(out), _i(out.stride(0)), _i(T), _i(slots.shape[0]), _i(p.heads),
        _i(p.dim_p), _i(p.dim), ctypes.c_float(p.decay_scale), ctypes.c_float(p.unit_eps), ctypes.c_float(p.eps),
        _ext.ptr(scratch), _i(_ext.num_sms(z.device)), _ext.ptr(_ext.status_word(z.device)), _ext.stream())
    if rc == -1:
        raise _ext.KernelError(f"delta_forward: {p.heads} heads of {p.dim_p} are outside the kernels' contract (width <= 512)")
    _ext.check(rc, "bg_delta_forward", kernels=3 if scratch is not None else 1)
    return out
