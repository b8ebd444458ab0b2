"""Linear-attention recurrences with a matrix state per head (``csrc/linear_state.cu``): the gated delta rule with a decay per
key channel, the mLSTM cell with its running maximum and normaliser, retention with a fixed decay per head, and HGRN2, whose forget
gate per key channel is also what is not written.  All of them decay the rows of S [key channels x value channels], add a rank-one
write and read S^T q; the output is divided by its root mean square per head, scaled by a weight and (except HGRN2's) gated.

The generalised delta rule (``ops/delta.py``) runs on the same state kernels.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, Optional, Sequence

import torch
import torch.nn.functional as F

from . import _ext
from .conv import rotate_ref
from .residual import _DT

RULES = {"channel_delta": 0, "mlstm": 1, "retention": 2, "hgrn2": 3}
_GATES = {"sigmoid": torch.sigmoid, "silu": F.silu}


@dataclass
class RecurrentParams:
    """One layer's recurrence.  Head widths are padded to multiples of 8 with zero channels (dim_p, vdim_p)."""
    rule: str
    heads: int
    dim_p: int
    vdim: int                                 # real value width: channels of the output norm's mean
    vdim_p: int
    norm_w: torch.Tensor                      # [heads * vdim_p] fp32 gain of the output norm
    eps: float
    gate: str = "sigmoid"                     # activation of the output gate
    q_scale: float = 1.0
    k_scale: float = 1.0
    qk_heads: int = 0                         # channel_delta: head h reads query / key head h // (heads / qk_heads); 0 = heads
    rate: Optional[torch.Tensor] = None       # channel_delta: [heads] exp(A_log)
    dt_bias: Optional[torch.Tensor] = None    # channel_delta: [heads * dim_p]
    i_bias: Optional[torch.Tensor] = None     # mlstm: [heads]
    f_bias: Optional[torch.Tensor] = None
    gate_cap: float = 1.0
    decay: Optional[torch.Tensor] = None      # retention: [heads]
    f_lower: Optional[torch.Tensor] = None    # hgrn2: [heads * dim_p] lower bounds of the forget gate (its bias is ``f_bias``, as wide)
    unit_eps: float = 1e-6                    # channel_delta: inside the root of the unit vectors
    den_eps: float = 1e-6                     # mlstm: added to the denominator

    @property
    def n_qk(self) -> int:
        return self.qk_heads or self.heads


class _Args(ctypes.Structure):
    """``bg::rec::Args`` of csrc/state_rule.cuh, field for field."""
    _fields_ = ([(n, ctypes.c_void_p) for n in (
        "q", "k", "v", "gate", "low", "beta", "gate_i", "gate_f", "bias0", "bias1", "rate", "rope", "norm_w", "state",
        "norm_state", "max_state", "cu", "slots", "has_initial", "out", "scratch", "status")]
        + [(n, ctypes.c_longlong) for n in ("slot_stride",)]
        + [(n, ctypes.c_int) for n in ("dt", "rule", "ld_q", "ld_k", "ld_v", "ld_gate", "ld_low", "ld_beta", "ld_gi", "ld_gf",
                                       "ld_rope", "ld_out", "T", "nseq", "H", "rep", "K", "V", "v_real", "silu", "num_sms")]
        + [(n, ctypes.c_float) for n in ("q_scale", "k_scale", "cap", "ueps", "eps", "den_eps")])


def scratch_floats(p: RecurrentParams, T: int) -> int:
    """fp32 words the prompt form needs: a record per (token, head), the scan's outputs, mLSTM's gates and denominators."""
    vectors = 4 if p.rule == "channel_delta" else 2
    return T * p.heads * (vectors * p.dim_p + 4 + p.vdim_p + (8 if p.rule == "mlstm" else 0))


def recurrent_forward(p: RecurrentParams, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: Optional[torch.Tensor],
                      state: Dict[str, torch.Tensor], slots: torch.Tensor, out: torch.Tensor,
                      cu: Optional[torch.Tensor] = None, cu_host: Optional[Sequence[int]] = None,
                      has_initial: Optional[torch.Tensor] = None, *, low: Optional[torch.Tensor] = None,
                      beta: Optional[torch.Tensor] = None, gate_i: Optional[torch.Tensor] = None,
                      gate_f: Optional[torch.Tensor] = None, rope: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q, k [T, qk_heads * dim_p], v, gate [T, heads * vdim_p] (None: no gate): fp32 column views; ``out`` [T, >= heads * vdim_p] in the operand
    dtype.  ``state``: "S" [slots, heads * dim_p * vdim_p] (and mLSTM's "n", "m"), strided views of the pool; slots [nseq] int32
    (< 0: skipped, zero output); ``cu`` [nseq + 1] int32 token ranges, None = one token per sequence; ``has_initial`` [nseq]
    int32, None = continue from the slot.

    channel_delta: ``low`` [T, heads * dim_p] decay pre-activation, ``beta`` [T, >= heads] write strength before its sigmoid.
    mlstm: ``gate_i`` / ``gate_f`` [T, >= heads] gate pre-activations without their biases.
    retention: ``rope`` [T, dims] (``conv.Rotary.table``) turns q and k.
    hgrn2: ``k`` is the pre-activation of the forget gate without its bias, q is read through SiLU."""
    if not q.is_cuda:
        nseq = len(slots)
        bounds = list(range(nseq + 1)) if cu is None and cu_host is None else list(cu_host if cu_host is not None else cu.tolist())
        return _forward_ref(p, q, k, v, gate, state, [int(x) for x in slots], out, bounds,
                            None if has_initial is None else [int(x) for x in has_initial], low, beta, gate_i, gate_f, rope)
    S = state["S"]
    for t in (q, k, v, gate, low, beta, gate_i, gate_f, rope, S):
        assert t is None or (t.dtype == torch.float32 and t.stride(1) == 1)
    assert out.stride(1) == 1 and slots.dtype == torch.int32
    T, a = q.shape[0], _Args()
    qk, n = p.n_qk * p.dim_p, p.heads * p.vdim_p
    for t, cols in ((q, qk), (k, qk), (v, n), (gate, n), (out, n), (low, p.heads * p.dim_p), (beta, p.heads), (gate_i, p.heads),
                    (gate_f, p.heads), (rope, 0)):
        assert t is None or (t.shape[0] == T and t.shape[1] >= cols), "rows or columns of an input do not match"
    assert S.shape[1] == p.heads * p.dim_p * p.vdim_p and (cu is None or cu.shape[0] == slots.shape[0] + 1)
    for name, cols in (("n", p.heads * p.dim_p), ("m", p.heads)) if p.rule == "mlstm" else ():
        t = state[name]                                       # parts of one pool: the kernels step all of them by S's slot stride
        assert t.dtype == torch.float32 and t.stride() == S.stride() and t.shape == (S.shape[0], cols)
    if p.rule == "hgrn2":
        assert p.f_bias.shape[0] == p.f_lower.shape[0] == p.heads * p.dim_p and p.f_bias.dtype == p.f_lower.dtype == torch.float32
    scratch = None
    if cu is not None or p.dim_p > 128 or p.vdim_p > 128:
        scratch = torch.empty(scratch_floats(p, T), dtype=torch.float32, device=q.device)
    tensors = dict(q=q, k=k, v=v, gate=gate, low=low, beta=beta, gate_i=gate_i, gate_f=gate_f,
                   bias0={"channel_delta": p.dt_bias, "hgrn2": p.f_bias}.get(p.rule, p.i_bias), bias1=p.f_bias,
                   rate={"retention": p.decay, "hgrn2": p.f_lower}.get(p.rule, p.rate), rope=rope, norm_w=p.norm_w, state=S,
                   norm_state=state.get("n"), max_state=state.get("m"), cu=cu, slots=slots, has_initial=has_initial, out=out,
                   scratch=scratch, status=_ext.status_word(q.device))
    for n, t in tensors.items():
        setattr(a, n, 0 if t is None else t.data_ptr())
    for n, t in dict(ld_q=q, ld_k=k, ld_v=v, ld_gate=gate, ld_low=low, ld_beta=beta, ld_gi=gate_i, ld_gf=gate_f, ld_rope=rope,
                     ld_out=out).items():
        setattr(a, n, 0 if t is None else t.stride(0))
    a.slot_stride, a.dt, a.rule, a.T, a.nseq, a.H, a.rep = (S.stride(0), _DT[out.dtype], RULES[p.rule], T, slots.shape[0],
                                                           p.heads, p.heads // p.n_qk)
    a.K, a.V, a.v_real, a.silu, a.num_sms = p.dim_p, p.vdim_p, p.vdim, int(p.gate == "silu"), _ext.num_sms(q.device)
    a.q_scale, a.k_scale, a.cap, a.ueps, a.eps, a.den_eps = p.q_scale, p.k_scale, p.gate_cap, p.unit_eps, p.eps, p.den_eps
    rc = _ext.lib().bg_recurrent_forward(ctypes.byref(a), _ext.stream())
    if rc == -1:
        raise _ext.KernelError(f"recurrent_forward: {p.heads} heads of {p.dim_p} x {p.vdim_p} are outside the kernels' "
                               "contract (key width <= 512)")
    _ext.check(rc, "bg_recurrent_forward", kernels=1 if scratch is None else 4 if p.rule == "mlstm" else 3)
    return out


# ---------------------------------------------------------------- CPU form
def _step_inputs(p, q, k, v, low, beta, gate_i, gate_f, rope):
    """Per token what the recurrence consumes: q, k [T, H, K], v [T, H, V] and the rule's own gates."""
    H, K, V, rep = p.heads, p.dim_p, p.vdim_p, p.heads // p.n_qk
    q, k = (t[:, :p.n_qk * K].float().view(-1, p.n_qk, K) for t in (q, k))
    v = v[:, :H * V].float().view(-1, H, V)
    if p.rule == "channel_delta":
        q, k = (t / torch.sqrt((t * t).sum(-1, keepdim=True) + p.unit_eps) for t in (q, k))
        g = torch.exp(-p.rate.view(H, 1) * F.softplus(low[:, :H * K].float().view(-1, H, K) + p.dt_bias.view(H, K)))
        extra = (g, torch.sigmoid(beta[:, :H].float()))
    elif p.rule == "mlstm":
        def cap(x, b):
            return p.gate_cap * torch.tanh((x[:, :H].float() + b) / p.gate_cap)
        extra = (cap(gate_i, p.i_bias), F.logsigmoid(cap(gate_f, p.f_bias)))
    elif p.rule == "hgrn2":
        f = p.f_lower + (1 - p.f_lower) * torch.sigmoid(k.reshape(-1, H * K) + p.f_bias)
        q, extra = F.silu(q), (f.view(-1, H, K),)
    else:
        q, k, extra = rotate_ref(q, rope), rotate_ref(k, rope), ()
    return (q * p.q_scale).repeat_interleave(rep, 1), (k * p.k_scale).repeat_interleave(rep, 1), v, extra


def _forward_ref(p, q, k, v, gate, state, slots, out, cu, has_initial, low, beta, gate_i, gate_f, rope):
    H, K, V = p.heads, p.dim_p, p.vdim_p
    qs, ks, vs, extra = _step_inputs(p, q, k, v, low, beta, gate_i, gate_f, rope)
    act = _GATES[p.gate]
    for s, slot in enumerate(slots):
        lo, hi = cu[s], cu[s + 1]
        if slot < 0:
            out[lo:hi].zero_()
            continue
        if hi <= lo:
            continue
        if has_initial is not None and not has_initial[s]:
            for t in state.values():
                t[slot].zero_()
        S = state["S"][slot].view(H, K, V).clone()
        if p.rule == "mlstm":
            n, m = state["n"][slot].view(H, K).clone(), state["m"][slot].clone()
        for t in range(lo, hi):
            write = ks[t].unsqueeze(-1)
            if p.rule == "channel_delta":
                g, b = extra[0][t], extra[1][t]
                S = g.unsqueeze(-1) * S
                S = S + write * (b.unsqueeze(-1) * (vs[t] - torch.einsum("hkv,hk->hv", S, ks[t]))).unsqueeze(1)
                o = torch.einsum("hkv,hk->hv", S, qs[t])
            elif p.rule == "mlstm":
                i, f = extra[0][t], extra[1][t]
                new = torch.maximum(f + m, i)
                keep, put = torch.exp(f + m - new), torch.exp(i - new)
                S = keep.view(H, 1, 1) * S + put.view(H, 1, 1) * write * vs[t].unsqueeze(1)
                n, m = keep.view(H, 1) * n + put.view(H, 1) * ks[t], new
                den = torch.maximum((n * qs[t]).sum(-1).abs(), torch.exp(-m)) + p.den_eps
                o = torch.einsum("hkv,hk->hv", S, qs[t]) / den.unsqueeze(-1)
            elif p.rule == "hgrn2":
                f = extra[0][t].unsqueeze(-1)
                S = f * S + (1 - f) * vs[t].unsqueeze(1)
                o = torch.einsum("hkv,hk->hv", S, qs[t])
            else:
                S = p.decay.view(H, 1, 1) * S + write * vs[t].unsqueeze(1)
                o = torch.einsum("hkv,hk->hv", S, qs[t])
            o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / p.vdim + p.eps)
            o = o.reshape(-1) * p.norm_w
            if gate is not None:
                o = o * act(gate[t, :H * V].float())
            out[t, :H * V] = o.to(out.dtype)
        state["S"][slot] = S.reshape(-1)
        if p.rule == "mlstm":
            state["n"][slot], state["m"][slot] = n.reshape(-1), m
    return out
