"""Token mixers of layer-listed models: their weights (``build_mixer``) and one step over projected tokens (``Mixer.run``).

A mixer lists the projections that read the layer input (``parts``); the block stacks them into one matrix and tells the mixer
where its columns of the GEMM output start (``seg``).  ``run`` reads those fp32 columns, uses and updates the caller's cache
(paged rows, state slots) and writes the operand of the output projection.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from ..config import MixerSpec, ModelConfig
from ..ops import conv, delta, gemm, recurrent, residual, talking
from ..ops.residual import pad_to
from .weights import WeightSource

DECAY_SCALE = math.exp(-0.5)       # decay = exp(-DECAY_SCALE * sigmoid(.)), so a channel keeps at least exp(-exp(-1/2)) a step
K_ALIGN = 64


@dataclass
class StepPlan:
    """Device tables of one step, shared by its layers."""
    lens: torch.Tensor                            # [T] int32: position + 1 (0 = padding row)
    row_seq: Optional[torch.Tensor]               # [T] int32 block-table row of each token, None = identity
    cu: Optional[torch.Tensor]                    # [nseq + 1] int32, None = one token per sequence
    cu_host: Optional[List[int]]
    slots: Optional[torch.Tensor]
    has_initial: Optional[torch.Tensor]
    ctx: Optional[List[int]] = None
    tiles: Dict[Tuple[int, int], Tuple] = field(default_factory=dict)      # chunk, window -> (tensor-core tiles, rows of short pieces)
    ropes: Dict[Tuple, torch.Tensor] = field(default_factory=dict)

    def rope(self, r: Optional[conv.Rotary]) -> Optional[torch.Tensor]:
        if r is None:
            return None
        if r.key not in self.ropes:
            self.ropes[r.key] = r.table(self.lens)
        return self.ropes[r.key]

    def attention_tiles(self, chunk: int, T: int, window: int = 0):
        """How the rows of a prompt step split over the attention kernels: pieces of a few tokens (decoded tokens among
        them) go row by row, the rest in 128-query tiles."""
        if (chunk, window) not in self.tiles:
            cu, least, dev = self.cu_host, talking.PREFILL_MIN_TOKENS, self.lens.device
            blocks = talking.work_blocks(talking.prefill_work(cu, self.ctx, chunk, least, window), T, dev)
            short = [t for a, b in zip(cu, cu[1:]) if b - a < least for t in range(a, b)]
            rows = seqs = None
            if blocks and short:
                rows = torch.tensor(short, dtype=torch.int32, device=dev)
                seqs = self.row_seq[rows.long()].contiguous()
            elif short:
                seqs = self.row_seq
            self.tiles[chunk, window] = (blocks, bool(short), rows, seqs)
        return self.tiles[chunk, window]


@dataclass
class Mixer:
    spec: MixerSpec
    cols: int                                     # columns of the output it writes
    suffix: str = ""                              # of its state parts' names
    parts: List[Tuple[str, torch.Tensor]] = field(default_factory=list)     # projections of the layer input (until stacked)
    o: Optional[torch.Tensor] = None              # [width, cols] output projection (until stacked)
    seg: Dict[str, Tuple[int, int]] = field(default_factory=dict)           # name -> (first column, width)
    w_low: Optional[torch.Tensor] = None          # second factor(s) of low-rank projections, [rows, rank_p]
    conv_w: Optional[torch.Tensor] = None         # channel_delta: [taps, conv channels] fp32
    rot: Optional[conv.Rotary] = None
    delta: Optional[delta.DeltaParams] = None
    talk: Optional[talking.TalkParams] = None
    prep: Optional[talking.HeadPrep] = None       # attention with biases or norms of its heads
    o_bias: Optional[torch.Tensor] = None         # [width] fp32 bias of the output projection, times the output's scale
    rec: Optional[recurrent.RecurrentParams] = None

    def column(self, z: torch.Tensor, name: str) -> torch.Tensor:
        o, n = self.seg[name]
        return z[:, o:o + n]

    def low(self, z: torch.Tensor, dtype: torch.dtype, act: str = "none") -> torch.Tensor:
        return gemm.rows_gemm(residual.cast_act(self.column(z, "low"), self.w_low.shape[1], dtype, act), self.w_low)

    def run(self, l: int, z: torch.Tensor, out: torch.Tensor, plan: StepPlan, meta, cache) -> None:
        if self.talk is not None:
            self._attention(l, z, out, plan, meta, cache)
            return
        if plan.slots is None:
            raise RuntimeError("a model with recurrent layers needs AttnMeta.state_slots")
        where = dict(cu=plan.cu, cu_host=plan.cu_host, has_initial=plan.has_initial)
        if self.delta is not None:
            delta.delta_forward(z, tuple(self.seg[x][0] for x in ("r", "k", "v", "g", "a")), self.low(z, out.dtype, "tanh"),
                                self.delta, cache.state.layer(l, "S" + self.suffix), plan.slots, out, **where)
            return
        p = self.rec
        state = {n: cache.state.layer(l, n + self.suffix) for n in self.spec.state_parts}
        if p.rule == "channel_delta":
            C, qk = self.spec.conv_channels, p.n_qk * p.dim_p
            low = self.low(z, out.dtype)
            x = torch.empty(z.shape[0], C, dtype=torch.float32, device=z.device)
            q0 = self.seg["q"][0]
            conv.causal_conv(z[:, q0:q0 + C], self.conv_w, state.pop("conv"), plan.slots, x, "silu", row_seq=plan.row_seq, **where)
            n = p.heads * p.dim_p
            recurrent.recurrent_forward(p, x[:, :qk], x[:, qk:2 * qk], x[:, 2 * qk:], low[:, n:], state, plan.slots, out,
                                        low=low[:, :n], beta=self.column(z, "b"), **where)
            return
        q, k, v, g = (self.column(z, x) for x in "qkvg")
        extra = (dict(gate_i=self.column(z, "i"), gate_f=self.column(z, "f")) if p.rule == "mlstm"
                 else dict(rope=plan.rope(self.rot)))
        recurrent.recurrent_forward(p, q, k, v, g, state, plan.slots, out, **where, **extra)

    def _attention(self, l: int, z, out, plan: StepPlan, meta, cache) -> None:
        k, p = self.seg["k"][0], self.talk
        kv, rope = cache.latent(l), plan.rope(self.rot)
        zq = self.column(z, "q")
        blocks, short, rows, seqs = [], True, None, plan.row_seq
        if plan.cu is not None and z.is_cuda and talking.prefill_supported(p, kv.dtype, kv.shape[1]):
            blocks, short, rows, seqs = plan.attention_tiles(p.chunk, z.shape[0], p.window)
        more = dict(rope=rope, gate=self.column(z, "gate") if "gate" in self.seg else None)
        operand = None
        if self.prep is not None:
            q0 = self.seg["q"][0]
            operand = talking.prepare_heads(z[:, q0:q0 + p.heads * p.dim_p + p.kv_row], meta.slot_mapping, kv, p, self.prep, rope,
                                            short, bool(blocks))
            more["rope"] = None                   # the queries have turned
        else:
            talking.kv_write(z[:, k:k + p.kv_row], meta.slot_mapping, kv, p, rope)
        if blocks:
            talking.attend_prefill(zq, p, kv, meta.block_table, out, blocks, operand=operand, **more)
        if short:
            talking.attend_rows(zq, p, kv, meta.block_table, plan.lens, out, seqs, rows, **more)


# ---------------------------------------------------------------- weights
def pad_cols(w: torch.Tensor, cols: int) -> torch.Tensor:
    return w if w.shape[1] == cols else torch.nn.functional.pad(w, (0, cols - w.shape[1]))


def pad_rows(w: torch.Tensor, rows: int) -> torch.Tensor:
    return w if w.shape[0] == rows else torch.nn.functional.pad(w, (0, 0, 0, rows - w.shape[0]))


def head_rows(w: torch.Tensor, heads: int, d: int, dp: int) -> torch.Tensor:
    """[heads * d, ...] -> [heads * dp, ...]: zero rows behind every head."""
    if d == dp:
        return w
    out = w.new_zeros(heads, dp, *w.shape[1:])
    out[:, :d] = w.view(heads, d, *w.shape[1:])
    return out.view(heads * dp, *w.shape[1:])


def stack_parts(parts: List[Tuple[Dict, str, torch.Tensor]], cols: int, dtype: torch.dtype) -> torch.Tensor:
    """One [rows, cols] matrix of all parts (each starts on a multiple of 8 rows); every part's place goes into its ``seg``."""
    row, stack = 0, []
    for seg, name, t in parts:
        seg[name] = (row, t.shape[0])
        stack.append(pad_rows(t.to(dtype), pad_to(t.shape[0], 8)))
        row += stack[-1].shape[0]
    return pad_cols(torch.cat(stack, 0), cols).contiguous()


def build_mixer(m: MixerSpec, p: str, src: WeightSource, cfg: ModelConfig, dtype: torch.dtype, index: int = 0) -> Mixer:
    """``p``: prefix of the tensor names; ``index``: place among the layer's mixers."""
    D, H, G, d, dp, dv, dvp = cfg.hidden_size, m.heads, m.qk_heads, m.dim, m.dim_p, m.vdim, m.vdim_p
    dev = src.device
    mx = Mixer(m, H * dvp, f".{index}" if index else "")

    def rows(name, heads, w, wp, kind="normal", tail=(D,)):
        return head_rows(src.get(p + name, (heads * w, *tail), kind), heads, w, wp)

    def vector(name, heads, w, wp, kind):
        return rows(name, heads, w, wp, kind, ()).float().contiguous()
    if m.kind == "attention":
        mx.parts = [("q", rows("q", H, d, dp)), ("k", rows("k", G, d, dp)), ("v", rows("v", G, dv, dvp))]
        if m.out_gate:
            mx.parts.append(("gate", src.get(p + "g", (H, D))))
        talk = src.get(p + "talk", (H, H)).float().contiguous() if m.talking else None
        mx.talk = talking.TalkParams(heads=H, kv_heads=G, dim_p=dp, vdim_p=dvp, scale=m.scale, chunk=m.chunk, sink=m.sink, talk=talk,
                                     window=m.window, keep=m.keep_first if m.window else 0, out_scale=m.out_scale)
        if m.bias or m.qk_norm or m.rot_interleaved:
            mx.prep = talking.HeadPrep(dim=d, eps=cfg.rms_eps, interleaved=m.rot_interleaved)
        if m.bias:
            mx.prep.bias = torch.cat([vector(x + ".b", n, w, wp, "bias") for x, n, w, wp in (("q", H, d, dp), ("k", G, d, dp),
                                                                                        ("v", G, dv, dvp))])
            mx.o_bias = src.get(p + "o.b", (D,), "bias").float() * m.out_scale
        if m.qk_norm:
            mx.prep.q_norm, mx.prep.k_norm = (vector(x + ".norm", 1, d, dp, "norm") for x in "qk")
    elif m.kind == "general_delta":
        mx.parts = [(x, rows(x, H, d, dp)) for x in ("r", "k", "v", "g", "a")]
        mx.parts.append(("low", src.get(p + "w1", (m.decay_rank, D))))
        mx.delta = delta.DeltaParams(w0=vector("w0", H, d, dp, "bias"), ab=vector("a.b", H, d, dp, "bias"),
                                     norm_w=vector("norm", H, d, dp, "norm"), heads=H, dim=d, dim_p=dp, decay_scale=DECAY_SCALE,
                                     eps=cfg.rms_eps)
        w2 = rows("w2", H, d, dp, tail=(m.decay_rank,))
        mx.w_low = pad_cols(w2.to(dtype), pad_to(m.decay_rank, K_ALIGN)).contiguous()
    else:
        mx.parts = [("q", rows("q", G, d, dp)), ("k", rows("k", G, d, dp)), ("v", rows("v", H, dv, dvp))]
        base = dict(rule=m.kind, heads=H, dim_p=dp, vdim=dv, vdim_p=dvp, eps=cfg.rms_eps)
        if m.kind == "channel_delta":
            mx.parts += [("b", src.get(p + "b", (H, D))),
                         ("low", torch.cat([src.get(p + "a1", (m.decay_rank, D)), src.get(p + "g1", (m.gate_rank, D))]))]
            ra, rg = m.decay_rank, m.gate_rank
            low = torch.zeros(H * (dp + dvp), pad_to(ra + rg, K_ALIGN), device=dev)       # both second factors in one product
            low[:H * dp, :ra] = rows("a2", H, d, dp, tail=(ra,))
            low[H * dp:, ra:ra + rg] = rows("g2", H, dv, dvp, tail=(rg,))
            mx.w_low = low.to(dtype).contiguous()
            taps = [rows(x + ".conv", h, w, wp, tail=(m.conv,)) for x, h, w, wp in (("q", G, d, dp), ("k", G, d, dp), ("v", H, dv, dvp))]
            mx.conv_w = torch.cat(taps, 0).float().t().contiguous()
            norm = head_rows(src.get(p + "norm", (dv,), "norm").repeat(H), H, dv, dvp)
            mx.rec = recurrent.RecurrentParams(**base, norm_w=norm.float().contiguous(), q_scale=d ** -0.5, qk_heads=G,
                                               rate=torch.exp(src.get(p + "A_log", (H,), "bias").float()),
                                               dt_bias=vector("dt_bias", H, d, dp, "bias"))
        elif m.kind == "mlstm":
            mx.parts += [("g", rows("g", H, dv, dvp)), ("i", src.get(p + "i", (H, D))), ("f", src.get(p + "f", (H, D)))]
            mx.rec = recurrent.RecurrentParams(**base, norm_w=vector("norm", H, dv, dvp, "norm"), q_scale=d ** -0.5,
                                               gate_cap=m.gate_cap, i_bias=src.get(p + "i.b", (H,), "bias").float().contiguous(),
                                               f_bias=src.get(p + "f.b", (H,), "bias").float().contiguous())
        else:
            mx.parts.append(("g", rows("g", H, dv, dvp)))
            mx.rec = recurrent.RecurrentParams(**base, norm_w=torch.full((H * dvp,), m.out_scale, device=dev), gate="silu", k_scale=d ** -0.5,
                                               decay=torch.tensor(m.decay, dtype=torch.float32, device=dev))
    mx.rot = conv.Rotary.make(m.rot_dims, m.rot_base, dev, m.rot_interleaved, m.yarn)
    mx.o = head_rows(src.get(p + "o", (D, H * dv)).t().contiguous(), H, dv, dvp).t()       # [D, heads * dvp]: zero columns
    return mx


def mixer_tensor_specs(m: MixerSpec, p: str, D: int, layer: int) -> List[Tuple[str, Tuple[int, ...], str, int]]:
    """(name, shape, init kind, layer) of a mixer's checkpoint tensors."""
    qk, kv, n, H = m.heads * m.dim, m.qk_heads * m.dim, m.heads * m.vdim, m.heads
    if m.kind == "attention":
        out = [("q", (qk, D), "normal"), ("k", (kv, D), "normal"), ("v", (m.kv_heads * m.vdim, D), "normal")]
        out += [("talk", (H, H), "normal")] if m.talking else []
        out += [("g", (H, D), "normal")] if m.out_gate else []
        out += [("q.b", (qk,), "bias"), ("k.b", (kv,), "bias"), ("v.b", (m.kv_heads * m.vdim,), "bias"), ("o.b", (D,), "bias")] if m.bias else []
        out += [("q.norm", (m.dim,), "norm"), ("k.norm", (m.dim,), "norm")] if m.qk_norm else []
    elif m.kind == "general_delta":
        out = [(x, (qk, D), "normal") for x in ("r", "k", "v", "g", "a")]
        out += [("w1", (m.decay_rank, D), "normal"), ("w2", (qk, m.decay_rank), "normal"), ("a.b", (qk,), "bias"),
                ("w0", (qk,), "bias"), ("norm", (qk,), "norm")]
    elif m.kind == "channel_delta":
        out = [("q", (kv, D), "normal"), ("k", (kv, D), "normal"), ("v", (n, D), "normal"), ("q.conv", (kv, m.conv), "normal"),
               ("k.conv", (kv, m.conv), "normal"), ("v.conv", (n, m.conv), "normal"), ("b", (H, D), "normal"),
               ("A_log", (H,), "bias"), ("norm", (m.vdim,), "norm"), ("a1", (m.decay_rank, D), "normal"),
               ("a2", (qk, m.decay_rank), "normal"), ("dt_bias", (qk,), "bias"), ("g1", (m.gate_rank, D), "normal"),
               ("g2", (n, m.gate_rank), "normal")]
    else:
        out = [("q", (qk, D), "normal"), ("k", (qk, D), "normal"), ("v", (n, D), "normal"), ("g", (n, D), "normal")]
        if m.kind == "mlstm":
            out += [("norm", (n,), "norm"), ("i", (H, D), "normal"), ("i.b", (H,), "bias"), ("f", (H, D), "normal"),
                    ("f.b", (H,), "bias")]
    return [(p + name, shape, kind, layer) for name, shape, kind in out + [("o", (D, n), "normal")]]
