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
from ..ops import conv, delta, gemm, latent, recurrent, residual, talking
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

    def latent_tiles(self, window: int, page: int):
        """The same for attention over latents in its expanded form: (expansions, rows of short pieces, their block-table rows and
        lengths), or no rows (None, None, None) when every piece is long."""
        key = ("latent", window)
        if key not in self.tiles:
            cu, least, dev = self.cu_host, talking.PREFILL_MIN_TOKENS, self.lens.device
            groups = latent.expansions(cu, self.ctx, window, page, dev)
            short = [t for a, b in zip(cu, cu[1:]) if b - a < least for t in range(a, b)]
            if not groups:
                self.tiles[key] = ([], None, self.row_seq, self.lens)
            elif short:
                rows = torch.tensor(short, dtype=torch.int32, device=dev)
                self.tiles[key] = (groups, rows, self.row_seq[rows.long()].contiguous(), self.lens[rows.long()].contiguous())
            else:
                self.tiles[key] = (groups, None, None, None)
        return self.tiles[key]


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
    lat: Optional[latent.LatentParams] = None

    def column(self, z: torch.Tensor, name: str) -> torch.Tensor:
        o, n = self.seg[name]
        return z[:, o:o + n]

    def low(self, z: torch.Tensor, dtype: torch.dtype, act: str = "none") -> torch.Tensor:
        return gemm.rows_gemm(residual.cast_act(self.column(z, "low"), self.w_low.shape[1], dtype, act), self.w_low)

    def run(self, l: int, z: torch.Tensor, out: torch.Tensor, plan: StepPlan, meta, cache) -> None:
        if self.talk is not None:
            self._attention(l, z, out, plan, meta, cache)
            return
        if self.lat is not None:
            self._latent(l, z, out, plan, meta, cache)
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
        if p.rule == "hgrn2":
            q, f, v = (self.column(z, x) for x in "qfv")
            recurrent.recurrent_forward(p, q, f, v, None, state, plan.slots, out, **where)
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

    def _latent(self, l: int, z, out, plan: StepPlan, meta, cache) -> None:
        p, dt = self.lat, out.dtype
        own = self.spec.kv_from < 0
        kv, rope = cache.latent(l if own else self.spec.kv_from), plan.rope(self.rot)
        cols = tuple(self.seg[x][0] if x in self.seg else None for x in ("dq", "c", "r"))
        q = gemm.rows_gemm(latent.prepare(z, cols, meta.slot_mapping, kv, p, rope, dt), p.w_uq)
        groups, rows, seqs, lens = [], None, plan.row_seq, plan.lens
        if plan.cu is not None and z.is_cuda and latent.prompt_supported(p, kv.dtype, kv.shape[1]):
            groups, rows, seqs, lens = plan.latent_tiles(p.window, kv.shape[1])
        if groups:
            latent.attend_prompt(q, p, kv, meta.block_table, rope, out, groups)
        if lens is None:
            return
        o = latent.attend(latent.queries(q, p, rope, rows, dt), p, kv, meta.block_table, lens, seqs)
        if rows is None:
            latent.head_product(o, p.w_uv, out.unflatten(1, (p.heads, p.vdim_p)))
            return
        short = torch.empty(rows.shape[0], p.heads, p.vdim_p, dtype=dt, device=out.device)
        latent.head_product(o, p.w_uv, short)
        out.index_copy_(0, rows.long(), short.view(rows.shape[0], -1))


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
        elif m.out_gate_all:
            mx.parts.append(("gate", rows("g", H, dv, dvp)))
        talk = src.get(p + "talk", (H, H)).float().contiguous() if m.talking else None
        mx.talk = talking.TalkParams(heads=H, kv_heads=G, dim_p=dp, vdim_p=dvp, scale=m.scale, chunk=m.chunk, sink=m.sink, talk=talk,
                                     window=m.window, keep=m.keep_first if m.window else 0, out_scale=m.out_scale, gate_all=m.out_gate_all,
                                     sinks=src.get(p + "sink", (H,), "bias").float().contiguous() if m.head_sinks else None)
        if m.bias or m.qk_norm or m.qk_norm_all or m.rot_interleaved:
            mx.prep = talking.HeadPrep(dim=d, eps=cfg.rms_eps, interleaved=m.rot_interleaved, whole=m.qk_norm_all)
        if m.bias:
            mx.prep.bias = torch.cat([vector(x + ".b", n, w, wp, "bias") for x, n, w, wp in (("q", H, d, dp), ("k", G, d, dp),
                                                                                        ("v", G, dv, dvp))])
        if m.out_bias:
            mx.o_bias = src.get(p + "o.b", (D,), "bias").float() * m.out_scale
        if m.qk_norm_all:
            mx.prep.q_norm, mx.prep.k_norm = (vector(x + ".norm", n, d, dp, "norm") for x, n in (("q", H), ("k", G)))
        elif m.qk_norm:
            mx.prep.q_norm, mx.prep.k_norm = (vector(x + ".norm", 1, d, dp, "norm") for x in "qk")
    elif m.kind == "latent_attention":
        mx.lat = _build_latent(mx, m, p, src, cfg, dtype)
    elif m.kind == "hgrn2":
        mx.parts = [("q", rows("q", H, d, dp)), ("f", rows("f", H, d, dp)), ("v", rows("v", H, dv, dvp))]
        norm = head_rows(src.get(p + "norm", (dv,), "norm").repeat(H), H, dv, dvp)
        mx.rec = recurrent.RecurrentParams(rule=m.kind, heads=H, dim_p=dp, vdim=dv, vdim_p=dvp, eps=cfg.rms_eps,
                                           norm_w=norm.float().contiguous(), f_bias=vector("f.b", H, d, dp, "bias"),
                                           f_lower=vector("lower", H, d, dp, "lower"))
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


def _build_latent(mx: Mixer, m: MixerSpec, p: str, src: WeightSource, cfg: ModelConfig, dtype: torch.dtype) -> latent.LatentParams:
    D, H, d, dp, rd, rp, R, Rp, dv, dvp = (cfg.hidden_size, m.heads, m.dim, m.dim_p, m.rot_dim, m.rot_p, m.kv_rank, m.rank_p, m.vdim,
                                           m.vdim_p)
    step = K_ALIGN if dtype == torch.bfloat16 else 8

    def gain(name, n):
        return torch.nn.functional.pad(src.get(p + name, (n,), "norm").float(), (0, pad_to(n, 8) - n)).contiguous()
    mx.parts = [("dq", src.get(p + "dq", (m.q_rank, D)))]
    own = m.kv_from < 0
    if own:
        dkv = src.get(p + "dkv", (R + rd, D))
        mx.parts += [("c", dkv[:R]), ("r", dkv[R:])]
    uq = src.get(p + "uq", (H * (d + rd), m.q_rank)).view(H, d + rd, m.q_rank)
    heads = uq.new_zeros(H, rp + dp, m.q_rank)                     # [rotated | rest]
    heads[:, :rd], heads[:, rp:rp + d] = uq[:, d:], uq[:, :d]
    uk = src.get(p + "uk", (H * d, R)).view(H, d, R)
    uv = src.get(p + "uv", (H * dv, R)).view(H, dv, R)
    w_uk = uk.new_zeros(H, Rp, pad_to(dp, step))
    w_uk[:, :R, :d] = uk.transpose(1, 2)
    w_uv = uv.new_zeros(H, dvp, pad_to(Rp, step))
    w_uv[:, :dv, :R] = uv
    w_up = None
    if dtype == torch.bfloat16:
        keys, values = (uk.new_zeros(H, n, pad_to(Rp + rp, step)) for n in (rp + dp, dvp))
        keys[:, torch.arange(rd), Rp + torch.arange(rd)] = 1.0      # the rotated part passes through, to every head
        keys[:, rp:rp + d, :R], values[:, :dv, :R] = uk, uv
        w_up = torch.cat([keys.flatten(0, 1), values.flatten(0, 1)]).to(dtype).contiguous()
    return latent.LatentParams(
        heads=H, dim_p=dp, rot_dim=rd, rot_p=rp, rank=R, rank_p=Rp, vdim_p=dvp, q_rank=m.q_rank, scale=m.scale, eps=cfg.rms_eps,
        window=m.window, sinks=src.get(p + "sink", (H,), "bias").float().contiguous(), q_norm=gain("dq.norm", m.q_rank),
        c_norm=gain("dkv.norm", R) if own else None, w_uq=pad_cols(heads.flatten(0, 1).to(dtype), pad_to(m.q_rank, K_ALIGN)).contiguous(),
        w_uk=w_uk.to(dtype).contiguous(), w_uv=w_uv.to(dtype).contiguous(), w_up=w_up)


def mixer_tensor_specs(m: MixerSpec, p: str, D: int, layer: int) -> List[Tuple[str, Tuple[int, ...], str, int]]:
    """(name, shape, init kind, layer) of a mixer's checkpoint tensors."""
    qk, kv, n, H = m.heads * m.dim, m.qk_heads * m.dim, m.heads * m.vdim, m.heads
    if m.kind == "attention":
        out = [("q", (qk, D), "normal"), ("k", (kv, D), "normal"), ("v", (m.kv_heads * m.vdim, D), "normal")]
        out += [("talk", (H, H), "normal")] if m.talking else []
        out += [("g", (H, D), "normal")] if m.out_gate else []
        out += [("g", (n, D), "normal")] if m.out_gate_all else []
        out += [("q.b", (qk,), "bias"), ("k.b", (kv,), "bias"), ("v.b", (m.kv_heads * m.vdim,), "bias")] if m.bias else []
        out += [("o.b", (D,), "bias")] if m.out_bias else []
        out += [("q.norm", (m.dim,), "norm"), ("k.norm", (m.dim,), "norm")] if m.qk_norm else []
        out += [("q.norm", (qk,), "norm"), ("k.norm", (kv,), "norm")] if m.qk_norm_all else []
        out += [("sink", (H,), "bias")] if m.head_sinks else []
    elif m.kind == "latent_attention":
        out = [("dq", (m.q_rank, D), "normal"), ("dq.norm", (m.q_rank,), "norm"), ("uq", (H * (m.dim + m.rot_dim), m.q_rank), "normal"),
               ("uk", (qk, m.kv_rank), "normal"), ("uv", (n, m.kv_rank), "normal"), ("sink", (H,), "bias")]
        if m.kv_from < 0:
            out += [("dkv", (m.kv_rank + m.rot_dim, D), "normal"), ("dkv.norm", (m.kv_rank,), "norm")]
    elif m.kind == "hgrn2":
        out = [("q", (qk, D), "normal"), ("f", (qk, D), "normal"), ("f.b", (qk,), "bias"), ("lower", (qk,), "lower"), ("v", (n, D), "normal"),
               ("norm", (m.vdim,), "norm")]
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
