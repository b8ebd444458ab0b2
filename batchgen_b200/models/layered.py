"""Layer-listed decoders (``ModelConfig.layer_specs``): every layer names its own token mixer and feed-forward, both read
one norm of an fp32 residual stream, and their outputs are added together (parallel block).  Nanurax is the family built
this way: generalised delta-rule layers (recurrent state per sequence) and chunked talking-heads attention layers (paged
KV), dense tanh-GELU or input-weighted clamped-SwiGLU mixture feed-forwards.

Same calling contract as ``Transformer``: ``forward(ids [T], meta, cache) -> fp32 logits``; all state lives in the caller's
``PagedKVCache`` (paged rows per attention layer, ``FlatStatePool`` slots for the recurrent layers), and a step may mix
pieces of prompts with single decoded tokens (``AttnMeta`` mode "prefill") or decode one token per sequence (mode "decode",
graph capturable).

A layer runs as: residual sum + norm (one kernel, which also adds the previous layer's outputs) -> one GEMM for everything
that reads the norm (mixer projections, router, shared-expert gate, dense or shared gate / up) -> the mixer's core and the
gated activation, written side by side -> one GEMM against [W_o | W_down], whose fp32 output is the layer's addend.  Routed
experts add their rows in the next residual kernel.  GEMM outputs stay fp32: what enters the recurrence, the scores, the
router and the residual sum is never rounded to 16 bits; GEMM operands are bf16, or fp32 in the 32-bit form of the model.

Widths: the contraction side of every operand is padded with zeros to a multiple of 64 (one TMA / MMA block), head widths
to multiples of 8, so any model size runs on the same kernels.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from ..config import LayerSpec, ModelConfig
from ..ops import delta, gemm, residual, talking
from ..ops import moe as moe_ops
from ..ops.moe import ExpertWeights
from ..ops.residual import pad_to
from ..utils.timing import null_timer
from .transformer import AttnMeta
from .weights import ParallelLayout, WeightSource

DECAY_SCALE = math.exp(-0.5)       # decay = exp(-DECAY_SCALE * sigmoid(.)), so a channel keeps at least exp(-exp(-1/2)) a step
K_ALIGN = 64


@dataclass
class LayeredLayer:
    spec: LayerSpec = None
    norm: torch.Tensor = None                     # [width] fp32
    w_in: torch.Tensor = None                     # [sum of segments, width_p]
    seg: Dict[str, Tuple[int, int]] = field(default_factory=dict)     # name -> (first column of the GEMM output, width)
    w_out: torch.Tensor = None                    # [width, mix_p + ff_p]: [W_o | W_down]
    mix_cols: int = 0                             # columns the mixer writes
    mix_p: int = 0                                # the same, padded to K_ALIGN
    ff_p: int = 0
    w_decay: torch.Tensor = None                  # delta: [heads * dim_p, rank_p], second factor of the decay projection
    delta: Optional[delta.DeltaParams] = None
    talk: Optional[talking.TalkParams] = None
    experts: Optional[ExpertWeights] = None


@dataclass
class LayeredWeights:
    embed: torch.Tensor = None                    # [vocab, width]
    final_norm: torch.Tensor = None
    lm_head: torch.Tensor = None                  # [vocab, width_p]
    layers: List[LayeredLayer] = field(default_factory=list)


def _pad_cols(w: torch.Tensor, cols: int) -> torch.Tensor:
    return w if w.shape[1] == cols else torch.nn.functional.pad(w, (0, cols - w.shape[1]))


def _pad_rows(w: torch.Tensor, rows: int) -> torch.Tensor:
    return w if w.shape[0] == rows else torch.nn.functional.pad(w, (0, 0, 0, rows - w.shape[0]))


def _head_rows(w: torch.Tensor, heads: int, d: int, dp: int) -> torch.Tensor:
    """[heads * d, ...] -> [heads * dp, ...]: zero rows behind every head."""
    if d == dp:
        return w
    out = w.new_zeros(heads, dp, *w.shape[1:])
    out[:, :d] = w.view(heads, d, *w.shape[1:])
    return out.view(heads * dp, *w.shape[1:])


def build_layered_weights(cfg: ModelConfig, layout: ParallelLayout, src: WeightSource, dtype: torch.dtype) -> LayeredWeights:
    """Tensor names follow the published checkpoint (``l<i>.mix.*``, ``l<i>.mlp.*``)."""
    if layout.tp_size > 1 or layout.ep_size > 1:
        raise NotImplementedError("layer-listed models run on one GPU per engine: use data-parallel cohorts (--dp-size)")
    D, V = cfg.hidden_size, cfg.vocab_size
    Kp = pad_to(D, K_ALIGN)
    w = LayeredWeights()
    w.embed = src.get("embed", (V, D)).to(dtype).contiguous()
    w.final_norm = src.get("final.norm", (D,), "norm").float().contiguous()
    w.lm_head = _pad_cols(src.get("head", (V, D)).to(dtype), Kp).contiguous()
    for i, spec in enumerate(cfg.layer_specs):
        m, f, p = spec.mixer, spec.mlp, f"l{i}.mix."
        lw = LayeredLayer(spec=spec, norm=src.get(f"l{i}.norm1", (D,), "norm").float().contiguous())
        parts: List[Tuple[str, torch.Tensor]] = []
        if m.recurrent:
            n, H, d, dp = m.heads * m.dim, m.heads, m.dim, m.dim_p
            parts += [(x, _head_rows(src.get(p + x, (n, D)), H, d, dp)) for x in ("r", "k", "v", "g", "a")]
            parts.append(("low", src.get(p + "w1", (m.decay_rank, D))))
            vec = lambda name, kind: _head_rows(src.get(p + name, (n,), kind).float(), H, d, dp).contiguous()   # noqa: E731
            lw.delta = delta.DeltaParams(w0=vec("w0", "bias"), ab=vec("a.b", "bias"), norm_w=vec("norm", "norm"), heads=H,
                                         dim=d, dim_p=dp, decay_scale=DECAY_SCALE, eps=cfg.rms_eps)
            w2 = _head_rows(src.get(p + "w2", (n, m.decay_rank)), H, d, dp)
            lw.w_decay = _pad_cols(w2.to(dtype), pad_to(m.decay_rank, K_ALIGN)).contiguous()
            o = src.get(p + "o", (D, n))
            heads_o, d_o, dp_o = H, d, dp
        else:
            H, G = m.heads, m.kv_heads
            parts += [("q", _head_rows(src.get(p + "q", (H * m.dim, D)), H, m.dim, m.dim_p)),
                      ("k", _head_rows(src.get(p + "k", (G * m.dim, D)), G, m.dim, m.dim_p)),
                      ("v", _head_rows(src.get(p + "v", (G * m.vdim, D)), G, m.vdim, m.vdim_p))]
            talk = src.get(p + "talk", (H, H)).float().contiguous() if m.talking else None
            lw.talk = talking.TalkParams(heads=H, kv_heads=G, dim_p=m.dim_p, vdim_p=m.vdim_p, scale=m.scale, chunk=m.chunk,
                                         sink=m.sink, talk=talk)
            o = src.get(p + "o", (D, H * m.vdim))
            heads_o, d_o, dp_o = H, m.vdim, m.vdim_p
        o = _head_rows(o.t().contiguous(), heads_o, d_o, dp_o).t()                  # [D, heads * dp]: zero columns
        lw.mix_cols = heads_o * dp_o
        lw.mix_p = pad_to(lw.mix_cols, K_ALIGN)
        outs = [_pad_cols(o, lw.mix_p)]
        q = f"l{i}.mlp."
        ff, prefix = (f.ff, q) if f.kind == "dense" else (f.shared_ff, q + "shared.") if f.kind == "moe" else (0, "")
        if f.kind == "moe":
            parts.append(("router", src.get(q + "router", (f.experts, D))))
            if ff:
                parts.append(("gate1", src.get(prefix + "sg", (1, D))))
            Fp = pad_to(f.ff, K_ALIGN)
            w13, wd = [], []
            for e in range(f.experts):
                ep = f"{q}e{e}."
                gu = [_pad_rows(src.get(ep + x, (f.ff, D)).to(dtype), Fp) for x in ("gate", "up")]
                w13.append(_pad_cols(torch.cat(gu, 0), Kp))
                wd.append(_pad_cols(src.get(ep + "down", (D, f.ff)).to(dtype), Fp))
            lw.experts = ExpertWeights(w13=torch.stack(w13), w2=torch.stack(wd), activation=f.activation, act_limit=f.limit)
        if ff:
            lw.ff_p = pad_to(ff, K_ALIGN)
            parts += [(x, _pad_rows(src.get(prefix + x, (ff, D)), lw.ff_p)) for x in ("gate", "up")]
            outs.append(_pad_cols(src.get(prefix + "down", (D, ff)), lw.ff_p))
        row, stack = 0, []
        for name, t in parts:
            lw.seg[name] = (row, t.shape[0])
            stack.append(_pad_rows(t.to(dtype), pad_to(t.shape[0], 8)))
            row += stack[-1].shape[0]
        lw.w_in = _pad_cols(torch.cat(stack, 0), Kp).contiguous()
        lw.w_out = torch.cat([t.to(dtype) for t in outs], 1).contiguous()
        w.layers.append(lw)
    return w


def layered_tensor_specs(cfg: ModelConfig) -> List[Tuple[str, Tuple[int, ...], str, int]]:
    """(name, shape, init kind, layer) of every checkpoint tensor (layer -1: embedding, final norm, head)."""
    D, V = cfg.hidden_size, cfg.vocab_size
    out = [("embed", (V, D), "normal", -1), ("final.norm", (D,), "norm", -1), ("head", (V, D), "normal", -1)]
    for i, s in enumerate(cfg.layer_specs):
        m, f, p, q = s.mixer, s.mlp, f"l{i}.mix.", f"l{i}.mlp."
        out.append((f"l{i}.norm1", (D,), "norm", i))
        if m.recurrent:
            n = m.heads * m.dim
            out += [(p + x, (n, D), "normal", i) for x in ("r", "k", "v", "g", "a")]
            out += [(p + "w1", (m.decay_rank, D), "normal", i), (p + "w2", (n, m.decay_rank), "normal", i),
                    (p + "a.b", (n,), "bias", i), (p + "w0", (n,), "bias", i), (p + "norm", (n,), "norm", i),
                    (p + "o", (D, n), "normal", i)]
        else:
            out += [(p + "q", (m.heads * m.dim, D), "normal", i), (p + "k", (m.kv_heads * m.dim, D), "normal", i),
                    (p + "v", (m.kv_heads * m.vdim, D), "normal", i), (p + "o", (D, m.heads * m.vdim), "normal", i)]
            if m.talking:
                out.append((p + "talk", (m.heads, m.heads), "normal", i))

        def ff(prefix, n):
            return [(prefix + "gate", (n, D), "normal", i), (prefix + "up", (n, D), "normal", i),
                    (prefix + "down", (D, n), "normal", i)]
        if f.kind == "dense":
            out += ff(q, f.ff)
        elif f.kind == "moe":
            out.append((q + "router", (f.experts, D), "normal", i))
            for e in range(f.experts):
                out += ff(f"{q}e{e}.", f.ff)
            if f.shared_ff:
                out += ff(q + "shared.", f.shared_ff) + [(q + "shared.sg", (1, D), "normal", i)]
    return out


@dataclass
class _Plan:
    """Device tables of one step, shared by its layers."""
    lens: torch.Tensor                            # [T] int32: position + 1 (0 = padding row)
    row_seq: Optional[torch.Tensor]               # [T] int32 block-table row of each token, None = identity
    cu: Optional[torch.Tensor]                    # [nseq + 1] int32, None = one token per sequence
    cu_host: Optional[List[int]]
    slots: Optional[torch.Tensor]
    has_initial: Optional[torch.Tensor]
    ctx: Optional[List[int]] = None
    tiles: Dict[int, Tuple] = field(default_factory=dict)      # attention chunk -> (tensor-core tiles, rows of short pieces)


class LayeredDecoder:
    def __init__(self, cfg: ModelConfig, weights: LayeredWeights, layout: Optional[ParallelLayout] = None, comm=None,
                 max_positions: int = 0):
        assert cfg.is_layered
        self.cfg, self.w, self.comm = cfg, weights, comm
        self.layout = layout or ParallelLayout()
        self.device = weights.embed.device
        self.dtype = weights.embed.dtype
        self.width_p = weights.lm_head.shape[1]
        self.timer = null_timer()
        self.attn_request_parallel = False
        self.streamer = None
        self.layer_hook = None                    # called with (layer, residual stream [T, width]) after every layer

    # ------------------------------------------------------------------ step tables
    def _plan(self, meta: AttnMeta, T: int) -> _Plan:
        if meta.mode == "decode":
            return _Plan(meta.seqlens, None, None, None, meta.state_slots, None)
        dev = self.device
        cu = meta.cu_seqlens
        cu_t = torch.tensor(cu, dtype=torch.int32, device=dev)
        counts = torch.tensor([b - a for a, b in zip(cu, cu[1:])], device=dev)
        row_seq = torch.repeat_interleave(torch.arange(len(cu) - 1, dtype=torch.int32, device=dev), counts, output_size=T)
        return _Plan((meta.positions + 1).to(torch.int32), row_seq, cu_t, list(cu), meta.state_slots, meta.state_has_initial,
                     list(meta.ctx_lens))

    def _tiles(self, plan: _Plan, chunk: int, T: int):
        """How the rows of a prompt step split over the attention kernels: pieces of a few tokens (decoded tokens among
        them) go row by row, the rest in 128-query tiles."""
        if chunk not in plan.tiles:
            cu, least = plan.cu_host, talking.PREFILL_MIN_TOKENS
            blocks = talking.work_blocks(talking.prefill_work(cu, plan.ctx, chunk, least), T, self.device)
            short = [t for a, b in zip(cu, cu[1:]) if b - a < least for t in range(a, b)]
            rows = seqs = None
            if blocks and short:
                rows = torch.tensor(short, dtype=torch.int32, device=self.device)
                seqs = plan.row_seq[rows.long()].contiguous()
            elif short:
                seqs = plan.row_seq
            plan.tiles[chunk] = (blocks, bool(short), rows, seqs)
        return plan.tiles[chunk]

    # ------------------------------------------------------------------ mixers
    def _delta(self, l: int, lw: LayeredLayer, z, out, plan: _Plan, cache) -> None:
        o, n = lw.seg["low"]
        low = residual.cast_act(z[:, o:o + n], lw.w_decay.shape[1], self.dtype, tanh=True)
        wl = gemm.rows_gemm(low, lw.w_decay)
        if plan.slots is None:
            raise RuntimeError("a model with recurrent layers needs AttnMeta.state_slots")
        delta.delta_forward(z, tuple(lw.seg[x][0] for x in ("r", "k", "v", "g", "a")), wl, lw.delta, cache.state.layer(l),
                            plan.slots, out, plan.cu, plan.cu_host, plan.has_initial)

    def _attention(self, l: int, lw: LayeredLayer, z, out, plan: _Plan, meta: AttnMeta, cache) -> None:
        q, k = lw.seg["q"], lw.seg["k"][0]
        kv = cache.latent(l)
        talking.kv_write(z[:, k:k + lw.talk.kv_row], meta.slot_mapping, kv)
        zq = z[:, q[0]:q[0] + q[1]]
        rows, seqs = None, plan.row_seq
        if plan.cu is not None and z.is_cuda and talking.prefill_supported(lw.talk, kv.dtype, kv.shape[1]):
            blocks, short, rows, seqs = self._tiles(plan, lw.talk.chunk, z.shape[0])
            talking.attend_prefill(zq, lw.talk, kv, meta.block_table, out, blocks)
            if not short:
                return
        talking.attend_rows(zq, lw.talk, kv, meta.block_table, plan.lens, out, seqs, rows)

    # ------------------------------------------------------------------ forward
    def forward(self, ids: torch.Tensor, meta: AttnMeta, cache) -> torch.Tensor:
        """ids [T] -> fp32 logits [len(logit_rows) or T, vocab]."""
        cfg, tm, w = self.cfg, self.timer, self.w
        T, D = ids.shape[0], cfg.hidden_size
        dev, dt = self.device, self.dtype
        plan = self._plan(meta, T)
        x = torch.empty(T, pad_to(D, 4), dtype=torch.float32, device=dev)
        first = dict(ids=ids.to(torch.int32), embed=w.embed, embed_scale=cfg.embed_scale)
        add = routed = pos = None
        for l, lw in enumerate(w.layers):
            f = lw.spec.mlp
            with tm.timed("norm", l):
                h = residual.residual_norm(x, lw.norm, cfg.rms_eps, D, self.width_p, dt, add=add, routed=routed, pos=pos,
                                           **first)
            if self.layer_hook is not None and l:
                self.layer_hook(l - 1, x[:, :D])
            first = {}
            with tm.timed("proj_in", l):
                z = gemm.rows_gemm(h, lw.w_in)
            padded = lw.mix_cols != lw.mix_p
            cat = (torch.zeros if padded else torch.empty)(T, lw.mix_p + lw.ff_p, dtype=dt, device=dev)
            with tm.timed("mixer_" + meta.mode, l):
                if lw.delta is not None:
                    self._delta(l, lw, z, cat[:, :lw.mix_cols], plan, cache)
                else:
                    self._attention(l, lw, z, cat[:, :lw.mix_cols], plan, meta, cache)
            if lw.ff_p:
                g0, s = lw.seg["gate"][0], lw.seg.get("gate1")
                with tm.timed("glu", l):
                    residual.glu(z[:, g0:], lw.ff_p, f.activation, f.limit if f.kind == "dense" else f.shared_limit,
                                 gate=None if s is None else z[:, s[0]:s[0] + 1], out=cat[:, lw.mix_p:])
            routed = pos = None
            if lw.experts is not None:
                r0 = lw.seg["router"][0]
                with tm.timed("moe", l):
                    idx, rw = moe_ops.router_topk(z[:, r0:r0 + f.experts], None, f.top, norm_topk_prob=False,
                                                  scoring="sigmoid", num_valid=meta.num_valid)
                    routed, pos = moe_ops.routed_rows(h, idx, rw, lw.experts, f.weight_on_input, meta.num_valid)
            with tm.timed("proj_out", l):
                add = gemm.rows_gemm(cat, lw.w_out)
        if self.layer_hook is not None:           # the last layer's outputs are only summed inside the final norm
            residual.residual_norm(x, w.final_norm, cfg.rms_eps, D, self.width_p, dt, add=add, routed=routed, pos=pos)
            add = routed = pos = None
            self.layer_hook(len(w.layers) - 1, x[:, :D])
        y = residual.residual_norm(x, w.final_norm, cfg.rms_eps, D, self.width_p, dt, add=add, routed=routed, pos=pos,
                                   rows=meta.logit_rows.long() if meta.logit_rows is not None else None, keep=False)
        with tm.timed("lm_head"):
            return gemm.rows_gemm(y, w.lm_head)
