"""Layer-listed decoders (``ModelConfig.layer_specs``): every layer names its own token mixer(s) and feed-forward around an
fp32 residual stream.  Three block forms:

* parallel (Nanurax): mixer and feed-forward read one RMS norm and their outputs are added together.  Generalised delta-rule
  layers and chunked talking-heads attention layers, dense tanh-GELU or input-weighted clamped-SwiGLU mixture feed-forwards.
* sandwich (Pamevik, Pitudra, ``ModelConfig.sandwich``): mixer, then feed-forward, each between two norms (``layer_norm``: with mean
  and bias; ``pre_norm`` off: only the output's) and behind an input convolution (``canon_taps``), or the mixer behind a shift towards
  the previous token (``token_shift``); a gated row of a table per token may follow (``side_dim``).  mLSTM, gated delta-rule with a
  decay per channel, and softmax attention beside retention, squared-ReLU feed-forwards; or HGRN2, windowed attention with sinks and
  attention over latents that layers may share, mixtures of squared-ReLU experts.
* hyper-connected (Bolisun, ``ModelConfig.streams``): mixer, then feed-forward, each behind an RMS norm that reads a weighted sum of
  several residual streams; its output joins all streams, which are mixed with one another.  Windowed attention with normed heads
  beside retention; clamped-SwiGLU feed-forwards and mixtures of experts; layers may share their weights.

Same calling contract as ``Transformer``: ``forward(ids [T], meta, cache) -> fp32 logits``; all state lives in the caller's
``PagedKVCache`` (paged rows per attention layer, ``FlatStatePool`` slots for everything else a sequence carries), and a step
may mix pieces of prompts with single decoded tokens (``AttnMeta`` mode "prefill") or decode one token per sequence (mode
"decode", graph capturable).

A parallel block runs as: residual sum + norm (one kernel, which also adds the previous layer's outputs) -> one GEMM for
everything that reads the norm (mixer projections, router, shared-expert gate, dense or shared gate / up) -> the mixer's core
and the gated activation, written side by side -> one GEMM against [W_o | W_down], whose fp32 output is the layer's addend.
Routed experts add their rows in the next residual kernel.  A sandwich block runs every sublayer as: norm of the previous
sublayer's output + residual sum + norm + input convolution (one kernel in decode, two in prompts) -> one GEMM for everything
that reads it -> core or activation -> one GEMM per output projection, whose fp32 output goes to the next norm kernel.  A hyper-
connected block does the same with one GEMM against both mixers' output projections side by side (their scales are in the
operands), and its norm kernel mixes the streams and gathers the routed experts' rows.  GEMM outputs stay fp32: what enters the recurrence, the scores, the router and the residual sum is never rounded to 16 bits; GEMM
operands are bf16, or fp32 in the 32-bit form of the model.

Widths: the contraction side of every operand is padded with zeros to a multiple of 64 (one TMA / MMA block), head widths
to multiples of 8, so any model size runs on the same kernels.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from ..config import LayerSpec, MlpSpec, ModelConfig
from ..ops import conv, gemm, residual
from ..ops import moe as moe_ops
from ..ops.moe import ExpertWeights
from ..ops.residual import pad_to
from ..utils.timing import null_timer
from .mixers import K_ALIGN, Mixer, StepPlan, build_mixer, mixer_tensor_specs, pad_cols, pad_rows, stack_parts
from .transformer import AttnMeta
from .weights import ParallelLayout, WeightSource


@dataclass
class LayeredLayer:
    """A parallel block."""
    spec: LayerSpec = None
    norm: torch.Tensor = None                     # [width] fp32
    w_in: torch.Tensor = None                     # [sum of segments, width_p]
    seg: Dict[str, Tuple[int, int]] = field(default_factory=dict)     # feed-forward part -> (first column of the GEMM output, width)
    w_out: torch.Tensor = None                    # [width, mix_p + ff_p]: [W_o | W_down]
    mix_p: int = 0                                # columns the mixer writes, padded to K_ALIGN
    ff_p: int = 0
    mixer: Mixer = None
    experts: Optional[ExpertWeights] = None


@dataclass
class Sublayer:
    """One half of a sandwich or hyper-connected block: mixer(s) side by side, or a feed-forward."""
    norm: Optional[residual.Norm]
    post: Optional[residual.Norm]                 # sandwich: norm of the output
    w_in: torch.Tensor                            # [columns, width_p]
    w_out: List[torch.Tensor]                     # per mixer W_o (hyper-connected: one matrix), or [W_down]: [width, operand width
                                                  # padded to K_ALIGN]
    mixers: List[Mixer] = field(default_factory=list)       # empty: feed-forward
    branch_w: Optional[Tuple[torch.Tensor, torch.Tensor]] = None      # weights of two mixers' output norms
    canon_w: Optional[torch.Tensor] = None        # [taps, width4] fp32 input convolution (a token shift is one of two taps)
    canon_part: str = ""                          # its state part
    ff: int = 0                                   # width of the dense or shared feed-forward (hyper-connected: padded to K_ALIGN)
    hc: Optional[residual.Hyper] = None           # hyper-connected blocks, with what follows
    bias: Optional[torch.Tensor] = None           # [width4] fp32, added to the output
    mlp: Optional[MlpSpec] = None
    seg: Dict[str, Tuple[int, int]] = field(default_factory=dict)     # feed-forward part -> (first column of the GEMM output, width)
    correction: Optional[torch.Tensor] = None     # [experts] fp32
    experts: Optional[ExpertWeights] = None
    side: Optional[torch.Tensor] = None           # [vocab, side dim] (a column view): this sublayer is the token's side input


@dataclass
class LayeredWeights:
    embed: torch.Tensor = None                    # [vocab, width]
    final_norm: torch.Tensor = None               # fp32 gain, or a ``residual.Norm`` (sandwich, hyper-connected)
    lm_head: torch.Tensor = None                  # [vocab, width_p]
    layers: List = field(default_factory=list)    # LayeredLayer, or lists of Sublayers
    side: Optional[torch.Tensor] = None           # [vocab, layers * side dim]


def build_layered_weights(cfg: ModelConfig, layout: ParallelLayout, src: WeightSource, dtype: torch.dtype) -> LayeredWeights:
    """Tensor names follow the published checkpoint (``l<i>.mix.*``, ``l<i>.mlp.*``)."""
    if layout.tp_size > 1 or layout.ep_size > 1:
        raise NotImplementedError("layer-listed models run on one GPU per engine: use data-parallel cohorts (--dp-size)")
    D, V = cfg.hidden_size, cfg.vocab_size
    Kp = pad_to(D, K_ALIGN)
    w = LayeredWeights()
    w.embed = src.get("embed", (V, D)).to(dtype).contiguous()
    w.final_norm = (_norm(src, "final.norm", cfg) if cfg.sandwich or cfg.streams
                    else src.get("final.norm", (D,), "norm").float().contiguous())
    w.lm_head = pad_cols(w.embed if cfg.tie_word_embeddings else src.get("head", (V, D)).to(dtype), Kp).contiguous()
    if cfg.side_dim:
        w.side = src.get("side.embed", (V, cfg.num_layers * cfg.side_dim)).to(dtype).contiguous()
    block = _build_hyper if cfg.streams else _build_sandwich if cfg.sandwich else _build_parallel
    own = {i: block(cfg, spec, f"l{i}.", src, dtype) for i, spec in enumerate(cfg.layer_specs) if spec.weights_of < 0}
    w.layers = [own[i if spec.weights_of < 0 else spec.weights_of] for i, spec in enumerate(cfg.layer_specs)]
    if cfg.side_dim:
        for i, layer in enumerate(w.layers):
            layer.append(_build_side(cfg, f"l{i}.", src, dtype, w.side[:, i * cfg.side_dim:(i + 1) * cfg.side_dim]))
    return w


def _vec(src: WeightSource, name: str, kind: str, D: int) -> torch.Tensor:
    return torch.nn.functional.pad(src.get(name, (D,), kind).float(), (0, pad_to(D, 4) - D)).contiguous()


def _norm(src: WeightSource, name: str, cfg: ModelConfig) -> residual.Norm:
    D = cfg.hidden_size
    return residual.Norm(_vec(src, name, "norm", D), _vec(src, name + ".b", "bias", D) if cfg.layer_norm else None, cfg.layer_norm)


def _build_side(cfg: ModelConfig, p: str, src: WeightSource, dtype: torch.dtype, table: torch.Tensor) -> Sublayer:
    D, n = cfg.hidden_size, cfg.side_dim
    gate = pad_cols(pad_rows(src.get(p + "side.gate", (n, D)).to(dtype), pad_to(n, 8)), pad_to(D, K_ALIGN)).contiguous()
    proj = pad_cols(src.get(p + "side.proj", (D, n)).to(dtype), pad_to(n, K_ALIGN)).contiguous()
    return Sublayer(None, residual.Norm(_vec(src, p + "side.norm", "norm", D)), gate, [proj], side=table)


def _build_sandwich(cfg: ModelConfig, spec: LayerSpec, p: str, src: WeightSource, dtype: torch.dtype) -> List[Sublayer]:
    D, f = cfg.hidden_size, spec.mlp
    Kp, W4 = pad_to(D, K_ALIGN), pad_to(D, 4)
    if f.kind not in ("none", "dense", "moe") or (f.kind != "none" and f.activation != "relu2") or f.shared_ff or f.correction:
        raise NotImplementedError("sandwich blocks carry squared-ReLU feed-forwards and mixtures of them without a shared one")
    prefixes = [p + "mix."] if spec.second is None else [p + "mix.left.", p + "mix.right."]
    mixers = [build_mixer(m, q, src, cfg, dtype, i) for i, (m, q) in enumerate(zip(spec.mixers, prefixes))]
    out = []
    for n in (1, 2) if f.kind != "none" else (1,):
        if cfg.pre_norm:
            s = Sublayer(_norm(src, f"{p}norm{n}", cfg), _norm(src, f"{p}norm{n}b", cfg), None, [])
        else:
            s = Sublayer(None, _norm(src, f"{p}norm{n}", cfg), None, [])
        if cfg.canon_taps:
            s.canon_part = f"canon{n}"
            taps = src.get(f"{p}canon{n}", (D, cfg.canon_taps)).float()
            s.canon_w = pad_rows(taps, W4).t().contiguous()
        elif cfg.token_shift and n == 1:
            s.canon_part, mu = "shift", _vec(src, p + "shift", "shift", D)
            s.canon_w = torch.stack([mu, -mu])                      # h + mu h' - mu h
        if n == 1:
            s.mixers = mixers
            s.w_in = stack_parts([(m.seg, name, t) for m in mixers for name, t in m.parts], Kp, dtype)
            s.w_out = [pad_cols(m.o.to(dtype), pad_to(m.cols, K_ALIGN)).contiguous() for m in mixers]
            for m in mixers:
                m.parts, m.o = [], None
            if spec.second is not None:
                s.branch_w = tuple(torch.nn.functional.pad(src.get(q + "out", (D,), "norm").float(), (0, W4 - D)).contiguous()
                                   for q in prefixes)
        elif f.kind == "moe":
            s.mlp = f
            s.w_in = stack_parts([(s.seg, "router", src.get(p + "mlp.router", (f.experts, D)))], Kp, dtype)
            s.w_out = []
            s.experts = _experts(f, p + "mlp.", src, D, dtype)
        else:
            s.ff = f.ff
            s.w_in = pad_cols(pad_rows(src.get(p + "mlp.up", (f.ff, D)).to(dtype), pad_to(f.ff, 8)), Kp).contiguous()
            s.w_out = [pad_cols(src.get(p + "mlp.down", (D, f.ff)).to(dtype), pad_to(f.ff, K_ALIGN)).contiguous()]
        out.append(s)
    return out


def _experts(f: MlpSpec, q: str, src: WeightSource, D: int, dtype: torch.dtype) -> ExpertWeights:
    Kp, Fp = pad_to(D, K_ALIGN), pad_to(f.ff, K_ALIGN)
    w13, wd = [], []
    for e in range(f.experts):
        ep = f"{q}e{e}."
        gu = [pad_rows(src.get(ep + x, (f.ff, D)).to(dtype), Fp) for x in (("up",) if f.activation == "relu2" else ("gate", "up"))]
        w13.append(pad_cols(torch.cat(gu, 0), Kp))
        wd.append(pad_cols(src.get(ep + "down", (D, f.ff)).to(dtype), Fp))
    return ExpertWeights(w13=torch.stack(w13), w2=torch.stack(wd), activation=f.activation, act_limit=f.limit)


def _build_hyper(cfg: ModelConfig, spec: LayerSpec, p: str, src: WeightSource, dtype: torch.dtype) -> List[Sublayer]:
    D, f, S = cfg.hidden_size, spec.mlp, cfg.streams
    Kp, W4 = pad_to(D, K_ALIGN), pad_to(D, 4)

    def sublayer(n):
        hc = [src.get(f"{p}hc{n}.{x}", shape, kind).float().contiguous()
              for x, shape, kind in (("in", (S,), "norm"), ("mix", (S, S), "mix"), ("out", (S,), "norm"))]
        return Sublayer(_norm(src, f"{p}norm{n}", cfg), None, None, [], hc=residual.Hyper(*hc))
    s = sublayer(1)
    prefixes = [p + "mix."] if spec.second is None else [p + "mix.left.", p + "mix.right."]
    s.mixers = [build_mixer(m, q, src, cfg, dtype, i) for i, (m, q) in enumerate(zip(spec.mixers, prefixes))]
    s.w_in = stack_parts([(m.seg, name, t) for m in s.mixers for name, t in m.parts], Kp, dtype)
    s.w_out = [torch.cat([pad_cols(m.o.to(dtype), pad_to(m.cols, K_ALIGN)) for m in s.mixers], 1).contiguous()]
    for m in s.mixers:
        m.parts, m.o = [], None
        if m.o_bias is not None:
            b = torch.nn.functional.pad(m.o_bias, (0, W4 - D))
            s.bias, m.o_bias = b if s.bias is None else s.bias + b, None
    out = [s]
    if f.kind == "none":
        return out
    s = sublayer(2)
    s.mlp, q, parts = f, p + "mlp.", []
    ff, prefix = (f.ff, q) if f.kind == "dense" else (f.shared_ff, q + "shared.")
    if f.kind == "moe":
        parts.append((s.seg, "router", src.get(q + "router", (f.experts, D))))
        if f.correction:
            s.correction = src.get(q + "correction", (f.experts,), "bias").float().contiguous()
        s.experts = _experts(f, q, src, D, dtype)
        if ff and f.shared_gate:
            raise NotImplementedError("hyper-connected blocks carry shared experts without a gate")
    if ff:
        s.ff = pad_to(ff, K_ALIGN)
        parts += [(s.seg, x, pad_rows(src.get(prefix + x, (ff, D)), s.ff)) for x in ("gate", "up")]
        s.w_out = [pad_cols(src.get(prefix + "down", (D, ff)).to(dtype), s.ff).contiguous()]
    s.w_in = stack_parts(parts, Kp, dtype)
    return out + [s]


def _build_parallel(cfg: ModelConfig, spec: LayerSpec, p: str, src: WeightSource, dtype: torch.dtype) -> LayeredLayer:
    D, f = cfg.hidden_size, spec.mlp
    Kp = pad_to(D, K_ALIGN)
    lw = LayeredLayer(spec=spec, norm=src.get(p + "norm1", (D,), "norm").float().contiguous())
    mx = lw.mixer = build_mixer(spec.mixer, p + "mix.", src, cfg, dtype)
    parts = [(mx.seg, name, t) for name, t in mx.parts]
    lw.mix_p = pad_to(mx.cols, K_ALIGN)
    outs = [pad_cols(mx.o, lw.mix_p)]
    mx.parts, mx.o = [], None
    q = p + "mlp."
    ff, prefix = (f.ff, q) if f.kind == "dense" else (f.shared_ff, q + "shared.") if f.kind == "moe" else (0, "")
    if f.kind == "moe":
        parts.append((lw.seg, "router", src.get(q + "router", (f.experts, D))))
        if ff:
            parts.append((lw.seg, "gate1", src.get(prefix + "sg", (1, D))))
        lw.experts = _experts(f, q, src, D, dtype)
    if ff:
        lw.ff_p = pad_to(ff, K_ALIGN)
        parts += [(lw.seg, x, pad_rows(src.get(prefix + x, (ff, D)), lw.ff_p)) for x in ("gate", "up")]
        outs.append(pad_cols(src.get(prefix + "down", (D, ff)), lw.ff_p))
    lw.w_in = stack_parts(parts, Kp, dtype)
    lw.w_out = torch.cat([t.to(dtype) for t in outs], 1).contiguous()
    return lw


def layered_tensor_specs(cfg: ModelConfig) -> List[Tuple[str, Tuple[int, ...], str, int]]:
    """(name, shape, init kind, layer) of every checkpoint tensor (layer -1: embedding, final norm, head)."""
    D, V = cfg.hidden_size, cfg.vocab_size

    def norm(name, l):
        return [(name, (D,), "norm", l)] + ([(name + ".b", (D,), "bias", l)] if cfg.layer_norm else [])
    out = [("embed", (V, D), "normal", -1), *norm("final.norm", -1)]
    out += [] if cfg.tie_word_embeddings else [("head", (V, D), "normal", -1)]
    out += [("side.embed", (V, cfg.num_layers * cfg.side_dim), "normal", -1)] if cfg.side_dim else []
    for i, s in enumerate(cfg.layer_specs):
        if s.weights_of >= 0:
            continue
        f, q = s.mlp, f"l{i}.mlp."
        prefixes = [f"l{i}.mix."] if s.second is None else [f"l{i}.mix.left.", f"l{i}.mix.right."]
        if cfg.sandwich:
            for n in ("1", "2") if f.kind != "none" else ("1",):
                out += norm(f"l{i}.norm{n}", i) + (norm(f"l{i}.norm{n}b", i) if cfg.pre_norm else [])
                if cfg.canon_taps:
                    out.append((f"l{i}.canon{n}", (D, cfg.canon_taps), "normal", i))
            if s.second is not None:
                out += [(q_ + "out", (D,), "norm", i) for q_ in prefixes]
            out += [(f"l{i}.shift", (D,), "shift", i)] if cfg.token_shift else []
            if cfg.side_dim:
                out += [(f"l{i}.side.gate", (cfg.side_dim, D), "normal", i), (f"l{i}.side.proj", (D, cfg.side_dim), "normal", i),
                        (f"l{i}.side.norm", (D,), "norm", i)]
        elif cfg.streams:
            S = cfg.streams
            for n in ("1", "2") if f.kind != "none" else ("1",):
                out += norm(f"l{i}.norm{n}", i)
                out += [(f"l{i}.hc{n}.in", (S,), "norm", i), (f"l{i}.hc{n}.out", (S,), "norm", i), (f"l{i}.hc{n}.mix", (S, S), "mix", i)]
        else:
            out += norm(f"l{i}.norm1", i)
        for m, p in zip(s.mixers, prefixes):
            out += mixer_tensor_specs(m, p, D, i)

        def ff(prefix, n):
            return [(prefix + "gate", (n, D), "normal", i), (prefix + "up", (n, D), "normal", i),
                    (prefix + "down", (D, n), "normal", i)]
        if f.kind == "dense":
            out += ff(q, f.ff)[1 if f.activation == "relu2" else 0:]
        elif f.kind == "moe":
            out.append((q + "router", (f.experts, D), "normal", i))
            out += [(q + "correction", (f.experts,), "bias", i)] if f.correction else []
            for e in range(f.experts):
                out += ff(f"{q}e{e}.", f.ff)[1 if f.activation == "relu2" else 0:]
            if f.shared_ff:
                out += ff(q + "shared.", f.shared_ff) + ([(q + "shared.sg", (1, D), "normal", i)] if f.shared_gate else [])
    return out


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

    def _plan(self, meta: AttnMeta, T: int) -> StepPlan:
        if meta.mode == "decode":
            return StepPlan(meta.seqlens, None, None, None, meta.state_slots, None)
        dev = self.device
        cu = meta.cu_seqlens
        cu_t = torch.tensor(cu, dtype=torch.int32, device=dev)
        counts = torch.tensor([b - a for a, b in zip(cu, cu[1:])], device=dev)
        row_seq = torch.repeat_interleave(torch.arange(len(cu) - 1, dtype=torch.int32, device=dev), counts, output_size=T)
        return StepPlan((meta.positions + 1).to(torch.int32), row_seq, cu_t, list(cu), meta.state_slots, meta.state_has_initial,
                        list(meta.ctx_lens))

    def _operand(self, T: int, cols: int, cols_p: int) -> torch.Tensor:
        """[T, cols_p] operand of an output projection whose writer fills the first ``cols`` columns."""
        return (torch.zeros if cols != cols_p else torch.empty)(T, cols_p, dtype=self.dtype, device=self.device)

    def forward(self, ids: torch.Tensor, meta: AttnMeta, cache) -> torch.Tensor:
        """ids [T] -> fp32 logits [len(logit_rows) or T, vocab]."""
        plan = self._plan(meta, ids.shape[0])
        cfg = self.cfg
        W4 = pad_to(cfg.hidden_size, 4)
        x = torch.empty(*((ids.shape[0], cfg.streams, W4) if cfg.streams else (ids.shape[0], W4)), dtype=torch.float32,
                        device=self.device)
        block = self._hyper if cfg.streams else self._sandwich if cfg.sandwich else self._parallel
        y = block(x, ids.to(torch.int32), plan, meta, cache)
        with self.timer.timed("lm_head"):
            return gemm.rows_gemm(y, self.w.lm_head)

    # ------------------------------------------------------------------ sandwich blocks
    def _enter(self, x, s: Sublayer, l: int, plan: StepPlan, cache, pending) -> torch.Tensor:
        """What a sublayer reads: the previous sublayer's output joins the residual stream, norm, input convolution."""
        D, eps = self.cfg.hidden_size, self.cfg.rms_eps
        args = (x, s.norm, eps, D, self.width_p, self.dtype)
        if s.canon_w is None:
            return residual.sandwich_norm(*args, **pending)
        hist = cache.state.layer(l, s.canon_part)
        if plan.cu is None:
            return residual.sandwich_norm(*args, **pending, canon=residual.Canon(s.canon_w, hist, plan.slots))
        h = residual.sandwich_norm(*args, **pending, raw=True) if s.norm is not None else x
        if s.norm is None:                        # the convolution reads the residual itself
            residual.sandwich_norm(*args, **pending, emit=False)
        y = torch.empty(x.shape[0], self.width_p, dtype=self.dtype, device=x.device)
        return conv.causal_conv(h, s.canon_w, hist, plan.slots, y, "residual", plan.cu, plan.cu_host, plan.row_seq, plan.has_initial)

    def _sandwich(self, x, ids, plan: StepPlan, meta: AttnMeta, cache) -> torch.Tensor:
        cfg, tm, w = self.cfg, self.timer, self.w
        T, D = x.shape[0], cfg.hidden_size
        if plan.slots is None and cfg.has_state:
            raise RuntimeError("a model with per-sequence state needs AttnMeta.state_slots")
        pending = dict(ids=ids, embed=w.embed, embed_scale=cfg.embed_scale)
        for l, layer in enumerate(w.layers):
            for i, s in enumerate(layer):
                with tm.timed("norm", l):
                    y = self._enter(x, s, l, plan, cache, pending)
                if self.layer_hook is not None and l and not i:
                    self.layer_hook(l - 1, x[:, :D])
                with tm.timed("proj_in", l):
                    z = gemm.rows_gemm(y, s.w_in)
                if s.experts is not None:
                    f = s.mlp
                    with tm.timed("moe", l):
                        idx, rw = moe_ops.router_topk(z[:, :f.experts], None, f.top, scoring=f.scoring, num_valid=meta.num_valid)
                        routed, pos = moe_ops.routed_rows(y, idx, rw, s.experts, False, meta.num_valid)
                    pending = dict(routed=routed, pos=pos, route_w=rw, post=s.post)
                    continue
                if s.mixers:
                    operands = []
                    with tm.timed("mixer_" + meta.mode, l):
                        for m, wo in zip(s.mixers, s.w_out):
                            operands.append(self._operand(T, m.cols, wo.shape[1]))
                            m.run(l, z, operands[-1][:, :m.cols], plan, meta, cache)
                elif s.side is not None:
                    with tm.timed("side", l):
                        operands = [residual.token_side(z, s.side, ids, s.w_out[0].shape[1], self.dtype)]
                else:
                    with tm.timed("act", l):
                        operands = [residual.cast_act(z[:, :s.ff], s.w_out[0].shape[1], self.dtype, "relu2")]
                with tm.timed("proj_out", l):
                    outs = [gemm.rows_gemm(o, wo) for o, wo in zip(operands, s.w_out)]
                pending = dict(add=outs[0], post=s.post)
                if len(outs) > 1:
                    pending.update(add2=outs[1], branch_w=s.branch_w)
        args = (x, w.final_norm, cfg.rms_eps, D, self.width_p, self.dtype)
        if self.layer_hook is not None:           # the last sublayer's output is only summed inside the final norm
            residual.sandwich_norm(*args, **pending)
            pending = {}
            self.layer_hook(len(w.layers) - 1, x[:, :D])
        return residual.sandwich_norm(*args, **pending, keep=False,
                                      rows=meta.logit_rows.long() if meta.logit_rows is not None else None)

    # ------------------------------------------------------------------ hyper-connected blocks
    def _hyper(self, x, ids, plan: StepPlan, meta: AttnMeta, cache) -> torch.Tensor:
        cfg, tm, w, dt = self.cfg, self.timer, self.w, self.dtype
        T, D = x.shape[0], cfg.hidden_size
        args = (D, self.width_p, dt)
        pending = dict(ids=ids, embed=w.embed, embed_scale=cfg.embed_scale)
        for l, layer in enumerate(w.layers):
            for i, s in enumerate(layer):
                with tm.timed("norm", l):
                    y = residual.hyper_norm(x, s.norm.w, cfg.rms_eps, *args, read=s.hc.read, **pending)
                if self.layer_hook is not None and l and not i:
                    self.layer_hook(l - 1, x[..., :D].sum(1))
                with tm.timed("proj_in", l):
                    z = gemm.rows_gemm(y, s.w_in)
                pending = dict(hc=s.hc, bias=s.bias)
                operand = None
                if s.mixers:
                    spans = [pad_to(m.cols, K_ALIGN) for m in s.mixers]
                    operand = self._operand(T, sum(m.cols for m in s.mixers), sum(spans))
                    with tm.timed("mixer_" + meta.mode, l):
                        at = 0
                        for m, n in zip(s.mixers, spans):
                            m.run(l, z, operand[:, at:at + m.cols], plan, meta, cache)
                            at += n
                elif s.ff:
                    with tm.timed("glu", l):
                        operand = residual.glu(z[:, s.seg["gate"][0]:], s.ff, s.mlp.activation,
                                               s.mlp.limit if s.mlp.kind == "dense" else s.mlp.shared_limit, dtype=dt)
                if s.experts is not None:
                    f, r0 = s.mlp, s.seg["router"][0]
                    with tm.timed("moe", l):
                        idx, rw = moe_ops.router_topk(z[:, r0:r0 + f.experts], s.correction, f.top, f.groups, f.keep_groups,
                                                      "always" if f.norm_weights else False, f.router_scale, f.scoring,
                                                      meta.num_valid, f.group_score)
                        routed, pos = moe_ops.routed_rows(y, idx, rw, s.experts, False, meta.num_valid)
                    pending.update(routed=routed, pos=pos, route_w=rw)
                if operand is not None:
                    with tm.timed("proj_out", l):
                        pending["add"] = gemm.rows_gemm(operand, s.w_out[0])
        final = (x, w.final_norm.w, cfg.rms_eps, *args)
        if self.layer_hook is not None:           # the last sublayer's output only joins the streams inside the final norm
            residual.hyper_norm(*final, **pending)
            pending = {}
            self.layer_hook(len(w.layers) - 1, x[..., :D].sum(1))
        return residual.hyper_norm(*final, **pending, keep=False,
                                   rows=meta.logit_rows.long() if meta.logit_rows is not None else None)

    # ------------------------------------------------------------------ parallel blocks
    def _parallel(self, x, ids, plan: StepPlan, meta: AttnMeta, cache) -> torch.Tensor:
        cfg, tm, w = self.cfg, self.timer, self.w
        T, D = x.shape[0], cfg.hidden_size
        dt = self.dtype
        first = dict(ids=ids, embed=w.embed, embed_scale=cfg.embed_scale)
        add = routed = pos = None
        for l, lw in enumerate(w.layers):
            f, mx = lw.spec.mlp, lw.mixer
            with tm.timed("norm", l):
                h = residual.residual_norm(x, lw.norm, cfg.rms_eps, D, self.width_p, dt, add=add, routed=routed, pos=pos,
                                           **first)
            if self.layer_hook is not None and l:
                self.layer_hook(l - 1, x[:, :D])
            first = {}
            with tm.timed("proj_in", l):
                z = gemm.rows_gemm(h, lw.w_in)
            cat = self._operand(T, mx.cols if mx.cols != lw.mix_p else lw.mix_p + lw.ff_p, lw.mix_p + lw.ff_p)
            with tm.timed("mixer_" + meta.mode, l):
                mx.run(l, z, cat[:, :mx.cols], plan, meta, cache)
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
        return residual.residual_norm(x, w.final_norm, cfg.rms_eps, D, self.width_p, dt, add=add, routed=routed, pos=pos,
                                      rows=meta.logit_rows.long() if meta.logit_rows is not None else None, keep=False)
