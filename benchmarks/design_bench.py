"""Layer-listed models (Nanurax, Pamevik, Bolisun, Pitudra) beside the framework's closest existing model at equal size.

``bench.py --workload nanurax | pamevik | bolisun | pitudra``: both models have four layers of a real model's size (width 2304, 32 heads of 128,
bf16), three recurrent layers to one attention layer.  Nanurax runs the generalised delta rule and chunked talking-heads
attention with one dense and three mixture feed-forwards (64 experts of which 8 run); Pamevik runs two channel-delta layers, an
mLSTM layer and attention beside retention, with dense feed-forwards.  The other one is a Kimi-Linear cut with KDA and MLA
layers and the same kinds of feed-forwards.  Bolisun runs four layers of windowed attention beside retention, with one dense and
three mixture feed-forwards; next to the Kimi-Linear cut (mixtures of the same size) it has Pamevik with four layers of attention
beside retention, whose dense feed-forwards hold as many weights as a token's experts.  Pitudra runs two HGRN2 layers, one of windowed
and one of latent attention, with four mixtures, next to a Kimi-Linear cut with four mixtures of as many weights.  Prefill is one packed forward over fresh prompts, decode is a captured step over
sequences with cached context; random weights, CUDA events, medians, the L2 flushed before every timed call.

``kernels`` of the result times the new kernels beside their likes (recurrences against KDA, decode attention against the
paged GQA kernel, prompt attention against the expanded MLA kernel, norms against the fused residual norm, latent attention against the MLA kernels; Bolisun's and Pitudra's others against
those of the designs before them) with the share of the measured roofline each reaches.
"""
from __future__ import annotations

import json
import math
import os
from typing import Callable, Dict, List

PREFILL = [(1, 4096), (8, 1024)]
DECODE = [(16, 2048), (64, 2048), (256, 2048)]


def _peaks(root: str) -> Dict[str, float]:
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    except (OSError, KeyError, ValueError):
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


class _Timer:
    def __init__(self, dev, steps: int, warmup: int):
        import torch
        self.torch, self.steps, self.warmup = torch, steps, warmup
        self.flush = torch.empty(300 << 20, dtype=torch.uint8, device=dev)

    def __call__(self, fn: Callable[[], object]) -> float:
        """Median milliseconds on the device."""
        t = self.torch
        for _ in range(self.warmup):
            fn()
        times = []
        for _ in range(self.steps):
            self.flush.zero_()
            a, b = t.cuda.Event(enable_timing=True), t.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            t.cuda.synchronize()
            times.append(a.elapsed_time(b))
        return sorted(times)[len(times) // 2]


def _closest(design: str):
    import dataclasses
    from batchgen_b200.config import get_model_config
    mlp = dict(first_k_dense=4) if design == "pamevik" else dict(n_routed_experts=64, num_experts_per_tok=8)
    if design == "pitudra":
        mlp.update(first_k_dense=0, n_shared_experts=0)
    out = [get_model_config("kimi-linear-48b", num_layers=4, kda_layers=(0, 1, 2), **mlp)]
    if design == "bolisun":
        cfg = get_model_config("pamevik-bench")
        out.insert(0, dataclasses.replace(cfg, name="pamevik-beside", layer_specs=cfg.layer_specs[-1:] * 4))
    return out


def _model_rates(cfg, dev, timer: _Timer) -> Dict[str, object]:
    import torch
    from batchgen_b200.config import EngineConfig
    from batchgen_b200.models import build_model
    from batchgen_b200.runtime.engine import Engine, _PrefillRow
    from batchgen_b200.runtime.graphs import DecodeGraphRunner
    model = build_model(cfg, device=dev, dtype="bf16", seed=0, gen_device=dev, max_positions=8192)
    most = max(b for b, _ in DECODE)
    ctx = max(c for _, c in DECODE)
    page = 64
    per = ctx // page + 1
    ecfg = EngineConfig(page_size=page, max_decode_batch=most, max_state_slots=most, device=str(dev), dtype="bf16")
    eng = Engine(model, ecfg, num_gpu_pages=most * per)
    pages = eng.kv.alloc.alloc(most * per)
    g = torch.Generator().manual_seed(0)
    out: Dict[str, object] = {"prefill": [], "decode": []}
    for b, n in PREFILL:
        need = n // page
        rows = [_PrefillRow(torch.randint(2, cfg.vocab_size, (n,), generator=g).tolist(), 0, pages[i * need:(i + 1) * need],
                            state_slot=i) for i in range(b)]
        ids, meta, T, _ = eng._rows_step(rows, [(i + 1) * n - 1 for i in range(b)])
        ms = timer(lambda: model.forward(ids, meta, eng.kv))
        out["prefill"].append({"prompts": b, "tokens_each": n, "ms": round(ms, 3), "tok_per_s": round(T / ms * 1e3)})
    if eng.kv.state is not None:
        eng.kv.state.rec.normal_(std=0.05)
    eng.kv.kv.normal_(std=0.5)
    run = DecodeGraphRunner(model, eng.kv, max_batch=most, max_pages_per_seq=per, num_buckets=1)
    run.bucketing.buckets = [b for b, _ in DECODE]
    for b, c in DECODE:
        lists = [pages[i * per:(i + 1) * per] for i in range(b)]
        run.stage([3] * b, [c - 1] * b, [p[(c - 1) // page] * page + (c - 1) % page for p in lists], [c] * b, lists,
                  list(range(b)) if run.state_slots is not None else None)
        run.replay(b, b)
        ms = timer(lambda: run.replay(b, b))
        out["decode"].append({"rows": b, "context": c, "ms": round(ms, 3), "tok_per_s": round(b / ms * 1e3)})
    del run, eng, model
    torch.cuda.empty_cache()
    return out


class _Rows:
    """Timed kernels with the share of the roofline each reaches."""

    def __init__(self, peaks):
        self.peaks, self.rows = peaks, []

    def __call__(self, name, size, ms, gbytes=0.0, tflop=0.0):
        r = {"kernel": name, "size": size, "us": round(ms * 1e3, 1)}
        share = []
        if gbytes:
            r["gb_per_s"] = round(gbytes / ms * 1e3)
            share.append(gbytes / ms * 1e3 / self.peaks["hbm_gbs"])
        if tflop:
            r["tflops"] = round(tflop / ms * 1e3, 1)
            share.append(tflop / ms * 1e3 / self.peaks["bf16_tflops"])
        r["of_" + self.peaks["source"]] = round(max(share), 3)
        self.rows.append(r)


H, G, D, PAGE = 32, 8, 128, 64
HD = H * D
STATE_CASES = [(64, 1), (256, 1), (1, 4096), (8, 1024)]        # sequences, tokens of each


def _state_case(dev, B: int, T: int):
    import torch
    R = B * T
    slots = torch.arange(B, dtype=torch.int32, device=dev)
    cu = None if T == 1 else torch.arange(0, R + 1, T, dtype=torch.int32, device=dev)
    init = None if T == 1 else torch.ones(B, dtype=torch.int32, device=dev)
    return R, f"{B} x {T} tokens", slots, cu, init


def _kda_row(dev, timer, add, B, T):
    import torch
    from batchgen_b200.ops import kda
    R, size, slots, cu, init = _state_case(dev, B, T)
    qkv, f = torch.randn(R, 4 * HD + 64, device=dev).bfloat16(), torch.randn(R, HD, device=dev).bfloat16()
    kp = kda.KDAParams(torch.randn(3 * HD, 4, device=dev), None, torch.randn(H, device=dev), torch.randn(HD, device=dev),
                       torch.ones(D, device=dev))
    cs, rs = torch.zeros(B, 3 * HD, 3, device=dev), torch.zeros(B, H, D, D, device=dev)
    ms = timer(lambda: kda.kda_forward(qkv[:, :3 * HD], f, qkv[:, 4 * HD:4 * HD + H], qkv[:, 3 * HD:4 * HD], kp, cs, rs,
                                       slots, cu, init, H, D, D ** -0.5, 1e-6))
    add("  KDA", size, ms, (R * HD * 12 + B * HD * (D * 8 + 3 * 3 * 8)) / 1e9)


def _decode_attention_rows(dev, timer, add, cases, talk, **more):
    import torch
    from batchgen_b200.ops import attention, talking
    for B, ctx in cases:
        n = B * ctx // PAGE
        cache = torch.randn(n, PAGE, 2 * G * D, device=dev).bfloat16()
        bt = torch.randperm(n, device=dev).to(torch.int32).view(B, -1).contiguous()
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q, out = torch.randn(B, HD, device=dev), torch.empty(B, HD, dtype=torch.bfloat16, device=dev)
        p = talking.TalkParams(H, G, D, D, D ** -0.5, ctx if talk is not None else 0, talk is not None, talk)
        extra = {k: f(lens) for k, f in more.items()}
        gb = B * ctx * 2 * G * D * 2 / 1e9
        add("attention, decode", f"{B} x {ctx} keys", timer(lambda: talking.attend_rows(q, p, cache, bt, lens, out, **extra)), gb)
        qb = q.bfloat16().view(B, H, D)
        sinks = torch.zeros(H, device=dev)
        add("  GQA decode", f"{B} x {ctx} keys",
            timer(lambda: attention.gqa_decode(qb, cache, bt, lens, G, D ** -0.5, sinks=sinks)), gb)


def _prompt_attention_rows(dev, timer, add, cases, talk, **more):
    import torch
    from batchgen_b200.ops import attention, talking
    for T, chunk in cases:
        n = T // PAGE
        cache = torch.randn(n, PAGE, 2 * G * D, device=dev).bfloat16()
        bt = torch.arange(n, device=dev, dtype=torch.int32).view(1, -1).contiguous()
        q, out = torch.randn(T, HD, device=dev), torch.empty(T, HD, dtype=torch.bfloat16, device=dev)
        mixed = talk is not None
        p = talking.TalkParams(H, G, D, D, D ** -0.5, chunk if mixed else 0, mixed, talk)
        extra = {k: f(torch.arange(1, T + 1, dtype=torch.int32, device=dev)) for k, f in more.items()}
        pairs = T * (chunk + 1) / 2
        blocks = talking.work_blocks(talking.prefill_work([0, T], [0], p.chunk), T, dev)
        size = f"{T} tokens" + (f", chunks of {chunk}" if mixed else "")
        add("attention, prompt", size, timer(lambda: talking.attend_prefill(q, p, cache, bt, out, blocks, **extra)), 0,
            pairs * 2 * H * (2 * D + (H if mixed else 0)) / 1e12)
        q3, kv = torch.randn(T, H, 192, device=dev).bfloat16(), torch.randn(T, H, 256, device=dev).bfloat16()
        kpe = torch.randn(T, 64, device=dev).bfloat16()
        cu = list(range(0, T + 1, chunk))
        work = attention.mha_prefill_work(cu, [0] * (len(cu) - 1), cu[:-1]).to(dev)
        add("  expanded MLA prompt", size, timer(lambda: attention.mha_prefill(q3, kv, kpe, work, 0.07)), 0,
            pairs * 2 * H * 320 / 1e12)


def _nanurax_kernels(dev, timer: _Timer, peaks) -> List[Dict[str, object]]:
    import torch
    from batchgen_b200.ops import delta
    add = _Rows(peaks)
    for B, T in STATE_CASES:
        R, size, slots, cu, init = _state_case(dev, B, T)
        z, wl = torch.randn(R, 5 * HD, device=dev), torch.randn(R, HD, device=dev)
        p = delta.DeltaParams(torch.randn(HD, device=dev), torch.randn(HD, device=dev), torch.ones(HD, device=dev), H, D, D,
                              math.exp(-0.5))
        st, out = torch.zeros(B + 1, HD * D, device=dev), torch.empty(R, HD, dtype=torch.bfloat16, device=dev)
        ms = timer(lambda: delta.delta_forward(z, tuple(i * HD for i in range(5)), wl, p, st, slots, out, cu, None, init))
        add("delta rule", size, ms, (R * HD * (6 * 4 + 2) + B * HD * D * 8) / 1e9)
        del z, wl
        _kda_row(dev, timer, add, B, T)
    talk = torch.randn(H, H, device=dev) / 6
    _decode_attention_rows(dev, timer, add, ((16, 4096), (64, 4096)), talk)
    _prompt_attention_rows(dev, timer, add, ((4096, 4096), (8192, 2048)), talk)
    return add.rows


def _pamevik_kernels(dev, timer: _Timer, peaks) -> List[Dict[str, object]]:
    import torch
    from batchgen_b200.ops import conv, fused, recurrent, residual
    bf, add = torch.bfloat16, _Rows(peaks)
    rot = conv.Rotary.make(D, 1e6, dev)
    for B, T in STATE_CASES:
        R, size, slots, cu, init = _state_case(dev, B, T)
        row_seq = None if T == 1 else torch.arange(B, dtype=torch.int32, device=dev).repeat_interleave(T)
        z, out = torch.randn(R, 5 * HD + 64, device=dev), torch.empty(R, HD, dtype=bf, device=dev)
        pool = torch.zeros(B + 1, HD * D + HD + H, device=dev)
        S = {"S": pool[:, :HD * D], "n": pool[:, HD * D:HD * (D + 1)], "m": pool[:, HD * (D + 1):]}
        q, k, v, g, low = (z[:, i * HD:(i + 1) * HD] for i in range(5))
        gates = z[:, 5 * HD:5 * HD + H]
        base = dict(heads=H, dim_p=D, vdim=D, vdim_p=D, norm_w=torch.ones(HD, device=dev), eps=1e-6)
        rules = {
            "channel_delta": (dict(rate=torch.ones(H, device=dev), dt_bias=torch.zeros(HD, device=dev)), dict(low=low, beta=gates), 5),
            "mlstm": (dict(i_bias=torch.zeros(H, device=dev), f_bias=torch.zeros(H, device=dev), gate_cap=15.0),
                      dict(gate_i=gates, gate_f=gates), 4),
            "retention": (dict(decay=torch.full((H,), 0.99, device=dev), gate="silu"),
                          dict(rope=rot.table(torch.arange(1, R + 1, dtype=torch.int32, device=dev))), 4)}
        for rule, (kw, more, columns) in rules.items():
            p = recurrent.RecurrentParams(rule, **base, **kw)
            st = {n: t for n, t in S.items() if n == "S" or rule == "mlstm"}
            ms = timer(lambda: recurrent.recurrent_forward(p, q, k, v, g, st, slots, out, cu, None, init, **more))
            add(rule, size, ms, (R * HD * (columns * 4 + 2) + B * HD * D * 8) / 1e9)
        _kda_row(dev, timer, add, B, T)
        w, hist = torch.randn(4, 3 * HD, device=dev), torch.zeros(B + 1, 9 * HD, device=dev)
        x = torch.empty(R, 3 * HD, device=dev)
        ms = timer(lambda: conv.causal_conv(z[:, :3 * HD], w, hist, slots, x, "silu", cu, None, row_seq, init))
        add("short convolutions", size, ms, (R * 3 * HD * 8 + B * 9 * HD * 8) / 1e9)
        del z, x
        Wd = 2304
        n1 = residual.Norm(torch.ones(Wd, device=dev), torch.zeros(Wd, device=dev), True)
        xs, a, b = (torch.randn(R, Wd, device=dev) for _ in range(3))
        cw, ch = torch.randn(4, Wd, device=dev), torch.zeros(B + 1, 3 * Wd, device=dev)
        pair = dict(add=a, add2=b, branch_w=(n1.w, n1.w), post=n1)
        if T == 1:
            canon = residual.Canon(cw, ch, slots)
            ms = timer(lambda: residual.sandwich_norm(xs, n1, 1e-6, Wd, Wd, bf, add=a, post=n1, canon=canon))
            add("norms + input convolution", size, ms, (R * Wd * (4 * 3 + 2) + B * Wd * 24) / 1e9)
        else:
            y = torch.empty(R, Wd, dtype=bf, device=dev)
            ms = timer(lambda: conv.causal_conv(residual.sandwich_norm(xs, n1, 1e-6, Wd, Wd, bf, add=a, post=n1, raw=True), cw, ch,
                                                slots, y, "residual", cu, None, row_seq, init))
            add("norms + input convolution", size, ms, R * Wd * (4 * 3 + 2) / 1e9)
        add("norms of two branches", size, timer(lambda: residual.sandwich_norm(xs, n1, 1e-6, Wd, Wd, bf, **pair)),
            R * Wd * (4 * 4 + 2) / 1e9)
        xb, rb = xs.to(bf), a.to(bf)
        ms = timer(lambda: fused.rmsnorm(xb, n1.w, 1e-6, residual=rb))
        add("  residual + RMS norm", size, ms, R * Wd * 8 / 1e9)
    rope, gate = rot.table, lambda lens: torch.randn(lens.shape[0], H, device=dev)
    _decode_attention_rows(dev, timer, add, ((16, 4096), (64, 4096)), None, rope=rope, gate=gate)
    _prompt_attention_rows(dev, timer, add, ((4096, 4096), (8192, 8192)), None, rope=rope, gate=gate)
    return add.rows


def _bolisun_kernels(dev, timer: _Timer, peaks) -> List[Dict[str, object]]:
    import torch
    from batchgen_b200.config import get_model_config
    from batchgen_b200.ops import conv, moe, recurrent, residual, talking
    bf, add = torch.bfloat16, _Rows(peaks)
    row, W, E, K, Fe = 2 * G * D, 2304, 64, 8, 1024
    left = get_model_config("bolisun-bench").layer_specs[0].mixer
    win, keep = left.window, left.keep_first
    rot = conv.Rotary.make(D, 1e6, dev, True, left.yarn)
    half = conv.Rotary.make(D, 1e6, dev)
    norm, bias = torch.ones(D, device=dev), torch.zeros(HD + row, device=dev)
    prep = talking.HeadPrep(D, 1e-6, bias, norm, norm, True)
    full = talking.TalkParams(H, G, D, D, D ** -0.5)
    near = talking.TalkParams(H, G, D, D, D ** -0.5, window=win, keep=keep, out_scale=0.5)
    gains = residual.Norm(torch.ones(W, device=dev), torch.zeros(W, device=dev), True)
    for B, T in STATE_CASES:
        R, size, slots, cu, init = _state_case(dev, B, T)
        prompt = T > 1
        z, out = torch.randn(R, 4 * HD, device=dev), torch.empty(R, HD, dtype=bf, device=dev)
        S = torch.zeros(B + 1, HD * D, device=dev)
        p = recurrent.RecurrentParams("retention", H, D, D, D, torch.full((HD,), 0.5, device=dev), 1e-6, "silu",
                                      decay=torch.full((H,), 0.99, device=dev))
        q, k, v, g = (z[:, i * HD:(i + 1) * HD] for i in range(4))
        ms = timer(lambda: recurrent.recurrent_forward(p, q, k, v, g, {"S": S}, slots, out, cu, None, init))
        add("retention", size, ms, (R * HD * 18 + B * HD * D * 8) / 1e9)
        _kda_row(dev, timer, add, B, T)
        # heads between projections and scores, beside the rotary cache write (and, in prompts, the query operand)
        n = -(-R // PAGE)
        cache, at = torch.zeros(n, PAGE, row, dtype=bf, device=dev), torch.arange(R, device=dev)
        lens = torch.arange(1, R + 1, dtype=torch.int32, device=dev)
        tab, tab2 = rot.table(lens), half.table(lens)
        gb = R * (HD + row) * 4 / 1e9 + R * (row * 2 + HD * (2 if prompt else 4) + D * 4) / 1e9
        ms = timer(lambda: talking.prepare_heads(z, at, cache, near, prep, tab, not prompt, prompt))
        add("heads: bias, norm, rotation, cache", size, ms, gb)
        if not prompt:
            ms = timer(lambda: talking.kv_write(z[:, :row], at, cache, full, tab2))
            add("  rotary cache write", size, ms, R * (row * 6 + D * 4) / 1e9)
        x, a = torch.randn(R, 2, W, device=dev), torch.randn(R, W, device=dev)
        ones, mix = torch.ones(2, device=dev), torch.eye(2, device=dev)
        hc = residual.Hyper(ones, mix, ones)
        ms = timer(lambda: residual.hyper_norm(x, gains.w, 1e-6, W, W, bf, read=ones, hc=hc, add=a, bias=gains.b))
        add("hyper-connection + norm", size, ms, R * W * (4 * 5 + 2) / 1e9)
        routed = torch.randn(R * K, W, device=dev)
        pos = torch.randperm(R * K, device=dev).to(torch.int32).view(R, K).contiguous()
        rw = torch.rand(R, K, device=dev)
        ms = timer(lambda: residual.hyper_norm(x, gains.w, 1e-6, W, W, bf, read=ones, hc=hc, add=a, routed=routed, pos=pos, route_w=rw))
        add("hyper-connection + norm + experts' rows", size, ms, R * W * (4 * (5 + K) + 2) / 1e9)
        x1 = x[:, 0].contiguous()
        ms = timer(lambda: residual.sandwich_norm(x1, gains, 1e-6, W, W, bf, add=a, post=gains))
        add("  norms of a sandwich block", size, ms, R * W * (4 * 3 + 2) / 1e9)
        ms = timer(lambda: residual.residual_norm(x1, gains.w, 1e-6, W, W, bf, add=a, routed=routed, pos=pos))
        add("  residual + norm + experts' rows", size, ms, R * W * (4 * (3 + K) + 2) / 1e9)
        logits, corr = torch.randn(R, E, device=dev), torch.zeros(E, device=dev)
        gb = R * (E * 4 + K * 8) / 1e9
        add("router", size, timer(lambda: moe.router_topk(logits, corr, K, 8, 4, "always", 2.5, "softmax_all", None, "max")), gb)
        add("  router, sigmoid", size, timer(lambda: moe.router_topk(logits, None, K, norm_topk_prob=False)), gb)
        idx, rw = moe.router_topk(logits, corr, K, 8, 4, "always", 2.5, "softmax_all", None, "max")
        h = torch.randn(R, W, device=dev).to(bf)
        w13, w2 = (torch.randn(E, *s, device=dev, dtype=bf) * 0.02 for s in ((2 * Fe, W), (W, Fe)))
        gb, tf = E * 3 * W * Fe * 2 / 1e9 + R * K * W * 4 / 1e9, R * K * 6 * W * Fe / 1e12
        for name, kind, on_input in (("experts", "silu", False), ("  experts, weighted input", "swiglu_oai", True)):
            ew = moe.ExpertWeights(w13, w2, activation=kind, act_limit=7.0)
            add(name, size, timer(lambda: moe.routed_rows(h, idx, rw, ew, on_input)), gb, tf)
        del x, a, routed, z, w13, w2
    for B, ctx in ((16, 4096), (64, 4096), (256, 4096)):
        n = B * ctx // PAGE
        cache = torch.randn(n, PAGE, row, device=dev).bfloat16()
        bt = torch.randperm(n, device=dev).to(torch.int32).view(B, -1).contiguous()
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q, out = torch.randn(B, HD, device=dev), torch.empty(B, HD, dtype=bf, device=dev)
        for name, p, keys in (("attention, decode, window", near, win + keep), ("  attention, decode", full, ctx)):
            add(name, f"{B} x {keys} of {ctx} keys", timer(lambda: talking.attend_rows(q, p, cache, bt, lens, out)),
                B * keys * row * 2 / 1e9)
        bts = bt[:, :(win + keep) // PAGE].contiguous()              # as many keys, one after the other
        short = torch.full((B,), win + keep, dtype=torch.int32, device=dev)
        add("  attention, decode", f"{B} x {win + keep} keys", timer(lambda: talking.attend_rows(q, full, cache, bts, short, out)),
            B * (win + keep) * row * 2 / 1e9)
        del cache
    for B, T in ((1, 4096), (8, 1024), (1, 16384)):
        n, R = T // PAGE, B * T
        cache = torch.randn(B * n, PAGE, row, device=dev).bfloat16()
        bt = torch.arange(B * n, device=dev, dtype=torch.int32).view(B, n).contiguous()
        qf = torch.randn(R, H, D, device=dev).bfloat16()
        q, out = torch.empty(R, HD, device=dev), torch.empty(R, HD, dtype=bf, device=dev)
        cu = list(range(0, R + 1, T))
        for name, p in (("attention, prompt, window", near), ("  attention, prompt", full)):
            blocks = talking.work_blocks(talking.prefill_work(cu, [0] * B, 0, 1, p.window), R, dev)
            seen = B * sum(p.most_keys(t) for t in range(1, T + 1))
            add(name, f"{B} x {T} tokens", timer(lambda: talking.attend_prefill(q, p, cache, bt, out, blocks, operand=qf)), 0,
                seen * 4 * H * D / 1e12)
        del cache, q, qf
    return add.rows


def _pitudra_kernels(dev, timer: _Timer, peaks) -> List[Dict[str, object]]:
    import torch
    from batchgen_b200.config import get_model_config
    from batchgen_b200.models import mixers
    from batchgen_b200.models.weights import WeightSource
    from batchgen_b200.ops import attention, conv, gemm, latent, moe, recurrent, residual, talking
    bf, add = torch.bfloat16, _Rows(peaks)
    cfg = get_model_config("pitudra-bench")
    att, W, E, K, side = cfg.layer_specs[1].mixer, 2304, 64, 8, cfg.side_dim
    row, win = att.kv_row, att.window
    near = talking.TalkParams(H, G, D, D, D ** -0.5, window=win, sinks=torch.zeros(H, device=dev), gate_all=True)
    plain = talking.TalkParams(H, G, D, D, D ** -0.5, window=win)
    whole = talking.HeadPrep(D, 1e-6, torch.zeros(HD + row, device=dev), torch.ones(HD, device=dev), torch.ones(G * D, device=dev), whole=True)
    single = talking.HeadPrep(D, 1e-6, torch.zeros(HD + row, device=dev), torch.ones(D, device=dev), torch.ones(D, device=dev), True)
    mx = mixers.build_mixer(cfg.layer_specs[3].mixer, "mix.", WeightSource(seed=1, device=dev, gen_device=dev), cfg, bf)
    lat = mx.lat
    gains = residual.Norm(torch.ones(W, device=dev), torch.zeros(W, device=dev), True)
    for B, T in STATE_CASES:
        R, size, slots, cu, init = _state_case(dev, B, T)
        prompt = T > 1
        row_seq = torch.arange(B, dtype=torch.int32, device=dev).repeat_interleave(T) if prompt else None
        z, out = torch.randn(R, 4 * HD, device=dev), torch.empty(R, HD, dtype=bf, device=dev)
        S = torch.zeros(B + 1, HD * D, device=dev)
        q, k, v, g = (z[:, i * HD:(i + 1) * HD] for i in range(4))
        base = dict(heads=H, dim_p=D, vdim=D, vdim_p=D, norm_w=torch.ones(HD, device=dev), eps=1e-6)
        p = recurrent.RecurrentParams("hgrn2", **base, f_bias=torch.zeros(HD, device=dev), f_lower=torch.full((HD,), 0.5, device=dev))
        ms = timer(lambda: recurrent.recurrent_forward(p, q, k, v, None, {"S": S}, slots, out, cu, None, init))
        add("HGRN2", size, ms, (R * HD * 14 + B * HD * D * 8) / 1e9)
        p = recurrent.RecurrentParams("retention", **base, gate="silu", decay=torch.full((H,), 0.99, device=dev))
        ms = timer(lambda: recurrent.recurrent_forward(p, q, k, v, g, {"S": S}, slots, out, cu, None, init))
        add("  retention", size, ms, (R * HD * 18 + B * HD * D * 8) / 1e9)
        _kda_row(dev, timer, add, B, T)
        n = -(-R // PAGE)
        cache, at = torch.zeros(n, PAGE, row, dtype=bf, device=dev), torch.arange(R, device=dev)
        tab = conv.Rotary.make(D, 1e6, dev).table(torch.arange(1, R + 1, dtype=torch.int32, device=dev))
        gb = R * (HD + row) * 4 / 1e9 + R * (row * 2 + HD * (2 if prompt else 4)) / 1e9
        add("heads: bias, norm over all, cache", size, timer(lambda: talking.prepare_heads(z, at, cache, near, whole, None, not prompt, prompt)), gb)
        ms = timer(lambda: talking.prepare_heads(z, at, cache, plain, single, tab, not prompt, prompt))
        add("  heads: bias, norm each, rotation, cache", size, ms, gb + R * D * 4 / 1e9)
        rope, rows = mixers.conv.Rotary.make(64, 1e6, dev).table(torch.arange(1, R + 1, dtype=torch.int32, device=dev)), torch.zeros(n, PAGE, 576, dtype=bf, device=dev)
        ms = timer(lambda: latent.prepare(z, (0, 1536, 2048), at, rows, lat, rope, bf))
        add("latents: norms, rotation, cache", size, ms, R * 2112 * 6 / 1e9)
        x, a = torch.randn(R, W, device=dev), torch.randn(R, W, device=dev)
        w2 = torch.rand(2, W, device=dev)
        hist, y = torch.zeros(B + 1, W, device=dev), torch.empty(R, W, dtype=bf, device=dev)

        def shift():
            if not prompt:
                return residual.sandwich_norm(x, None, 1e-6, W, W, bf, add=a, post=gains, canon=residual.Canon(w2, hist, slots))
            residual.sandwich_norm(x, None, 1e-6, W, W, bf, add=a, post=gains, emit=False)
            return conv.causal_conv(x, w2, hist, slots, y, "residual", cu, None, row_seq, init)
        add("norm of the output + token shift", size, timer(shift), (R * W * (4 * 3 + 2) + B * W * 8) / 1e9)
        add("norm of the output", size, timer(lambda: residual.sandwich_norm(x, None, 1e-6, W, W, bf, add=a, post=gains)), R * W * 14 / 1e9)
        routed = torch.randn(R * K, W, device=dev)
        pos = torch.randperm(R * K, device=dev).to(torch.int32).view(R, K).contiguous()
        rw = torch.rand(R, K, device=dev)
        ms = timer(lambda: residual.sandwich_norm(x, None, 1e-6, W, W, bf, routed=routed, pos=pos, route_w=rw, post=gains))
        add("norm of the experts' sum", size, ms, R * W * (4 * (2 + K) + 2) / 1e9)
        ms = timer(lambda: residual.sandwich_norm(x, gains, 1e-6, W, W, bf, add=a, post=gains))
        add("  norms of a sandwich block", size, ms, R * W * (4 * 3 + 2) / 1e9)
        ms = timer(lambda: residual.residual_norm(x, gains.w, 1e-6, W, W, bf, add=a, routed=routed, pos=pos))
        add("  residual + norm + experts' rows", size, ms, R * W * (4 * (3 + K) + 2) / 1e9)
        zs, table, ids = torch.randn(R, side, device=dev), torch.randn(9999, 4 * side, device=dev, dtype=bf), torch.randint(0, 9999, (R,), device=dev).to(torch.int32)
        add("token side input", size, timer(lambda: residual.token_side(zs, table[:, side:2 * side], ids, side, bf)), R * side * 8 / 1e9)
        logits = torch.randn(R, E, device=dev)
        idx, rw = moe.router_topk(logits, None, K, scoring="softmax")
        h = torch.randn(R, W, device=dev).to(bf)
        for name, kind, ff in (("experts", "relu2", 1536), ("  experts, gated", "silu", 1024)):
            w13 = torch.randn(E, ff if kind == "relu2" else 2 * ff, W, device=dev, dtype=bf) * 0.02
            ew = moe.ExpertWeights(w13, torch.randn(E, W, ff, device=dev, dtype=bf) * 0.02, activation=kind)
            flops = 2 * W * ff * (2 if kind == "relu2" else 3)
            add(name, size, timer(lambda: moe.routed_rows(h, idx, rw, ew, False)), E * flops / 1e9 + R * K * W * 4 / 1e9, R * K * flops / 1e12)
            del w13, ew
        del x, a, routed, z
    for B, ctx in ((16, 4096), (64, 4096), (256, 4096)):
        n = B * ctx // PAGE
        cache = torch.randn(n, PAGE, row, device=dev).bfloat16()
        bt = torch.randperm(n, device=dev).to(torch.int32).view(B, -1).contiguous()
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q, gate, out = torch.randn(B, HD, device=dev), torch.randn(B, HD, device=dev), torch.empty(B, HD, dtype=bf, device=dev)
        for name, p, more in (("attention, decode, window, sinks, gates", near, dict(gate=gate)), ("  attention, decode, window", plain, {})):
            add(name, f"{B} x {win} of {ctx} keys", timer(lambda: talking.attend_rows(q, p, cache, bt, lens, out, **more)), B * win * row * 2 / 1e9)
        del cache
    for B, ctx in ((16, 2048), (64, 2048), (256, 2048), (16, 4096), (64, 4096)):
        n = B * ctx // PAGE
        cache = torch.randn(n, PAGE, 576, device=dev).bfloat16()
        bt = torch.randperm(n, device=dev).to(torch.int32).view(B, -1).contiguous()
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        qa = torch.randn(B, H, 576, device=dev).bfloat16()
        gb, tf = B * ctx * 576 * 2 / 1e9, B * ctx * H * 1088 * 2 / 1e12
        add("latent attention, decode", f"{B} x {ctx} keys", timer(lambda: latent.attend(qa, lat, cache, bt, lens)), gb, tf)
        ms = timer(lambda: attention.mla_decode(qa[..., :512], qa[..., 512:], cache, bt, lens, lat.scale, 512))
        add("  MLA decode", f"{B} x {ctx} keys", ms, gb, tf)
        del cache
    for B in (16, 64, 256):
        q = torch.randn(B, H * 192, device=dev)
        rope = mx.rot.table(torch.arange(1, B + 1, dtype=torch.int32, device=dev))
        add("latent queries", f"{B} tokens", timer(lambda: latent.queries(q, lat, rope, None, bf)), (B * H * (192 * 4 + 576 * 2) + H * 128 * 512 * 2) / 1e9)
    for B, T in ((1, 4096), (8, 1024), (1, 16384)):
        n, R = T // PAGE, B * T
        cu = list(range(0, R + 1, T))
        cache = torch.randn(B * n, PAGE, row, device=dev).bfloat16()
        bt = torch.arange(B * n, device=dev, dtype=torch.int32).view(B, n).contiguous()
        qf = torch.randn(R, H, D, device=dev).bfloat16()
        q, gate, out = torch.randn(R, HD, device=dev), torch.randn(R, HD, device=dev), torch.empty(R, HD, dtype=bf, device=dev)
        blocks = talking.work_blocks(talking.prefill_work(cu, [0] * B, 0, 1, win), R, dev)
        tf = B * sum(near.most_keys(t) for t in range(1, T + 1)) * 4 * H * D / 1e12
        for name, p, more in (("attention, prompt, window, sinks, gates", near, dict(gate=gate)), ("  attention, prompt, window", plain, {})):
            add(name, f"{B} x {T} tokens", timer(lambda: talking.attend_prefill(q, p, cache, bt, out, blocks, operand=qf, **more)), 0, tf)
        # whole latents' prompt path; then its attention alone, and the expanded MLA kernel on the same keys and values
        cache = torch.randn(B * n, PAGE, 576, device=dev).bfloat16()
        ql = torch.randn(R, H * 192, device=dev)
        rope = mx.rot.table(torch.arange(1, T + 1, dtype=torch.int32, device=dev).repeat(B))
        groups = latent.expansions(cu, [0] * B, lat.window, PAGE, dev)
        seen = B * sum(min(t, lat.window) for t in range(1, T + 1))
        add("latents: expansion and attention, prompt", f"{B} x {T} tokens", timer(lambda: latent.attend_prompt(ql, lat, cache, bt, rope, out, groups)), 0,
            (seen * 2 * H * 320 + R * 2 * 512 * H * 256) / 1e12)
        e = lat.expanded
        up = torch.randn(B * n, PAGE, e.kv_row, device=dev).bfloat16()
        add("latents: attention, prompt", f"{B} x {T} tokens",
            timer(lambda: [talking.attend_prefill(ql, e, up, x.table, out, x.blocks, rope=rope) for x in groups]), 0, seen * 2 * H * 320 / 1e12)
        q3, kv = torch.randn(R, H, 192, device=dev).bfloat16(), torch.randn(R, H, 256, device=dev).bfloat16()
        kpe = torch.randn(R, 64, device=dev).bfloat16()
        work = attention.mha_prefill_work(cu, [0] * B, cu[:-1]).to(dev)
        add("  expanded MLA prompt", f"{B} x {T} tokens", timer(lambda: attention.mha_prefill(q3, kv, kpe, work, 0.07)), 0,
            B * T * (T + 1) / 2 * 2 * H * 320 / 1e12)
        c, wk = torch.randn(R, 512, device=dev).bfloat16(), torch.randn(H * 256, 512, device=dev).bfloat16()
        cw = torch.randn(R, 576, device=dev).bfloat16()
        add("latents: expansion product", f"{R} rows", timer(lambda: gemm.bf16_gemm(cw, lat.w_up)), 0, R * 2 * 512 * H * 256 / 1e12)
        add("  MLA expansion product", f"{R} rows", timer(lambda: gemm.bf16_gemm(c, wk)), 0, R * 2 * 512 * H * 256 / 1e12)
        del cache, q, qf, up, ql
    return add.rows


def run(args, root: str, design: str) -> int:
    import torch
    from batchgen_b200.config import get_model_config
    from batchgen_b200.ops import _ext
    from batchgen_b200.utils.clocks import ClockSampler
    assert args.gpus == 1, "the design benchmark runs on one GPU"
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    _ext.lib()
    peaks = _peaks(root)
    timer = _Timer(dev, args.steps, max(args.warmup, 3))
    sampler = ClockSampler(0).start()
    l0 = _ext.LAUNCHES["count"]
    models = {}
    for cfg in (get_model_config(f"{design}-bench"), *_closest(design)):
        models[cfg.name] = _model_rates(cfg, dev, timer)
    kernels = {"nanurax": _nanurax_kernels, "pamevik": _pamevik_kernels, "bolisun": _bolisun_kernels, "pitudra": _pitudra_kernels}[design](dev, timer, peaks)
    _ext.check_status()
    step = models[f"{design}-bench"]["decode"][1]
    print(json.dumps({
        "metric": f"decode tokens/s, 64 rows at 2,048 context, four layers ({design.capitalize()})", "value": step["tok_per_s"],
        "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": timer.warmup, "ms_per_step": step["ms"],
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"model": f"{design}-bench", "closest": list(models)[1:], "l2": "flushed before every call",
                   "parallelism": "1 GPU"},
        "models": models, "kernels": kernels, "peaks": peaks, "clocks": sampler.stop(),
        "gpu_launches": _ext.LAUNCHES["count"] - l0}))
    return 0
