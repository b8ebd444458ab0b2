"""Layer-listed model (Nanurax) beside the framework's closest existing model at equal size.

``bench.py --workload nanurax``: both models have four layers of a real model's size (width 2304, 32 heads of 128, 64
experts of which 8 run, one dense and three mixture feed-forwards, bf16): three recurrent layers to one attention layer.
Nanurax runs the generalised delta rule and chunked talking-heads attention, the other one is a Kimi-Linear cut with KDA and
MLA layers.  Prefill is one packed forward over fresh prompts, decode is a captured step over sequences with cached context;
random weights, CUDA events, medians, the L2 flushed before every timed call.

``kernels`` of the result times the new kernels beside their likes (recurrence against KDA, decode attention against the
paged GQA kernel, prompt attention against the expanded MLA kernel) with the share of the measured roofline each reaches.
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


def _closest():
    from batchgen_b200.config import get_model_config
    return get_model_config("kimi-linear-48b", num_layers=4, kda_layers=(0, 1, 2), n_routed_experts=64, num_experts_per_tok=8)


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


def _kernels(dev, timer: _Timer, peaks) -> List[Dict[str, object]]:
    import torch
    from batchgen_b200.ops import attention, delta, kda, talking
    H, G, D, page = 32, 8, 128, 64
    HD, bf = H * D, torch.bfloat16
    rows: List[Dict[str, object]] = []

    def add(name, size, ms, gbytes=0.0, tflop=0.0):
        r = {"kernel": name, "size": size, "us": round(ms * 1e3, 1)}
        share = []
        if gbytes:
            r["gb_per_s"] = round(gbytes / ms * 1e3)
            share.append(gbytes / ms * 1e3 / peaks["hbm_gbs"])
        if tflop:
            r["tflops"] = round(tflop / ms * 1e3, 1)
            share.append(tflop / ms * 1e3 / peaks["bf16_tflops"])
        r["of_" + peaks["source"]] = round(max(share), 3)
        rows.append(r)
    for B, T in ((64, 1), (256, 1), (1, 4096), (8, 1024)):
        R, size = B * T, f"{B} x {T} tokens"
        slots = torch.arange(B, dtype=torch.int32, device=dev)
        cu = None if T == 1 else torch.arange(0, R + 1, T, dtype=torch.int32, device=dev)
        init = None if T == 1 else torch.ones(B, dtype=torch.int32, device=dev)
        z, wl = torch.randn(R, 5 * HD, device=dev), torch.randn(R, HD, device=dev)
        p = delta.DeltaParams(torch.randn(HD, device=dev), torch.randn(HD, device=dev), torch.ones(HD, device=dev), H, D, D,
                              math.exp(-0.5))
        st, out = torch.zeros(B + 1, HD * D, device=dev), torch.empty(R, HD, dtype=bf, device=dev)
        ms = timer(lambda: delta.delta_forward(z, tuple(i * HD for i in range(5)), wl, p, st, slots, out, cu, None, init))
        add("delta rule", size, ms, (R * HD * (6 * 4 + 2) + B * HD * D * 8) / 1e9)
        del z, wl
        qkv, f = torch.randn(R, 4 * HD + 64, device=dev).to(bf), torch.randn(R, HD, device=dev).to(bf)
        kp = kda.KDAParams(torch.randn(3 * HD, 4, device=dev), None, torch.randn(H, device=dev), torch.randn(HD, device=dev),
                           torch.ones(D, device=dev))
        cs, rs = torch.zeros(B, 3 * HD, 3, device=dev), torch.zeros(B, H, D, D, device=dev)
        ms = timer(lambda: kda.kda_forward(qkv[:, :3 * HD], f, qkv[:, 4 * HD:4 * HD + H], qkv[:, 3 * HD:4 * HD], kp, cs, rs,
                                           slots, cu, init, H, D, D ** -0.5, 1e-6))
        add("  KDA", size, ms, (R * HD * 12 + B * HD * (D * 8 + 3 * 3 * 8)) / 1e9)
    talk = torch.randn(H, H, device=dev) / 6
    for B, ctx in ((16, 4096), (64, 4096)):
        n = B * ctx // page
        cache = torch.randn(n, page, 2 * G * D, device=dev).to(bf)
        bt = torch.randperm(n, device=dev).to(torch.int32).view(B, -1).contiguous()
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q, out = torch.randn(B, HD, device=dev), torch.empty(B, HD, dtype=bf, device=dev)
        p = talking.TalkParams(H, G, D, D, D ** -0.5, ctx, True, talk)
        gb = B * ctx * 2 * G * D * 2 / 1e9
        add("attention, decode", f"{B} x {ctx} keys", timer(lambda: talking.attend_rows(q, p, cache, bt, lens, out)), gb)
        qb = q.to(bf).view(B, H, D)
        sinks = torch.zeros(H, device=dev)
        add("  GQA decode", f"{B} x {ctx} keys",
            timer(lambda: attention.gqa_decode(qb, cache, bt, lens, G, D ** -0.5, sinks=sinks)), gb)
    for T, chunk in ((4096, 4096), (8192, 2048)):
        n = T // page
        cache = torch.randn(n, page, 2 * G * D, device=dev).to(bf)
        bt = torch.arange(n, device=dev, dtype=torch.int32).view(1, -1).contiguous()
        q, out = torch.randn(T, HD, device=dev), torch.empty(T, HD, dtype=bf, device=dev)
        p = talking.TalkParams(H, G, D, D, D ** -0.5, chunk, True, talk)
        pairs = T * (chunk + 1) / 2
        blocks = talking.work_blocks(talking.prefill_work([0, T], [0], chunk), T, dev)
        size = f"{T} tokens, chunks of {chunk}"
        add("attention, prompt", size, timer(lambda: talking.attend_prefill(q, p, cache, bt, out, blocks)), 0,
            pairs * 2 * H * (2 * D + H) / 1e12)
        q3, kv = torch.randn(T, H, 192, device=dev).to(bf), torch.randn(T, H, 256, device=dev).to(bf)
        kpe = torch.randn(T, 64, device=dev).to(bf)
        cu = list(range(0, T + 1, chunk))
        work = attention.mha_prefill_work(cu, [0] * (len(cu) - 1), cu[:-1]).to(dev)
        add("  expanded MLA prompt", size, timer(lambda: attention.mha_prefill(q3, kv, kpe, work, 0.07)), 0,
            pairs * 2 * H * 320 / 1e12)
    return rows


def run(args, root: str) -> int:
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
    for cfg in (get_model_config("nanurax-bench"), _closest()):
        models[cfg.name] = _model_rates(cfg, dev, timer)
    kernels = _kernels(dev, timer, peaks)
    _ext.check_status()
    value = models["nanurax-bench"]["decode"][1]["tok_per_s"]
    print(json.dumps({
        "metric": "decode tokens/s, 64 rows at 2,048 context, four layers (Nanurax)", "value": value, "unit": "tokens/s",
        "n_gpus": 1, "steps": args.steps, "warmup": timer.warmup, "ms_per_step": models["nanurax-bench"]["decode"][1]["ms"],
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"model": "nanurax-bench", "closest": "kimi-linear cut to four layers", "l2": "flushed before every call",
                   "parallelism": "1 GPU"},
        "models": models, "kernels": kernels, "peaks": peaks, "clocks": sampler.stop(),
        "gpu_launches": _ext.LAUNCHES["count"] - l0}))
    return 0
