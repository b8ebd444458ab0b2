"""Small Nanurax configurations and models for the tests."""
import torch

import nanurax_oracle as oracle


def delta(heads, dim, mlp=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, chunk, mlp=None, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                      "mask": {"size": chunk}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit, shared=None, shared_limit=0.7):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def config(vocab, width, layers, eps=1e-5, scale=7.0):
    return {"architecture": "Nanurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


# sizes that leave nothing equal, aligned or 1 by accident, and one where everything is
CONFIGS = {
    # odd widths everywhere: no size is a multiple of 8, value heads wider than key heads, several experts a token
    "odd": config(203, 100, [delta(3, 20, dense(90)), attention(6, 2, 12, 20, 37, moe(36, 7, 3, 0.9, 52)),
                             delta(2, 36, moe(44, 5, 2, 1.1))], eps=3e-5),
    # attention first and twice, with different shapes; a layer without a feed-forward; mixtures without a shared expert
    "twice": config(160, 128, [attention(4, 4, 32, 16, 64, None), delta(1, 64, moe(64, 4, 4, 2.0, 64)),
                               attention(8, 1, 40, 24, 100, dense(192))], scale=1.0),
    # one head of everything, one expert
    "ones": config(96, 64, [attention(1, 1, 16, 16, 16, moe(64, 1, 1, 1.0, 64)), delta(1, 16, dense(64))]),
    # recurrent layers only: no paged rows at all
    "recurrent": config(120, 72, [delta(2, 24, dense(72)), delta(4, 8, None)]),
    # attention only: no state slots
    "attention": config(120, 96, [attention(9, 3, 16, 16, 50, dense(64)), attention(2, 1, 48, 48, 130, None)]),
}


def weights_of(d, seed=0, rank=11):
    return oracle.random_weights(d, seed, rank)


def build(d, weights, device="cpu", dtype="fp32"):
    from batchgen_b200.config import nanurax_config
    from batchgen_b200.models import build_model
    ranks = {i: weights[f"l{i}.mix.w1"].shape[0] for i in range(len(d["layers"])) if f"l{i}.mix.w1" in weights}
    cfg = nanurax_config(d, "test-nanurax", ranks)
    return build_model(cfg, device=device, dtype=dtype, loader=lambda name, shape: weights[name])


def engine(model, tokens=1024, slots=4, page=64, **kw):
    from batchgen_b200.config import EngineConfig
    from batchgen_b200.runtime.engine import Engine
    dev = str(model.device)
    return Engine(model, EngineConfig(page_size=page, device=dev, dtype="bf16" if model.dtype == torch.bfloat16 else "fp32",
                                      max_decode_batch=slots, max_state_slots=slots, enable_cuda_graph=False, **kw),
                  num_gpu_pages=-(-tokens // page))


def prompt(d, n, seed=0):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, d["vocab"], (n,), generator=g).tolist()


def error(got, want):
    """Root mean square of the difference of centred logits, relative to the reference's spread (worst row)."""
    return float(row_errors(got, want).max())


def chooses_experts(d):
    """Some router picks fewer experts than there are: 16-bit rounding can flip a close choice."""
    return any(l["mlp"] and l["mlp"]["kind"] == "moe" and l["mlp"]["router"]["top"] < l["mlp"]["router"]["experts"]
               for l in d["layers"])


def row_errors(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    got, want = got - got.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()


def close(got, want, tol, d):
    """Every row within ``tol``; in 16 bits a model that chooses experts may have rows past a flipped close choice."""
    e = row_errors(got, want)
    if tol > 1e-3 and chooses_experts(d):
        return bool((e > tol).double().mean() <= 0.15 and e.median() < tol / 2)
    return bool(e.max() < tol)


def run_pieces(eng, seq, tokens, sizes):
    """Feed ``tokens`` in pieces of the given sizes (the last size repeats); logits of every position."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        out.append(eng.extend([(seq, tokens[at:at + n], range(n))]).float().cpu())
        at, i = at + n, i + 1
    return torch.cat(out)
