"""Small Pitudra configurations and models for the tests."""
import json
import random

import pitudra_oracle as oracle
from nanurax_models import engine, error, prompt, row_errors, run_pieces  # noqa: F401  (shared by the tests)


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def hgrn2(heads, dim, vdim, mlp=None):
    return {"type": "hgrn2", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def _mask(window):
    """No window: every earlier token is seen."""
    return {"mask": {"size": window}} if window else {}


def attention(heads, kv_heads, dim, vdim, window, mlp=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5}
    return {"type": "attention", "mlp": mlp, "mixer": {**m, **_mask(window)}}


def latent(heads, dim, rot, vdim, q_rank, kv_rank, window, mlp=None, base=700.0, kv_from=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, **_mask(window),
         "scale": scale or 1.3 * (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def config(vocab, width, layers, side=None, eps=1e-5):
    d = {"architecture": "Pitudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side:
        d["token_side"] = {"dim": side}
    return d


CONFIGS = {
    # nothing equal, aligned or 1; latents borrowed by two layers, one of them with a longer window than their owner
    "odd": config(203, 99, [latent(5, 20, 6, 12, 35, 50, 37, moe(44, 7, 3)), hgrn2(3, 20, 28, moe(36, 5, 2)),
                            attention(6, 2, 12, 20, 23, moe(52, 6, 1)), latent(3, 12, 6, 28, 51, 50, 90, moe(28, 3, 2), kv_from=0),
                            hgrn2(2, 36, 12), latent(7, 9, 6, 9, 13, 50, 5, kv_from=0)], 11, 3e-5),
    # one head, one expert, windows of the position alone; no side input
    "ones": config(96, 64, [attention(1, 1, 8, 8, 1, moe(24, 1, 1), 1.0), latent(1, 8, 2, 8, 8, 8, 1, moe(16, 6, 6)),
                            hgrn2(1, 8, 8, moe(16, 4, 1))]),
    # whole tiles everywhere, windows on page borders
    "whole": config(160, 128, [hgrn2(2, 128, 128, moe(128, 8, 2)), attention(8, 1, 64, 64, 64, moe(64, 4, 2)),
                               latent(4, 64, 64, 64, 128, 128, 128, moe(64, 4, 2), 1e6), attention(2, 2, 128, 128, 0)], 64),
    # heads and latents wider than the tensor-core kernels take, wider states than the decode ring takes, more than 32 heads
    "wide": config(120, 72, [latent(2, 200, 72, 264, 40, 584, 40, moe(40, 5, 2)), hgrn2(1, 152, 136, moe(48, 3, 1)),
                             attention(3, 1, 264, 72, 90), latent(35, 8, 72, 16, 24, 584, 300, kv_from=0),
                             latent(33, 24, 8, 16, 40, 520, 0)], 136),
    # latent layers alone, several widths of the score kernel
    "latents": config(140, 80, [latent(16, 16, 16, 24, 32, 200, 100, moe(32, 12, 5)), latent(4, 24, 8, 16, 24, 96, 33),
                                latent(24, 16, 16, 32, 40, 200, 64, moe(24, 4, 2), kv_from=0), latent(20, 32, 32, 32, 64, 400, 200)], 24),
    # recurrent layers only: no paged rows at all
    "recurrent": config(110, 60, [hgrn2(4, 16, 24, moe(20, 3, 1)), hgrn2(2, 24, 40)], 7),
}


def without_choices(d):
    """The same design with every expert chosen: rounding flips nothing."""
    d = json.loads(json.dumps(d))
    for x in d["layers"]:
        if x["mlp"]:
            x["mlp"]["router"]["top"] = x["mlp"]["router"]["experts"]
    return d


def random_config(seed):
    """A design of random sizes, constants and order of layers."""
    r = random.Random(seed)
    layers, owners = [], []
    for i in range(r.randint(1, 5)):
        e = r.randint(1, 9)
        f = moe(r.randint(3, 90), e, r.randint(1, min(e, 6))) if r.random() < 0.7 else None
        kind = r.random()
        if kind < 0.3:
            layers.append(hgrn2(r.randint(1, 4), r.randint(1, 80), r.randint(1, 80), f))
        elif kind < 0.55:
            g = r.choice((1, 1, 2, 3))
            layers.append(attention(g * r.randint(1, 5), g, r.randint(1, 70), r.randint(1, 90), r.randint(1, 150), f))
        else:
            j = r.choice(owners) if owners and r.random() < 0.5 else None
            rank, rot, base = ((layers[j]["mixer"][k] for k in ("kv_rank", "rot_dim", "rot")) if j is not None
                               else (r.randint(2, 150), 2 * r.randint(1, 20), {"base": r.choice((20.0, 1e4, 3e5))}))
            layers.append(latent(r.randint(1, 20), r.randint(1, 60), rot, r.randint(1, 60), r.randint(2, 90), rank, r.randint(1, 150), f,
                                 base["base"], j))
            if j is None:
                owners.append(i)
    return config(r.randint(30, 300), r.randint(9, 140), layers, r.choice((None, r.randint(1, 50))), 10 ** r.uniform(-6, -4))


def weights_of(d, seed=0, settled=False):
    return oracle.random_weights(d, seed, settled)


def build(d, weights, device="cpu", dtype="fp32"):
    from batchgen_b200.config import pitudra_config
    from batchgen_b200.models import build_model
    return build_model(pitudra_config(d, "test-pitudra"), device=device, dtype=dtype, loader=lambda name, shape: weights[name])
