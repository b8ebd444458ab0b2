"""Small Bolisun configurations and models for the tests."""
import json
import random

import bolisun_oracle as oracle
from nanurax_models import engine, error, prompt, row_errors, run_pieces  # noqa: F401  (shared by the tests)


def scaling(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def layer(left, mask, rot, right, mlp=None, scales=(0.8, 1.2), scale=None):
    """left: (heads, kv_heads, dim, vdim); mask: (size, kept first); rot: (dims, base, scaling or None); right: (decays, dim, vdim)."""
    h, g, d, dv = left
    r = {"dims": rot[0], "base": rot[1]}
    if rot[2]:
        r["scaling"] = rot[2]
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left_scale": scales[0], "right_scale": scales[1],
        "left": {"heads": h, "kv_heads": g, "dim": d, "vdim": dv, "scale": scale or 1.3 * d ** -0.5, "rot": r,
                 "mask": {"size": mask[0], "keep_first": mask[1]}},
        "right": {"heads": len(right[0]), "dim": right[1], "vdim": right[2], "decay": list(right[0])}}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top, scale=1.7, groups=None, shared=0):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def again(d, j):
    return {**d, "weights_of": j}


def config(vocab, width, streams, layers, eps=1e-5, embed=1.5):
    return {"architecture": "Bolisun", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": embed}, "layers": layers}


_ODD = layer((6, 2, 20, 28), (37, 9), (12, 700.0, scaling(5.0, 90, 6.0, 0.7)), ((0.8, 0.95, 0.999), 20, 12),
             moe(44, 15, 4, 1.9, (5, 2), 60), (1.3, 0.6))
_ONE = layer((1, 1, 8, 16), (1, 0), (2, 100.0, None), ((0.9,), 8, 8), moe(24, 1, 1, 0.7), (1.0, 1.0), 1.0)
CONFIGS = {
    # nothing equal, aligned or 1; a mixture layer that runs three times, once before its own place
    "odd": config(203, 99, 3, [again(_ODD, 2), layer((9, 3, 12, 20), (50, 70), (6, 50.0, scaling(3.0, 40, 9.0, 2.0)),
                                                     ((0.7, 0.99), 28, 36), dense(76, 0.9), (0.5, -0.9)),
                               _ODD, layer((2, 2, 36, 12), (23, 0), (36, 9000.0, None), ((0.96,), 12, 20)), again(_ODD, 0)], 3e-5),
    # one stream, one head, one expert, a window of the position alone, then one more with a single kept token
    "ones": config(96, 64, 1, [_ONE, layer((1, 1, 16, 8), (1, 1), (16, 30.0, scaling(1.0, 64, 4.0, 1.0)), ((1.0,), 16, 16),
                                           moe(16, 6, 1, 2.2, (6, 1), 8))], embed=1.0),
    # whole tiles everywhere, windows and kept tokens on page borders
    "whole": config(160, 128, 2, [layer((2, 2, 128, 128), (64, 64), (128, 1e4, scaling(8.0, 256, 32.0, 1.0)),
                                        ((0.97, 0.99), 128, 128), dense(128, 1.1)),
                                  layer((8, 1, 64, 64), (128, 32), (64, 1e6, None), ((0.95,) * 4, 64, 64),
                                        moe(64, 8, 2, 1.0, (2, 1), 64))]),
    # heads wider than the prompt kernel takes, wider states than the decode ring takes, more streams than one block of them
    "wide": config(120, 72, 5, [layer((2, 1, 264, 72), (40, 3), (96, 700.0, scaling(2.0, 50, 3.0, 1.0)), ((0.93,), 152, 136),
                                      moe(40, 7, 3, 1.2)), layer((3, 3, 72, 264), (90, 20), (72, 200.0, None), ((0.6, 0.98), 40, 200),
                                                                 dense(48, 2.0))]),
    # mixtures without groups or a shared expert, many streams
    "streams": config(140, 80, 9, [layer((4, 4, 16, 24), (30, 2), (16, 80.0, None), ((0.9, 0.99), 16, 24), moe(32, 12, 5)),
                                   layer((4, 2, 24, 16), (300, 0), (8, 80.0, scaling(6.0, 30, 4.0, 0.5)), ((0.99, 0.5), 24, 16))]),
}


def without_choices(d):
    """The same design with every expert chosen: rounding flips nothing."""
    d = json.loads(json.dumps(d))
    for x in d["layers"]:
        if (x["mlp"] or {}).get("kind") == "moe":
            x["mlp"]["router"].pop("groups", None)
            x["mlp"]["router"]["top"] = x["mlp"]["router"]["experts"]
    return d


def random_config(seed):
    """A design of random sizes, constants and order of layers."""
    r = random.Random(seed)

    def some():
        g = r.choice((1, 1, 2, 3))
        d, rd = r.randint(2, 40) * 2, 0
        rd = r.randint(1, d // 2) * 2
        sc = scaling(r.choice((1.0, 2.5, 16.0)), r.randint(20, 400), r.uniform(4, 40), r.uniform(0.3, 3)) if r.random() < 0.7 else None
        kind = r.random()
        f = None if kind < 0.2 else dense(r.randint(3, 150), r.uniform(0.4, 3))
        if kind > 0.55:
            count, size = r.randint(1, 5), r.randint(1, 5)
            keep = r.randint(1, count)
            f = moe(r.randint(3, 90), count * size, r.randint(1, min(keep * size, 6)), r.uniform(0.5, 3),
                    (count, keep) if r.random() < 0.8 or keep < count else None, r.choice((0, r.randint(3, 90))))
        return layer((g * r.randint(1, 5), g, d, r.randint(1, 90)), (r.randint(1, 150), r.choice((0, 1, r.randint(2, 90)))),
                     (rd, r.choice((20.0, 1e4, 3e5)), sc), ([r.uniform(0.5, 1.0) for _ in range(r.randint(1, 4))],
                                                            r.randint(1, 80), r.randint(1, 80)), f,
                     (r.uniform(0.2, 1.5), r.uniform(-1.5, 1.5)))
    layers = [some() for _ in range(r.randint(1, 4))]
    for _ in range(r.randint(0, 2)):
        j = r.randrange(len(layers))
        layers.append(again(layers[j], j))
    return config(r.randint(30, 300), r.randint(9, 140), r.randint(1, 6), layers, 10 ** r.uniform(-6, -4), r.uniform(0.5, 4))


def weights_of(d, seed=0, settled=False):
    return oracle.random_weights(d, seed, settled)


def build(d, weights, device="cpu", dtype="fp32"):
    from batchgen_b200.config import bolisun_config
    from batchgen_b200.models import build_model
    return build_model(bolisun_config(d, "test-bolisun"), device=device, dtype=dtype, loader=lambda name, shape: weights[name])
