"""Small Pamevik configurations and models for the tests."""
import pamevik_oracle as oracle
from nanurax_models import engine, error, prompt, row_errors, run_pieces  # noqa: F401  (shared by the tests)


def channel_delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def parallel(left, right, mlp=None, scale=None):
    """left: (heads, kv_heads, dim, vdim, rotary dims, base); right: (decays, dim, vdim, rotary dims, base)."""
    h, g, d, dv, rd, base = left
    decay, rdim, rdv, rrd, rbase = right
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": h, "kv_heads": g, "dim": d, "vdim": dv, "scale": scale or d ** -0.5, "rot": {"base": base, "dims": rd}},
        "right": {"heads": len(decay), "dim": rdim, "vdim": rdv, "decay": decay, "rot": {"base": rbase, "dims": rrd}}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(vocab, width, layers, eps=1e-5, taps=4):
    return {"architecture": "Pamevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "layers": layers}


CONFIGS = {
    # nothing equal, aligned or 1: shared key heads, partial rotations of different bases, every layer's own sizes
    "odd": config(203, 100, [channel_delta(6, 2, 20, 28, 3, dense(90)),
                             parallel((6, 2, 12, 20, 8, 300.0), ([0.8, 0.95, 0.999], 20, 12, 14, 5000.0), dense(76)),
                             mlstm(3, 12, 36, 7.0), channel_delta(2, 2, 36, 12, 4)], eps=3e-5, taps=3),
    # one head of everything, convolutions of a single tap
    "ones": config(96, 64, [parallel((1, 1, 16, 16, 16, 100.0), ([0.9], 8, 8, 8, 100.0)), channel_delta(1, 1, 8, 16, 1, dense(64)),
                            mlstm(1, 8, 8, 3.0, dense(32))], taps=1),
    # heads as wide as the decode kernels take, whole tiles everywhere
    "whole": config(160, 128, [mlstm(2, 128, 128, 20.0, dense(128)), channel_delta(1, 1, 128, 64, 2),
                               parallel((4, 4, 64, 64, 64, 1e4), ([0.97, 0.99], 64, 128, 64, 1e4), dense(64))], taps=2),
    # wider than that: decoding goes through the scan; long convolutions
    "wide": config(120, 136, [channel_delta(2, 1, 136, 48, 6), mlstm(1, 40, 200, 11.0),
                              parallel((2, 1, 160, 72, 96, 700.0), ([0.93], 232, 152, 100, 900.0), dense(48))], taps=7),
    # recurrent layers only: no paged rows at all
    "recurrent": config(120, 72, [mlstm(2, 24, 16, 9.0, dense(72)), channel_delta(4, 4, 8, 24, 5), mlstm(3, 8, 40, 15.0)], taps=4),
    # attention beside retention only, twice, with different row widths
    "beside": config(120, 96, [parallel((9, 3, 16, 40, 6, 50.0), ([0.6, 0.99], 24, 16, 24, 1e5), dense(64)),
                               parallel((2, 1, 48, 24, 48, 1e6), ([0.9, 0.95, 0.97, 0.5], 16, 32, 2, 10.0))], taps=5),
}


def weights_of(d, seed=0, ranks=(11, 9)):
    return oracle.random_weights(d, seed, ranks)


def build(d, weights, device="cpu", dtype="fp32"):
    from batchgen_b200.config import pamevik_config
    from batchgen_b200.models import build_model
    ranks = {i: (weights[f"l{i}.mix.a1"].shape[0], weights[f"l{i}.mix.g1"].shape[0]) for i in range(len(d["layers"]))
             if f"l{i}.mix.a1" in weights}
    return build_model(pamevik_config(d, "test-pamevik", ranks), device=device, dtype=dtype, loader=lambda name, shape: weights[name])
