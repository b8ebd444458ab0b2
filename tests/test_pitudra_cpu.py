"""Pitudra on the CPU path: configuration, weights from a directory, engine steps in any cut, scheduler and CLI."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import pitudra_models as pm
import pitudra_oracle as oracle

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F64 = torch.float64


def _save(path, d, weights):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(d, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))


def _gen(seed):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------- the plain implementation itself
def test_plain_rotation_pairs_halves():
    x = torch.zeros(3, 1, 4, dtype=F64)
    x[:, 0, 0], x[:, 0, 3] = 1.0, 2.0
    y = oracle.rotate(x, 100.0)
    for p in range(3):
        want = [np.cos(p), -2 * np.sin(p * 0.1), np.sin(p), 2 * np.cos(p * 0.1)]
        assert torch.allclose(y[p, 0], torch.tensor(want, dtype=F64))


def test_plain_window_shift_and_norms_on_cases_with_known_answers():
    assert [[j for j in range(5) if oracle.visible(5, 2)[i, j]] for i in range(5)] == [[0], [0, 1], [1, 2], [2, 3], [3, 4]]
    h = torch.tensor([[1.0, 2.0], [5.0, 6.0], [7.0, 0.0]])
    assert oracle.token_shift(h, torch.tensor([0.25, 1.0])).tolist() == [[0.75, 0.0], [4.0, 2.0], [6.5, 6.0]]
    x = torch.tensor([[1.0, 3.0]], dtype=F64)
    assert torch.allclose(oracle.layer_norm(x, torch.tensor([2.0, 2.0]), torch.tensor([0.5, 0.0]), 0.0), torch.tensor([[-1.5, 2.0]], dtype=F64))
    assert torch.allclose(oracle.rms(torch.tensor([[3.0, 4.0]], dtype=F64), 3.5), torch.tensor([[0.75, 1.0]], dtype=F64))


def test_plain_sink_takes_its_share_and_has_no_value():
    s = torch.log(torch.tensor([[1.0, 2.0, 50.0]], dtype=F64))
    p = oracle.sink_softmax(s, torch.tensor([[True, True, False]]), torch.log(torch.tensor(5.0, dtype=F64)))
    assert torch.allclose(p, torch.tensor([[1 / 8, 2 / 8, 0]], dtype=F64))
    p = oracle.sink_softmax(s - 700, torch.tensor([[True, True, False]]), torch.tensor(600.0, dtype=F64))
    assert float(p.sum()) == 0


def test_plain_recurrence_router_and_expert_on_cases_with_known_answers():
    half, one = torch.full((3, 1, 1), 0.5, dtype=F64), torch.ones(3, 1, 1, dtype=F64)
    assert torch.allclose(oracle.hgrn2(one, half, one)[0].flatten(), torch.tensor([0.5, 0.75, 0.875], dtype=F64))
    assert float(oracle.forget(torch.tensor(0.0), torch.tensor(0.6))) == pytest.approx(0.8)
    idx, w = oracle.route(torch.log(torch.tensor([[1.0, 9.0, 3.0, 2.0]], dtype=F64)), 2)
    assert idx.tolist() == [[1, 2]] and torch.allclose(w, torch.tensor([[0.75, 0.25]], dtype=F64))
    w = {"up": torch.tensor([[1.0], [-1.0]]), "down": torch.tensor([[1.0, 10.0]])}
    assert oracle.expert(torch.tensor([[2.0], [-3.0]]), w, "").flatten().tolist() == [4.0, 90.0]


# ---------------------------------------------------------------- mechanisms of the CPU path
def test_routed_rows_join_behind_their_norm_and_the_next_sublayer_reads_the_residual():
    from batchgen_b200.ops import residual
    T, D, g = 5, 10, _gen(4)
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    x, routed = torch.zeros(T, 12), torch.zeros(9, 12)
    x[:, :D], routed[:, :D] = r(T, D), r(9, D)
    x[:, D:] = float("nan")                          # what memory held before
    pos = torch.randint(-1, 9, (T, 4), generator=g).to(torch.int32)
    rw, w, b = torch.rand(T, 4, generator=g), torch.zeros(12), torch.zeros(12)
    w[:D], b[:D] = 1 + 0.2 * r(D), r(D)
    y = sum(torch.where(pos[:, k:k + 1] >= 0, rw[:, k:k + 1] * routed[pos[:, k].clamp_min(0).long()], torch.zeros(1)) for k in range(4))[:, :D]
    want = x[:, :D] + oracle.layer_norm(y, w[:D], b[:D], 1e-5)
    h = residual.sandwich_norm(x, None, 1e-5, D, 64, torch.float32, routed=routed, pos=pos, route_w=rw, post=residual.Norm(w, b, True))
    assert torch.allclose(x[:, :D], want, atol=1e-5) and torch.allclose(h[:, :D], want, atol=1e-5) and float(h[:, D:].abs().sum()) == 0
    assert float(x[:, D:].abs().sum()) == 0
    before = x.clone()
    assert residual.sandwich_norm(x, None, 1e-5, D, 64, torch.float32, add=y, post=residual.Norm(w), emit=False) is None
    assert torch.allclose(x[:, :D], before[:, :D] + oracle.rms(y, 1e-5) * w[:D], atol=1e-5)


def test_token_shift_is_a_convolution_of_two_taps():
    from batchgen_b200.ops import conv
    g = _gen(5)
    h, mu, hist = torch.randn(9, 12, generator=g), torch.rand(12, generator=g), torch.full((2, 12), 7.0)
    w = torch.stack([mu, -mu])
    out = torch.zeros(9, 64)
    conv.causal_conv(h, w, hist, torch.tensor([1]), out, "residual", cu_host=[0, 9], has_initial=[0])
    assert torch.allclose(out[:, :12], oracle.token_shift(h, mu), atol=1e-6) and torch.equal(hist[1], h[8]) and float(hist[0, 0]) == 7


def test_side_rows_and_squared_relu_experts():
    from batchgen_b200.ops import moe, residual
    g = _gen(6)
    z, table, ids = torch.randn(7, 16, generator=g), torch.randn(5, 11, generator=g), torch.tensor([0, 4, 2, 2, 1, 3, 0], dtype=torch.int32)
    y = residual.token_side(z, table, ids, 64, torch.float32)
    assert torch.allclose(y[:, :11], oracle.gelu_tanh(z[:, :11]) * table[ids.long()], atol=1e-6) and float(y[:, 11:].abs().sum()) == 0
    w = {f"e{e}.{x}": torch.randn(*s, generator=g) for e in range(3) for x, s in (("up", (20, 12)), ("down", (12, 20)))}
    ew = moe.ExpertWeights(torch.stack([w[f"e{e}.up"] for e in range(3)]), torch.stack([w[f"e{e}.down"] for e in range(3)]), activation="relu2")
    x, idx = torch.randn(4, 12, generator=g), torch.tensor([[0, 2], [1, 0], [2, 1], [0, 1]], dtype=torch.int32)
    rows, pos = moe.routed_rows(x, idx, torch.ones(4, 2), ew, False)
    for t in range(4):
        for k in range(2):
            assert torch.allclose(rows[pos[t, k]], oracle.expert(x[t], w, f"e{int(idx[t, k])}."), atol=1e-4)


@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_one_outstanding_key_at_every_kind_of_place(kind):
    """The query asks for exactly one key: the window's first key and the one before it, page borders, neighbours, itself; with a small
    sink it answers, with a large one it does not."""
    from batchgen_b200.ops import latent, talking
    n, i, window, H, d, dv, page = 150, 140, 70, 2, 16, 8, 16
    bt = torch.arange(10).view(1, -1).flip(1).to(torch.int32)
    for j in (0, i - window, i - window + 1, i - window + 2, 63, 64, 79, 80, i - 1, i):
        g = _gen(j)
        q, k, v = (0.1 * torch.randn(n, h, w, generator=g) for h, w in ((H, d), (1, d), (1, dv)))
        q[i, :, 3] = 6.0
        k[j, :, 3] = 9.0
        v[j] += 50.0
        for sink in (-3.0, 80.0):
            sinks = torch.tensor([sink, 2.0])
            if kind == "latent":                                    # the value is the row's own head of numbers
                v = k[..., :dv]
                p = latent.LatentParams(H, 8, 8, 8, dv, dv, dv, 1, 1.0, 0.0, window, sinks, None, None, None, None, None)
            seen = oracle.visible(n, window)
            want = oracle.attention(q, k, v, 1.0, seen, sinks)[i]
            assert (float(want[1].abs().max()) > (40 if kind == "attention" else 8)) == (i - window < j)
            cache = torch.zeros(10, page, d + dv if kind == "attention" else d)
            rows = torch.cat([k[:, 0], v[:, 0]], 1) if kind == "attention" else k[:, 0]
            slots = bt[0, torch.arange(n) // page].long() * page + torch.arange(n) % page
            talking.kv_write(rows, slots, cache)
            lens = torch.arange(1, n + 1)
            seq = torch.zeros(n, dtype=torch.int32)
            if kind == "attention":
                out = torch.zeros(n, H * dv)
                talking.attend_rows(q.reshape(n, -1), talking.TalkParams(H, 1, d, dv, 1.0, window=window, sinks=sinks), cache, bt, lens, out, seq)
            else:
                out = latent.attend(q.contiguous(), p, cache, bt, lens, seq)
            assert torch.allclose(out.view(n, H, dv)[i], want, atol=1e-4), (j, sink)


# ---------------------------------------------------------------- whole model, any cut
@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name):
    d = pm.CONFIGS[name]
    w = pm.weights_of(d, seed=1)
    toks = pm.prompt(d, 150)
    trace = []
    want = oracle.forward(d, w, toks, F64, trace)
    model = pm.build(d, w)
    layers = {}
    model.layer_hook = lambda l, x: layers.__setitem__(l, x.clone())
    eng = pm.engine(model)
    s = eng.open_sequence()
    assert pm.error(eng.extend([(s, toks, range(150))]), want) < 5e-5
    for l, x in enumerate(trace):
        assert torch.allclose(layers[l].double(), x, atol=2e-4 * float(x.abs().max())), l
    model.layer_hook = None
    eng.close_sequence(s)
    for sizes in ([2], [1], [63, 1, 2, 5], [100, 1]):
        s = eng.open_sequence()
        assert pm.error(pm.run_pieces(eng, s, toks, sizes), want) < 5e-5, sizes
        eng.close_sequence(s)
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("seed", range(8))
def test_random_designs(seed):
    d = pm.random_config(seed)
    w = pm.weights_of(d, seed)
    toks = pm.prompt(d, 90)
    want = oracle.forward(d, w, toks, F64)
    eng = pm.engine(pm.build(d, w))
    for sizes in ([90], [31, 2, 1]):
        assert pm.error(pm.run_pieces(eng, eng.open_sequence(), toks, sizes), want) < 1e-4


def test_every_weight_takes_part():
    """A tensor that is read but not used would not show in a comparison with itself: changing any one of them has to change
    the logits, and by the same amount as in the plain implementation."""
    d = pm.CONFIGS["odd"]
    base = pm.weights_of(d, seed=4)
    toks = pm.prompt(d, 45)
    plain = oracle.forward(d, base, toks, F64)
    names = [n for n in sorted(base) if ".mlp.e" not in n or n.split(".")[2] in ("e0", "e2", "e5")]
    for name in names:
        w = dict(base)
        w[name] = base[name] + (0.3 * base[name].std() + 0.02) * torch.randn(base[name].shape, generator=_gen(5))
        if name.endswith("lower"):
            w[name] = w[name].clamp(0.01, 0.99)
        want = oracle.forward(d, w, toks, F64)
        assert pm.error(plain, want) > 2e-3, name
        eng = pm.engine(pm.build(d, w))
        assert pm.error(eng.extend([(eng.open_sequence(), toks, range(45))]), want) < 1e-4, name


def test_borrowed_latents_take_no_room_in_the_cache():
    d = pm.CONFIGS["odd"]
    eng = pm.engine(pm.build(d, pm.weights_of(d)))
    assert sorted(eng.kv.layer_rows) == [0, 2] and eng.kv.layer_rows[0][1] == 56 + 8 and eng.cfg.kv_cache_dim == 64 + 2 * (16 + 24)


def test_unequal_batches_equal_each_request_alone_and_places_are_used_again():
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=2)
    eng = pm.engine(pm.build(d, w), tokens=64 * 7)
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((130, 1, 41, 77, 3, 64))]
    want = [oracle.forward(d, w, p, F64) for p in prompts]
    live, at, got = {}, [0] * 6, [[] for _ in prompts]
    order, rng = list(range(6)), _gen(5)
    while order or live:
        while order and len(live) < 3:
            live[order[0]] = eng.open_sequence()
            order.pop(0)
        pieces = []
        for i, s in live.items():
            if torch.rand(1, generator=rng) < 0.25 and len(live) > 1:
                continue                                      # left out of this step
            n = min(int(torch.randint(1, 40, (1,), generator=rng)), len(prompts[i]) - at[i])
            pieces.append((i, s, n))
        if not pieces:
            continue
        out = eng.extend([(s, prompts[i][at[i]:at[i] + n], range(n)) for i, s, n in pieces])
        for (i, s, n), rows in zip(pieces, out.split([p[2] for p in pieces])):
            got[i].append(rows)
            at[i] += n
            if at[i] == len(prompts[i]):
                eng.close_sequence(live.pop(i))
    for g, x in zip(got, want):
        assert pm.error(torch.cat(g), x) < 5e-5
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


def _greedy(d, w, toks, n):
    toks = list(toks)
    for _ in range(n):
        toks.append(int(oracle.forward(d, w, toks, F64)[-1].argmax()))
    return toks[-n:]


def test_greedy_generation_through_the_scheduler_with_chunks_holds_and_evictions():
    from batchgen_b200.config import EngineConfig
    from batchgen_b200.runtime.engine import Engine
    from batchgen_b200.runtime.sequence import SamplingParams
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=3)
    model = pm.build(d, w)
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((50, 9, 33, 21))]
    want = [_greedy(d, w, p, 20) for p in prompts]
    params = SamplingParams(max_new_tokens=20, ignore_eos=True)
    assert pm.engine(model).generate(prompts, params) == want
    # pieces of at most 16 prompt tokens, few state slots and pages of 8 tokens: rows wait, are evicted and recomputed
    tight = pm.engine(model, tokens=8 * 14, slots=3, page=8, max_prefill_tokens=16, initial_gpu_page_buffer=1,
                      extension_gpu_page_buffer=1, decision_frequency_pages=1)
    assert tight.generate(prompts, params) == want
    assert tight.stats.evictions > 0 and tight.stats.prefill_chunks > 0
    # a host tier: parked rows keep their state
    ecfg = EngineConfig(page_size=8, max_decode_batch=4, max_state_slots=3, initial_gpu_page_buffer=1,
                        extension_gpu_page_buffer=1, decision_frequency_pages=1, enable_cuda_graph=False)
    parked = Engine(model, ecfg, num_gpu_pages=14, num_host_pages=60)
    assert parked.generate(prompts, params) == want
    assert parked.stats.holds > 0 and parked.host_state.offloads > 0 and parked.host_state.loads > 0


# ---------------------------------------------------------------- registry, directories, command line
def test_config_directory_registry_and_validation(tmp_path):
    from batchgen_b200.ckpt.converter import convert_dir
    from batchgen_b200.config import ModelConfig, get_model_config, list_models, pitudra_config
    from batchgen_b200.models import build_model
    from batchgen_b200.models.weights import checkpoint_tensor_specs
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=4)
    _save(str(tmp_path / "m"), d, w)
    cfg = get_model_config(str(tmp_path / "m"))
    assert cfg.family == "pitudra" and cfg.token_shift and not cfg.pre_norm and cfg.side_dim == 11 and not cfg.is_mla
    assert [s.mixer.kv_from for s in cfg.layer_specs] == [-1, -1, -1, 0, -1, 0]
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg and {"tiny-pitudra", "pitudra-bench"} <= set(list_models())
    toks = pm.prompt(d, 40)
    want = oracle.forward(d, w, toks)
    eng = pm.engine(build_model(cfg))
    assert pm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), want) < 5e-5
    # the names the framework writes are the ones it reads; a converted copy of the directory serves as well
    for c in (d, pm.CONFIGS["ones"]):
        assert {n: s for n, s, _, _ in checkpoint_tensor_specs(pitudra_config(c))} == oracle.tensor_shapes(c)
    vectors = ("shift", "b", "lower", "sink", "norm1", "norm2")
    small = sum(t.numel() for k, t in w.items() if k.split(".")[-1] in vectors and not k.endswith((".q.b", ".k.b", ".v.b")))
    norms = sum(t.numel() for k, t in w.items() if k.endswith((".mix.norm", "side.norm", "dq.norm", "dkv.norm", "final.norm")))
    assert cfg.param_count() == sum(t.numel() for t in w.values()) - small - norms
    convert_dir(str(tmp_path / "m"), str(tmp_path / "c"))
    conv = get_model_config(str(tmp_path / "c"))
    assert conv.layer_specs == cfg.layer_specs
    eng = pm.engine(build_model(conv))
    assert pm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), want) < 5e-5
    mixer = lambda i, **kw: (lambda x: x["layers"][i]["mixer"].update(kw))      # noqa: E731
    for edit, match in ((lambda x: x["layers"][1].update(type="other_kind"), "other_kind"),
                        (mixer(2, kv_heads=4), "divide"), (mixer(2, mask={"size": 0}), "window"),
                        (mixer(0, rot={"base": 9.0, "dims": 4}), "rotary"), (mixer(3, kv_from=1), "none of its own"),
                        (mixer(5, kv_from=3), "none of its own"), (mixer(3, kv_from=3), "none of its own"),
                        (mixer(3, kv_rank=49), "another shape"), (mixer(5, rot={"base": 1.5, "dims": 6}), "another shape"),
                        (lambda x: x["layers"][0]["mlp"]["router"].update(top=8), "top 8"),
                        (lambda x: x["layers"][0]["mlp"].update(kind="sparse"), "sparse")):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(ValueError, match=match):
            pitudra_config(bad)
    del w["l2.mlp.e3.up"]
    _save(str(tmp_path / "short"), d, w)
    with pytest.raises(KeyError, match="l2.mlp.e3.up"):
        build_model(get_model_config(str(tmp_path / "short")))


def test_trace_replay_command(tmp_path):
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=6)
    _save(str(tmp_path / "m"), d, w)
    a, b = pm.prompt(d, 70, 1), pm.prompt(d, 30, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:69], "want": [0, 18]}, {"id": "b", "tokens": b, "want": [29]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[69:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype",
                        "float32", "--device", "cpu", "--out", str(out), "--max-tokens", "192"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", text=True, capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    la, lb = oracle.forward(d, w, a), oracle.forward(d, w, b)
    got = torch.from_numpy(np.fromfile(out / "1.f32", "<f4").reshape(3, -1).copy())
    assert pm.error(got, torch.stack([la[50], la[68], lb[29]])) < 5e-5
    got = torch.from_numpy(np.fromfile(out / "2.f32", "<f4").reshape(1, -1).copy())
    assert pm.error(got, la[69:70]) < 5e-5


def test_planner_and_preflight_know_the_design():
    from batchgen_b200.config import EngineConfig, get_model_config, pitudra_config
    from batchgen_b200.runtime import planner
    from batchgen_b200.runtime.kv_cache import PagedKVCache, host_page_bytes
    from batchgen_b200.server.preflight import PreflightError, model_contract
    cfg = get_model_config("pitudra-bench")
    assert cfg.kv_cache_dim == 8 * 256 + 576 and host_page_bytes(cfg, 64) == 64 * (8 * 256 + 576) * 2
    ecfg = EngineConfig(max_decode_batch=64, max_prefill_tokens=8192)
    assert planner.state_pool_bytes(cfg, ecfg) == 64 * 4 * (2 * 32 * 128 * 128 + 4 * 2304)
    dense, experts = planner.weight_bytes_per_rank(cfg, 1, 1)
    assert experts == 4 * 64 * 2 * 2304 * 1536 * 2
    assert planner.plan_deployment(cfg, ecfg, planner.MACHINES["b200"]).fits
    tiny = get_model_config("tiny-pitudra")
    kv = PagedKVCache(tiny, 2, 16, "cpu", torch.float32, state_slots=3)
    assert kv.state.row_floats >= tiny.layered_state_floats_per_seq() and kv.state.layer(2, "shift").shape == (4, 120)
    assert model_contract(tiny, 1, True)
    with pytest.raises(PreflightError, match="one GPU"):
        model_contract(tiny, 2, True)
    for layer, match in ((pm.hgrn2(1, 520, 8), "512"), (pm.latent(1, 8, 8, 8, 8, 1600, 4), "latent"),
                         (pm.attention(300, 2, 128, 8, 4), "norm"), (pm.attention(1, 1, 8, 8, 4, pm.moe(8, 40, 17)), "experts")):
        with pytest.raises(PreflightError, match=match):
            model_contract(pitudra_config(pm.config(64, 64, [layer])), 1, True)


def test_server_serves_a_model_directory(tmp_path):
    import time

    from fastapi.testclient import TestClient

    from batchgen_b200.server.http_server import create_app
    from batchgen_b200.server.server_args import ServerArgs, validate_server_args
    d = pm.config(300, 48, [pm.latent(4, 8, 4, 8, 16, 24, 12, pm.moe(24, 6, 2)), pm.hgrn2(2, 8, 16), pm.attention(4, 2, 8, 8, 9, pm.moe(16, 3, 1)),
                            pm.latent(2, 8, 4, 8, 16, 24, 30, kv_from=0)], 8)
    w = pm.weights_of(d, seed=8)
    _save(str(tmp_path / "m"), d, w)
    args = validate_server_args(ServerArgs(
        model=str(tmp_path / "m"), device="cpu", tokenizer="ids", page_size=16, num_gpu_pages=64, initial_gpu_page_buffer=2,
        extension_gpu_page_buffer=1, decision_frequency_pages=1, storage_path=str(tmp_path / "store"), startup_timeout=120.0,
        watchdog_timeout=0.0, max_model_len=256))
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((30, 5))]
    lines = [{"custom_id": f"r{i}", "method": "POST", "url": "/v1/completions",
              "body": {"model": "m", "prompt": p, "max_tokens": 6, "temperature": 0, "ignore_eos": True}}
             for i, p in enumerate(prompts)]
    with TestClient(create_app(args)) as c:
        data = "\n".join(map(json.dumps, lines)) + "\n"
        f = c.post("/v1/files", files={"file": ("in.jsonl", data.encode(), "application/jsonl")}, data={"purpose": "batch"}).json()
        b = c.post("/v1/batches", json={"input_file_id": f["id"], "endpoint": "/v1/completions"}).json()
        for _ in range(1200):
            b = c.get(f"/v1/batches/{b['id']}").json()
            if b["status"] in ("completed", "failed"):
                break
            time.sleep(0.1)
        assert b["status"] == "completed" and b["request_counts"]["completed"] == 2, b
        out = {o["custom_id"]: o["response"]["body"]["choices"][0]["text"] for o in
               map(json.loads, c.get(f"/v1/files/{b['output_file_id']}/content").text.splitlines())}
    for i, p in enumerate(prompts):
        assert out[f"r{i}"].split() == [str(t) for t in _greedy(d, w, p, 6)]
