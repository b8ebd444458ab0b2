"""Bolisun on the CPU path: configuration, weights from a directory, engine steps in any cut, scheduler and CLI."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import bolisun_models as bm
import bolisun_oracle as oracle

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
def test_plain_rotation_pairs_neighbours_and_keeps_the_rest():
    x = torch.zeros(3, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 4] = 1.0, 2.0, 7.0
    y = oracle.rotate(x, 100.0, 4)
    for p in range(3):
        want = [np.cos(p), np.sin(p), -2 * np.sin(p * 0.1), 2 * np.cos(p * 0.1), 7.0, 0]
        assert torch.allclose(y[p, 0], torch.tensor(want, dtype=F64))


def test_plain_frequencies_of_scaled_positions():
    # base e^2, 8 dimensions: pair i turns once in 2 pi e^(i / 2) positions
    base, original = math.exp(2.0), 2 * math.pi * math.exp(1.0)
    sc = bm.scaling(4.0, original, math.exp(0.9), math.exp(-0.4))          # pairs 0.2 and 2.8: the ramp runs from 0 to 3
    f, g = oracle.frequencies(8, base), oracle.frequencies(8, base, sc)
    for i, ramp in enumerate((0.0, 1 / 3, 2 / 3, 1.0)):
        assert abs(g[i] - f[i] * (1 - 0.75 * ramp)) < 1e-12
    same = oracle.frequencies(8, base, bm.scaling(4.0, original, 1.0, 1.0))    # an empty ramp: a step after the pair
    assert [round(a / b, 9) for a, b in zip(same, f)] == [1, 1, 1, 0.25]
    assert torch.allclose(oracle.rotate(torch.ones(1, 1, 8, dtype=F64), base, 8, sc), torch.tensor(0.1 * math.log(4.0) + 1, dtype=F64))


def test_plain_window_keeps_the_first_tokens():
    rows = {i: [j for j in range(8) if oracle.visible(8, 3, 2)[i, j]] for i in range(8)}
    assert rows[0] == [0] and rows[3] == [0, 1, 2, 3] and rows[4] == [0, 1, 2, 3, 4] and rows[7] == [0, 1, 5, 6, 7]


def test_plain_router_on_cases_with_known_answers():
    z = torch.log(torch.tensor([[0.05, 0.3, 0.25, 0.1, 0.2, 0.1]], dtype=F64))
    corr = torch.tensor([-1.0, -1.0, -0.2, -0.3, -2.0, -2.0], dtype=F64)
    # choice scores: -0.95 -0.7 | 0.05 -0.2 | -1.8 -1.9; the second and the first group stay
    idx, w = oracle.route(z, corr, {"top": 3, "scale": 2.0, "groups": {"count": 3, "keep": 2}})
    assert idx[0].tolist() == [2, 3, 1] and torch.allclose(w[0], torch.tensor([0.25, 0.1, 0.3], dtype=F64) * 2 / 0.65)
    idx, w = oracle.route(z, corr, {"top": 2, "scale": 0.5, "groups": {"count": 3, "keep": 1}})
    assert idx[0].tolist() == [2, 3]
    idx, w = oracle.route(z, 0 * corr, {"top": 1, "scale": 3.0})
    assert idx[0].tolist() == [1] and abs(float(w) - 3.0) < 1e-12


def test_plain_hyper_step_mixes_the_old_streams():
    w = {"in": torch.tensor([1.0, 2.0]), "mix": torch.tensor([[1.0, 10.0], [100.0, 1000.0]]), "out": torch.tensor([1.0, -1.0])}
    xs = torch.tensor([[[3.0]], [[0.5]]])
    got = oracle.hyper_step(xs, w, "", torch.ones(1), lambda h: 7 * h, 0.0)                 # reads 3 + 1, normed to 1
    assert got.flatten().tolist() == [3.0 + 50.0 + 7.0, 30.0 + 500.0 - 7.0]


def test_plain_retention_on_a_case_with_a_known_answer():
    one = torch.ones(3, 1, 1, dtype=F64)
    o, _ = oracle.retention(one, one, one, torch.tensor([0.5], dtype=F64))
    assert torch.allclose(o.flatten(), torch.tensor([1.0, 1.5, 1.75], dtype=F64))


# ---------------------------------------------------------------- mechanisms of the CPU path
@pytest.mark.parametrize("sc", [None, bm.scaling(5.0, 120, 9.0, 0.5), bm.scaling(3.0, 30, 2.0, 2.0), bm.scaling(1.0, 9, 40.0, 8.0)])
def test_rotary_tables_follow_the_plain_form(sc):
    from batchgen_b200.ops.conv import Rotary, rotate_ref
    x = torch.randn(40, 3, 22, dtype=F64, generator=_gen(1))
    for dims, base in ((2, 10.0), (14, 70.0), (22, 1e6)):
        yarn = tuple(sc[k] for k in ("factor", "original", "fast", "slow")) if sc else ()
        r = Rotary.make(dims, base, "cpu", True, yarn)
        assert torch.allclose(rotate_ref(x, r.table(torch.arange(40) + 1), True), oracle.rotate(x, base, dims, sc), atol=2e-5)


def test_router_follows_the_plain_form():
    from batchgen_b200.ops import moe
    z, corr = torch.randn(40, 12, generator=_gen(2)), 0.3 * torch.randn(12, generator=_gen(3)) - 0.5
    for top, groups in ((3, (4, 2)), (1, (3, 3)), (4, (2, 1)), (5, None), (1, None), (1, (12, 1))):
        r = {"top": top, "scale": 1.3, "groups": {"count": groups[0], "keep": groups[1]} if groups else None}
        idx, w = oracle.route(z.double(), corr.double(), r)
        i2, w2 = moe.router_topk(z, corr, top, *(groups or (1, 1)), "always", 1.3, "softmax_all", None, "max")
        assert torch.equal(idx, i2.long()) and torch.allclose(w, w2.double(), atol=1e-6)


def test_streams_and_experts_rows_join_as_in_the_plain_form():
    from batchgen_b200.ops import residual
    T, S, D, g = 5, 3, 10, _gen(4)
    x = torch.zeros(T, S, 12)
    x[..., :D] = torch.randn(T, S, D, generator=g)
    hc = residual.Hyper(torch.randn(S, generator=g), torch.randn(S, S, generator=g), torch.randn(S, generator=g))
    add, bias, routed = torch.randn(T, 12, generator=g), torch.randn(12, generator=g), torch.randn(9, 12, generator=g)
    pos = torch.randint(-1, 9, (T, 4), generator=g).to(torch.int32)
    rw, w, nxt = torch.rand(T, 4, generator=g), torch.randn(12, generator=g), torch.randn(S, generator=g)
    y = add + bias + sum(torch.where(pos[:, k:k + 1] >= 0, rw[:, k:k + 1] * routed[pos[:, k].clamp_min(0).long()], torch.zeros(1))
                         for k in range(4))
    want = torch.stack([sum(hc.mix[s, t] * x[:, s] for s in range(S)) + hc.share[t] * y for t in range(S)], 1)[..., :D]
    h = residual.hyper_norm(x, w, 1e-5, D, 64, torch.float32, read=nxt, hc=hc, add=add, bias=bias, routed=routed, pos=pos, route_w=rw)
    assert torch.allclose(x[..., :D], want, atol=1e-5)
    assert torch.allclose(h[:, :D], oracle.rms(sum(nxt[s] * want[:, s] for s in range(S)), 1e-5) * w[:D], atol=1e-5)
    assert float(h[:, D:].abs().sum()) == 0


# ---------------------------------------------------------------- whole model, any cut
@pytest.mark.parametrize("name", sorted(bm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name):
    d = bm.CONFIGS[name]
    w = bm.weights_of(d, seed=1)
    toks = bm.prompt(d, 150)
    trace = []
    want = oracle.forward(d, w, toks, F64, trace)
    model = bm.build(d, w)
    layers = {}
    model.layer_hook = lambda l, x: layers.__setitem__(l, x.clone())
    eng = bm.engine(model)
    s = eng.open_sequence()
    assert bm.error(eng.extend([(s, toks, range(150))]), want) < 5e-5
    for l, x in enumerate(trace):
        assert torch.allclose(layers[l].double(), x, atol=2e-4 * float(x.abs().max())), l
    model.layer_hook = None
    eng.close_sequence(s)
    for sizes in ([2], [1], [63, 1, 2, 5], [100, 1]):
        s = eng.open_sequence()
        assert bm.error(bm.run_pieces(eng, s, toks, sizes), want) < 5e-5, sizes
        eng.close_sequence(s)
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("seed", range(6))
def test_random_designs(seed):
    d = bm.random_config(seed)
    w = bm.weights_of(d, seed)
    toks = bm.prompt(d, 90)
    want = oracle.forward(d, w, toks, F64)
    eng = bm.engine(bm.build(d, w))
    for sizes in ([90], [31, 2, 1]):
        assert bm.error(bm.run_pieces(eng, eng.open_sequence(), toks, sizes), want) < 1e-4


def test_every_weight_takes_part():
    """A tensor that is read but not used would not show in a comparison with itself: changing any one of them has to change
    the logits, and by the same amount as in the plain implementation."""
    d = bm.CONFIGS["odd"]
    base = bm.weights_of(d, seed=4)
    toks = bm.prompt(d, 45)
    plain = oracle.forward(d, base, toks, F64)
    names = [n for n in sorted(base) if ".e" not in n or n.split(".")[2] in ("e0", "e7", "e14")]
    for name in names:
        w = dict(base)
        w[name] = base[name] + (0.3 * base[name].std() + 0.02) * torch.randn(base[name].shape, generator=_gen(5))
        want = oracle.forward(d, w, toks, F64)
        # (adding the same to every score of a softmax changes nothing: of a key's bias only what rotates differently shows)
        assert bm.error(plain, want) > (1e-3 if name.endswith("k.b") else 2e-3), name
        eng = bm.engine(bm.build(d, w))
        assert bm.error(eng.extend([(eng.open_sequence(), toks, range(45))]), want) < 1e-4, name


def test_layers_that_share_weights_have_states_of_their_own():
    d = bm.CONFIGS["odd"]
    w = bm.weights_of(d, seed=7)
    model = bm.build(d, w)
    assert model.w.layers[0] is model.w.layers[2] and model.w.layers[4] is model.w.layers[2]
    eng = bm.engine(model)
    s = eng.open_sequence()
    eng.extend([(s, bm.prompt(d, 30), [29])])
    a, b = (eng.kv.state.layer(l, "S.1") for l in (0, 2))
    assert a.data_ptr() != b.data_ptr() and float((a - b).abs().max()) > 1e-3
    assert float((eng.kv.latent(0) - eng.kv.latent(4)).abs().max()) > 1e-3


def test_unequal_batches_equal_each_request_alone_and_places_are_used_again():
    d = bm.CONFIGS["odd"]
    w = bm.weights_of(d, seed=2)
    eng = bm.engine(bm.build(d, w), tokens=64 * 7)
    prompts = [bm.prompt(d, n, i) for i, n in enumerate((130, 1, 41, 77, 3, 64))]
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
        assert bm.error(torch.cat(g), x) < 5e-5
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
    d = bm.CONFIGS["odd"]
    w = bm.weights_of(d, seed=3)
    model = bm.build(d, w)
    prompts = [bm.prompt(d, n, i) for i, n in enumerate((50, 9, 33, 21))]
    want = [_greedy(d, w, p, 20) for p in prompts]
    params = SamplingParams(max_new_tokens=20, ignore_eos=True)
    assert bm.engine(model).generate(prompts, params) == want
    # pieces of at most 16 prompt tokens, few state slots and pages of 8 tokens: rows wait, are evicted and recomputed
    tight = bm.engine(model, tokens=8 * 14, slots=3, page=8, max_prefill_tokens=16, initial_gpu_page_buffer=1,
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
    from batchgen_b200.config import ModelConfig, bolisun_config, get_model_config, list_models
    from batchgen_b200.models import build_model
    from batchgen_b200.models.weights import checkpoint_tensor_specs
    d = bm.CONFIGS["odd"]
    w = bm.weights_of(d, seed=4)
    _save(str(tmp_path / "m"), d, w)
    cfg = get_model_config(str(tmp_path / "m"))
    assert cfg.family == "bolisun" and cfg.streams == 3 and cfg.tie_word_embeddings and not cfg.is_mla
    assert [s.weights_of for s in cfg.layer_specs] == [2, -1, -1, -1, 2]
    a, f = cfg.layer_specs[2].mixer, cfg.layer_specs[2].mlp
    assert (a.window, a.keep_first, a.yarn) == (37, 9, (5.0, 90.0, 6.0, 0.7)) and cfg.layer_specs[1].second.out_scale == -0.9
    assert (f.groups, f.keep_groups, f.router_scale, f.shared_ff) == (5, 2, 1.9, 60)
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg and {"tiny-bolisun", "bolisun-bench"} <= set(list_models())
    toks = bm.prompt(d, 40)
    want = oracle.forward(d, w, toks)
    eng = bm.engine(build_model(cfg))
    assert bm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), want) < 5e-5
    # the names the framework writes are the ones it reads; a converted copy of the directory serves as well
    assert {n: s for n, s, _, _ in checkpoint_tensor_specs(cfg)} == {k: tuple(t.shape) for k, t in w.items()}
    assert cfg.param_count() == sum(t.numel() for k, t in w.items() if ".hc" not in k and "correction" not in k
                                    and (".norm" not in k or "left" in k))
    convert_dir(str(tmp_path / "m"), str(tmp_path / "c"))
    conv = get_model_config(str(tmp_path / "c"))
    assert conv.layer_specs == cfg.layer_specs
    eng = bm.engine(build_model(conv))
    assert bm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), want) < 5e-5
    for edit, match in ((lambda x: x["layers"][1].update(type="other_kind"), "other_kind"),
                        (lambda x: x["layers"][1]["mixer"]["left"].update(kv_heads=4), "divide"),
                        (lambda x: x["layers"][1]["mixer"]["left"]["rot"].update(dims=16), "rotary"),
                        (lambda x: x["layers"][1]["mixer"]["left"]["mask"].update(size=0), "window"),
                        (lambda x: x["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5, 0.5]), "decays"),
                        (lambda x: x["layers"][2]["mlp"]["router"].update(top=7), "groups"),
                        (lambda x: x["layers"][4].update(mlp=None), "differs"),
                        (lambda x: x["layers"][2].update(weights_of=4), "weights of"),
                        (lambda x: x["layers"][1]["mlp"].update(kind="sparse"), "sparse")):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(ValueError, match=match):
            bolisun_config(bad)
    del w["l2.mlp.e3.up"]
    _save(str(tmp_path / "short"), d, w)
    with pytest.raises(KeyError, match="l2.mlp.e3.up"):
        build_model(get_model_config(str(tmp_path / "short")))


def test_trace_replay_command(tmp_path):
    d = bm.CONFIGS["odd"]
    w = bm.weights_of(d, seed=6)
    _save(str(tmp_path / "m"), d, w)
    a, b = bm.prompt(d, 70, 1), bm.prompt(d, 30, 2)
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
    assert bm.error(got, torch.stack([la[50], la[68], lb[29]])) < 5e-5
    got = torch.from_numpy(np.fromfile(out / "2.f32", "<f4").reshape(1, -1).copy())
    assert bm.error(got, la[69:70]) < 5e-5


def test_planner_and_preflight_know_the_design():
    from batchgen_b200.config import EngineConfig, bolisun_config, get_model_config
    from batchgen_b200.runtime import planner
    from batchgen_b200.runtime.kv_cache import PagedKVCache, host_page_bytes
    from batchgen_b200.server.preflight import PreflightError, model_contract
    cfg = get_model_config("bolisun-bench")
    assert cfg.kv_cache_dim == 4 * 8 * 256 and host_page_bytes(cfg, 64) == 64 * 4 * 8 * 256 * 2
    ecfg = EngineConfig(max_decode_batch=64, max_prefill_tokens=8192)
    assert planner.state_pool_bytes(cfg, ecfg) == 64 * 4 * 4 * 32 * 128 * 128
    dense, experts = planner.weight_bytes_per_rank(cfg, 1, 1)
    assert experts == 2 * 64 * 3 * 2304 * 1024 * 2               # the fourth layer has none of its own
    assert planner.plan_deployment(cfg, ecfg, planner.MACHINES["b200"]).fits
    tiny = get_model_config("tiny-bolisun")
    kv = PagedKVCache(tiny, 2, 16, "cpu", torch.float32, state_slots=3)
    assert kv.state.row_floats >= tiny.layered_state_floats_per_seq() and kv.state.layer(2, "S.1").shape == (4, 3 * 16 * 40)
    assert model_contract(tiny, 1, True)
    with pytest.raises(PreflightError, match="one GPU"):
        model_contract(tiny, 2, True)
    args = dict(mask=(4, 1), rot=(8, 10.0, None), right=((0.5,), 8, 8))
    for x, match in ((bm.config(64, 64, 17, [bm.layer((1, 1, 8, 8), **args)]), "streams"),
                     (bm.config(64, 64, 2, [bm.layer((1, 1, 1032, 8), **args)]), "1024"),
                     (bm.config(64, 64, 2, [bm.layer((1, 1, 8, 8), mlp=bm.moe(8, 80, 2, groups=(40, 2)), **args)]), "groups")):
        with pytest.raises(PreflightError, match=match):
            model_contract(bolisun_config(x), 1, True)


def test_server_serves_a_model_directory(tmp_path):
    import time

    from fastapi.testclient import TestClient

    from batchgen_b200.server.http_server import create_app
    from batchgen_b200.server.server_args import ServerArgs, validate_server_args
    d = bm.config(300, 48, 2, [bm.layer((4, 2, 8, 8), (12, 2), (8, 60.0, None), ((0.9,), 8, 16), bm.dense(40, 1.0)),
                               bm.layer((2, 1, 16, 8), (9, 0), (8, 60.0, None), ((0.7, 0.99), 8, 16), bm.moe(24, 6, 2, groups=(3, 2)))])
    w = bm.weights_of(d, seed=8)
    _save(str(tmp_path / "m"), d, w)
    args = validate_server_args(ServerArgs(
        model=str(tmp_path / "m"), device="cpu", tokenizer="ids", page_size=16, num_gpu_pages=64, initial_gpu_page_buffer=2,
        extension_gpu_page_buffer=1, decision_frequency_pages=1, storage_path=str(tmp_path / "store"), startup_timeout=120.0,
        watchdog_timeout=0.0, max_model_len=256))
    prompts = [bm.prompt(d, n, i) for i, n in enumerate((30, 5))]
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
