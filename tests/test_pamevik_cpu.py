"""Pamevik on the CPU path: configuration, weights from a directory, engine steps in any cut, scheduler and CLI."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import pamevik_models as pm
import pamevik_oracle as oracle

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _save(path, d, weights):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(d, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))


def _gen(seed):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------- the plain implementation itself
def test_plain_convolution_sees_the_last_taps_only():
    x = torch.zeros(6, 2)
    x[1] = torch.tensor([1.0, 2.0])
    w = torch.tensor([[1.0, 10.0, 100.0], [2.0, 20.0, 200.0]])
    y = oracle.causal_conv(x, w)
    assert y[:, 0].tolist() == [0, 100, 10, 1, 0, 0] and y[:, 1].tolist() == [0, 400, 40, 4, 0, 0]


def test_plain_rotation_pairs_halves_and_keeps_the_rest():
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 7.0
    y = oracle.rotate(x, 100.0, 4)
    for p in range(3):
        assert torch.allclose(y[p, 0], torch.tensor([np.cos(p), 0, np.sin(p), 0, 0, 7.0], dtype=torch.float64))


def test_plain_cells_on_cases_with_known_answers():
    one = torch.ones(1, 1, 1, dtype=torch.float64)
    # retention: geometric sum of equal writes
    o, _ = oracle.retention(one.repeat(3, 1, 1), one.repeat(3, 1, 1), one.repeat(3, 1, 1), torch.tensor([0.5], dtype=torch.float64))
    assert torch.allclose(o.flatten(), torch.tensor([1.0, 1.5, 1.75], dtype=torch.float64))
    # delta rule with full strength and no decay stores the last value of a key
    v = torch.tensor([3.0, -2.0], dtype=torch.float64).view(2, 1, 1)
    o, S = oracle.gated_delta(one.repeat(2, 1, 1), one.repeat(2, 1, 1), v, one.repeat(2, 1, 1), torch.ones(2, 1, dtype=torch.float64))
    assert torch.allclose(o.flatten(), v.flatten()) and float(S) == -2.0
    # mLSTM: with tiny input gates the denominator is exp(-m), with large ones the normaliser
    for i, want in ((-4.0, np.exp(-4.0) * 3.0), (2.0, 3.0)):
        g = torch.full((1, 1), i, dtype=torch.float64)
        o, (_, n, m) = oracle.mlstm(one, one, 3.0 * one, g, torch.zeros(1, 1, dtype=torch.float64))
        assert abs(float(o) - want) < 1e-5 and float(m) == max(i, 0.0)


# ---------------------------------------------------------------- mechanisms of the CPU path
def test_convolution_and_rotary_table_follow_the_plain_forms():
    from batchgen_b200.ops.conv import Rotary, causal_conv, rotate_ref
    for taps in (1, 2, 5):
        x, w = torch.randn(23, 12, generator=_gen(taps)), torch.randn(12, taps, generator=_gen(9))
        want = oracle.causal_conv(x, w)
        hist = torch.full((3, (taps - 1) * 12), 7.0)                         # what an earlier sequence left
        out, at = torch.empty(23, 16), 0
        for n in (1, 2, 1, 9, 3, 7):
            causal_conv(x[at:at + n], w.t().contiguous(), hist, torch.tensor([1]), out[at:at + n], "silu",
                        cu_host=[0, n], has_initial=[int(at > 0)])
            at += n
        assert torch.allclose(out[:, :12], torch.nn.functional.silu(want), atol=1e-5) and float(out[:, 12:].abs().sum()) == 0
    x = torch.randn(40, 3, 10, dtype=torch.float64, generator=_gen(1))
    r = Rotary.make(6, 70.0, "cpu")
    got = rotate_ref(x, r.table(torch.arange(40) + 1))
    assert torch.allclose(got, oracle.rotate(x, 70.0, 6), atol=1e-5)


# ---------------------------------------------------------------- whole model, any cut
@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name):
    d = pm.CONFIGS[name]
    w = pm.weights_of(d, seed=1)
    toks = pm.prompt(d, 150)
    trace = []
    want = oracle.forward(d, w, toks, torch.float64, trace)
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


def test_every_weight_takes_part():
    """A tensor that is read but not used would not show in a comparison with itself: changing any one of them has to change
    the logits, and by the same amount as in the plain implementation."""
    d = pm.CONFIGS["odd"]
    base = pm.weights_of(d, seed=4)
    toks = pm.prompt(d, 24)
    for name in sorted(base):
        w = dict(base)
        w[name] = base[name] + 0.3 * base[name].std() * torch.randn(base[name].shape, generator=_gen(5))
        want = oracle.forward(d, w, toks, torch.float64)
        assert pm.error(oracle.forward(d, base, toks, torch.float64), want) > 2e-3, name
        eng = pm.engine(pm.build(d, w))
        assert pm.error(eng.extend([(eng.open_sequence(), toks, range(24))]), want) < 1e-4, name


def test_unequal_batches_equal_each_request_alone_and_places_are_used_again():
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=2)
    eng = pm.engine(pm.build(d, w), tokens=64 * 7)
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((130, 1, 41, 77, 3, 64))]
    want = [oracle.forward(d, w, p, torch.float64) for p in prompts]
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
        toks.append(int(oracle.forward(d, w, toks, torch.float64)[-1].argmax()))
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
    # a host tier: parked rows keep their state, the convolutions' inputs and the running maximum with it
    ecfg = EngineConfig(page_size=8, max_decode_batch=4, max_state_slots=3, initial_gpu_page_buffer=1,
                        extension_gpu_page_buffer=1, decision_frequency_pages=1, enable_cuda_graph=False)
    parked = Engine(model, ecfg, num_gpu_pages=14, num_host_pages=60)
    assert parked.generate(prompts, params) == want
    assert parked.stats.holds > 0 and parked.host_state.offloads > 0 and parked.host_state.loads > 0


# ---------------------------------------------------------------- registry, directories, command line
def test_config_directory_registry_and_validation(tmp_path):
    from batchgen_b200.ckpt.converter import convert_dir
    from batchgen_b200.config import ModelConfig, get_model_config, list_models, pamevik_config
    from batchgen_b200.models import build_model
    from batchgen_b200.models.weights import checkpoint_tensor_specs
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=4, ranks=(13, 5))
    _save(str(tmp_path / "m"), d, w)
    cfg = get_model_config(str(tmp_path / "m"))
    assert cfg.family == "pamevik" and cfg.sandwich and cfg.layer_norm and cfg.canon_taps == 3 and not cfg.is_mla
    assert (cfg.layer_specs[0].mixer.decay_rank, cfg.layer_specs[3].mixer.gate_rank) == (13, 5)
    assert cfg.layer_specs[1].second.decay == (0.8, 0.95, 0.999) and cfg.layer_specs[2].mlp.kind == "none"
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg and {"tiny-pamevik", "pamevik-bench"} <= set(list_models())
    toks = pm.prompt(d, 40)
    want = oracle.forward(d, w, toks)
    eng = pm.engine(build_model(cfg))
    assert pm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), want) < 5e-5
    # the names the framework writes are the ones it reads; a converted copy of the directory serves as well
    assert {n: s for n, s, _, _ in checkpoint_tensor_specs(cfg)} == {k: tuple(t.shape) for k, t in w.items()}
    convert_dir(str(tmp_path / "m"), str(tmp_path / "c"))
    conv = get_model_config(str(tmp_path / "c"))
    assert conv.layer_specs == cfg.layer_specs
    eng = pm.engine(build_model(conv))
    assert pm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), want) < 5e-5
    for edit, match in ((lambda x: x["layers"][0].update(type="other_kind"), "other_kind"),
                        (lambda x: x["layers"][0]["mixer"].update(kv_heads=4), "divide"),
                        (lambda x: x["layers"][1]["mixer"]["left"]["rot"].update(dims=16), "rotary"),
                        (lambda x: x["layers"][1]["mixer"]["right"].update(decay=[0.5]), "decays"),
                        (lambda x: x["layers"][0]["mlp"].update(kind="sparse"), "sparse")):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(ValueError, match=match):
            pamevik_config(bad)
    del w["l2.mix.f.b"]
    _save(str(tmp_path / "short"), d, w)
    with pytest.raises(KeyError, match="l2.mix.f.b"):
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
    from batchgen_b200.config import EngineConfig, get_model_config
    from batchgen_b200.runtime import planner
    from batchgen_b200.runtime.kv_cache import PagedKVCache, host_page_bytes
    from batchgen_b200.server.preflight import PreflightError, model_contract
    cfg = get_model_config("pamevik-bench")
    assert cfg.kv_cache_dim == 8 * 256 and host_page_bytes(cfg, 64) == 64 * 8 * 256 * 2
    S, canon, conv = 32 * 128 * 128, 3 * 2304, 3 * 3 * 32 * 128
    per = 4 * (4 * S + 8 * canon + 2 * conv + 32 * 128 + 32)
    ecfg = EngineConfig(max_decode_batch=64, max_prefill_tokens=8192)
    assert planner.state_pool_bytes(cfg, ecfg) == 64 * per
    assert planner.plan_deployment(cfg, ecfg, planner.MACHINES["b200"]).fits
    tiny = get_model_config("tiny-pamevik")
    kv = PagedKVCache(tiny, 2, 16, "cpu", torch.float32, state_slots=3)
    assert kv.state.row_floats >= tiny.layered_state_floats_per_seq() and kv.state.layer(1, "S.1").shape == (4, 2 * 16 * 40)
    assert model_contract(tiny, 1, True)
    with pytest.raises(PreflightError, match="one GPU"):
        model_contract(tiny, 2, True)
    wide = pm.config(64, 64, [pm.mlstm(1, 520, 8, 1.0)])
    from batchgen_b200.config import pamevik_config
    with pytest.raises(PreflightError, match="512"):
        model_contract(pamevik_config(wide), 1, True)


def test_server_serves_a_model_directory(tmp_path):
    import time

    from fastapi.testclient import TestClient

    from batchgen_b200.server.http_server import create_app
    from batchgen_b200.server.server_args import ServerArgs, validate_server_args
    d = pm.config(300, 48, [pm.mlstm(2, 16, 8, 5.0, pm.dense(40)),
                            pm.parallel((4, 2, 8, 8, 8, 60.0), ([0.9], 8, 16, 4, 60.0))], taps=2)
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
