"""Nanurax on the CPU path: configuration, weights from a directory, engine steps in any cut, scheduler and CLI."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import nanurax_models as nm
import nanurax_oracle as oracle

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _save(path, d, weights):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(d, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))


# ---------------------------------------------------------------- mechanisms
def test_glu_forms_and_their_clamps():
    from batchgen_b200.ops import residual
    g = torch.Generator().manual_seed(0)
    z = 3 * torch.randn(9, 24, generator=g)
    eye = torch.eye(12)
    w, gate = torch.rand(9, generator=g), torch.randn(9, 1, generator=g)
    want = oracle.gelu_tanh(z[:, :12]) * z[:, 12:]
    assert torch.allclose(residual.glu(z, 12, "gelu_tanh"), want, atol=1e-5)
    # through identity weights the expert's body is the activation alone
    want = torch.stack([oracle.clamped_expert(torch.cat([w[i] * z[i]]), torch.cat([eye, 0 * eye], 1),
                                              torch.cat([0 * eye, eye], 1), eye, 0.8) for i in range(9)])
    got = residual.glu(z, 12, "swiglu_oai", 0.8, row_scale=w, gate=gate)
    assert torch.allclose(got, want * torch.sigmoid(gate), atol=1e-5)


def test_sink_softmax_and_chunk_edges():
    seen = oracle.visible_chunk(7, 3)
    assert seen[3].tolist() == [False, False, False, True, False, False, False]
    assert seen[5].tolist() == [False] * 3 + [True] * 3 + [False]
    p = oracle.sink_softmax(torch.zeros(7, 7), seen)
    assert torch.allclose(p.sum(-1), torch.tensor([1 / 2, 2 / 3, 3 / 4, 1 / 2, 2 / 3, 3 / 4, 1 / 2]))


def test_router_keeps_plain_scores():
    from batchgen_b200.ops import moe
    g = torch.Generator().manual_seed(3)
    h, r = torch.randn(6, 10, generator=g), torch.randn(5, 10, generator=g)
    idx, val = oracle.route(h, r, 3)
    i2, w2 = moe.router_topk(h @ r.T, None, 3, norm_topk_prob=False, scoring="sigmoid")
    assert torch.equal(idx.sort(-1)[0], i2.long().sort(-1)[0])
    assert torch.allclose(val.sort(-1)[0], w2.sort(-1)[0], atol=1e-6)


# ---------------------------------------------------------------- whole model, any cut
@pytest.mark.parametrize("name", sorted(nm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name):
    d = nm.CONFIGS[name]
    w = nm.weights_of(d, seed=1)
    toks = nm.prompt(d, 150)
    trace = []
    want = oracle.forward(d, w, toks, torch.float64, trace)
    model = nm.build(d, w)
    layers = {}
    model.layer_hook = lambda l, x: layers.__setitem__(l, x.clone())
    eng = nm.engine(model)
    s = eng.open_sequence()
    assert nm.error(eng.extend([(s, toks, range(150))]), want) < 2e-5
    for l, x in enumerate(trace):
        assert torch.allclose(layers[l].double(), x, atol=2e-4 * float(x.abs().max())), l
    model.layer_hook = None
    eng.close_sequence(s)
    for sizes in ([2], [1], [63, 1, 2, 5], [100, 1]):
        s = eng.open_sequence()
        assert nm.error(nm.run_pieces(eng, s, toks, sizes), want) < 2e-5, sizes
        eng.close_sequence(s)
    assert eng.kv.alloc.num_used == 0 and (eng.kv.state is None or eng.kv.state.num_free == 4)


def test_unequal_batches_equal_each_request_alone_and_places_are_used_again():
    d = nm.CONFIGS["odd"]
    w = nm.weights_of(d, seed=2)
    model = nm.build(d, w)
    eng = nm.engine(model, tokens=64 * 7)
    prompts = [nm.prompt(d, n, i) for i, n in enumerate((130, 1, 41, 77, 3, 64))]
    want = [oracle.forward(d, w, p, torch.float64) for p in prompts]
    live, at, got = {}, [0] * 6, [[] for _ in prompts]
    order, rng = list(range(6)), torch.Generator().manual_seed(5)
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
        assert nm.error(torch.cat(g), x) < 2e-5
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


def _greedy(d, w, toks, n):
    toks = list(toks)
    for _ in range(n):
        toks.append(int(oracle.forward(d, w, toks, torch.float64)[-1].argmax()))
    return toks[-n:]


def test_greedy_generation_through_the_scheduler_with_chunks_holds_and_evictions():
    from batchgen_b200.runtime.sequence import SamplingParams
    d = nm.CONFIGS["odd"]
    w = nm.weights_of(d, seed=3)
    model = nm.build(d, w)
    prompts = [nm.prompt(d, n, i) for i, n in enumerate((50, 9, 33, 21))]
    want = [_greedy(d, w, p, 30) for p in prompts]
    params = SamplingParams(max_new_tokens=30, ignore_eos=True)
    assert nm.engine(model).generate(prompts, params) == want
    # pieces of at most 16 prompt tokens, few state slots and pages of 8 tokens: rows wait, are evicted and recomputed
    tight = nm.engine(model, tokens=8 * 16, slots=3, page=8, max_prefill_tokens=16, initial_gpu_page_buffer=1,
                      extension_gpu_page_buffer=1, decision_frequency_pages=1)
    assert tight.generate(prompts, params) == want
    assert tight.stats.evictions > 0 and tight.stats.prefill_chunks > 0
    # a host tier: parked rows keep their state
    from batchgen_b200.config import EngineConfig
    from batchgen_b200.runtime.engine import Engine
    ecfg = EngineConfig(page_size=8, max_decode_batch=4, max_state_slots=3, initial_gpu_page_buffer=1,
                        extension_gpu_page_buffer=1, decision_frequency_pages=1, enable_cuda_graph=False)
    parked = Engine(model, ecfg, num_gpu_pages=16, num_host_pages=60)
    assert parked.generate(prompts, params) == want
    assert parked.stats.holds > 0 and parked.host_state.offloads > 0 and parked.host_state.loads > 0


# ---------------------------------------------------------------- registry, directories, command line
def test_config_directory_registry_and_validation(tmp_path):
    from batchgen_b200.config import LayerSpec, ModelConfig, get_model_config, list_models, nanurax_config
    from batchgen_b200.models import build_model
    d = nm.CONFIGS["twice"]
    w = nm.weights_of(d, seed=4, rank=9)
    _save(str(tmp_path / "m"), d, w)
    cfg = get_model_config(str(tmp_path / "m"))
    assert cfg.family == "nanurax" and cfg.layer_specs[1].mixer.decay_rank == 9 and not cfg.is_mla
    assert cfg.layer_specs[0].mlp.kind == "none" and cfg.layer_specs[1].mlp.top == 4
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg
    assert isinstance(cfg.layer_specs[2], LayerSpec) and {"tiny-nanurax", "nanurax-bench"} <= set(list_models())
    toks = nm.prompt(d, 40)
    eng = nm.engine(build_model(cfg))
    assert nm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), oracle.forward(d, w, toks)) < 2e-5
    # the names the framework writes are the ones it reads; a converted copy of the directory serves as well
    from batchgen_b200.ckpt.converter import convert_dir
    from batchgen_b200.models.weights import checkpoint_tensor_specs
    assert {n: s for n, s, _, _ in checkpoint_tensor_specs(cfg)} == {k: tuple(t.shape) for k, t in w.items()}
    convert_dir(str(tmp_path / "m"), str(tmp_path / "c"))
    conv = get_model_config(str(tmp_path / "c"))
    assert conv.layer_specs == cfg.layer_specs
    eng = nm.engine(build_model(conv))
    assert nm.error(eng.extend([(eng.open_sequence(), toks, range(40))]), oracle.forward(d, w, toks)) < 2e-5
    bad = json.loads(json.dumps(d))
    bad["layers"][0]["type"] = "something_else"
    with pytest.raises(ValueError, match="something_else"):
        nanurax_config(bad)
    del w["l2.mix.talk"]
    _save(str(tmp_path / "short"), d, w)
    with pytest.raises(KeyError, match="l2.mix.talk"):
        build_model(get_model_config(str(tmp_path / "short")))
    (tmp_path / "other").mkdir()
    (tmp_path / "other" / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    with pytest.raises(KeyError, match="Unknown"):
        get_model_config(str(tmp_path / "other"))


def test_trace_replay_command(tmp_path):
    d = nm.CONFIGS["odd"]
    w = nm.weights_of(d, seed=6)
    _save(str(tmp_path / "m"), d, w)
    a, b = nm.prompt(d, 70, 1), nm.prompt(d, 30, 2)
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
    assert sorted(os.listdir(out)) == ["1.f32", "2.f32"]
    la, lb = oracle.forward(d, w, a), oracle.forward(d, w, b)
    got = torch.from_numpy(np.fromfile(out / "1.f32", "<f4").reshape(3, -1).copy())
    assert nm.error(got, torch.stack([la[50], la[68], lb[29]])) < 2e-5
    got = torch.from_numpy(np.fromfile(out / "2.f32", "<f4").reshape(1, -1).copy())
    assert nm.error(got, la[69:70]) < 2e-5


def test_steps_that_do_not_fit_are_refused():
    from batchgen_b200.runtime.kv_cache import OutOfPages
    d = nm.CONFIGS["odd"]
    eng = nm.engine(nm.build(d, nm.weights_of(d)), tokens=64)
    with pytest.raises(OutOfPages):
        eng.extend([(eng.open_sequence(), nm.prompt(d, 65), [])])
    with pytest.raises(ValueError, match="place"):
        eng.extend([(eng.open_sequence(), [1, 2], [2])])


def test_planner_and_preflight_know_the_design():
    from batchgen_b200.config import EngineConfig, get_model_config
    from batchgen_b200.runtime import planner
    from batchgen_b200.runtime.kv_cache import host_page_bytes
    cfg = get_model_config("nanurax-bench")
    assert cfg.kv_cache_dim == 8 * 256 and host_page_bytes(cfg, 64) == 64 * 8 * 256 * 2
    ecfg = EngineConfig(max_decode_batch=64, max_prefill_tokens=8192)
    assert planner.state_pool_bytes(cfg, ecfg) == 64 * 3 * 32 * 128 * 128 * 4
    plan = planner.plan_deployment(cfg, ecfg, planner.MACHINES["b200"])
    assert plan.fits and plan.expert_bytes == 3 * 64 * 3 * 2304 * 1024 * 2
    assert planner.layered_workspace_bytes(cfg) > 4 * 5 * 4096


def test_server_serves_a_model_directory(tmp_path):
    import time

    from fastapi.testclient import TestClient

    from batchgen_b200.server.http_server import create_app
    from batchgen_b200.server.preflight import PreflightError, model_contract, run_all_preflights
    from batchgen_b200.server.server_args import ServerArgs, ServerArgsError, validate_server_args
    d = nm.config(300, 48, [nm.delta(2, 16, nm.dense(40)), nm.attention(4, 2, 8, 8, 24, nm.moe(24, 3, 1, 1.0, 32))])
    w = nm.weights_of(d, seed=8)
    _save(str(tmp_path / "m"), d, w)
    args = validate_server_args(ServerArgs(
        model=str(tmp_path / "m"), device="cpu", tokenizer="ids", page_size=16, num_gpu_pages=64, initial_gpu_page_buffer=2,
        extension_gpu_page_buffer=1, decision_frequency_pages=1, storage_path=str(tmp_path / "store"), startup_timeout=120.0,
        watchdog_timeout=0.0, max_model_len=256))
    assert run_all_preflights(args)
    prompts = [nm.prompt(d, n, i) for i, n in enumerate((30, 5))]
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
    with pytest.raises(ServerArgsError):
        validate_server_args(ServerArgs(model=str(tmp_path / "nothing")))
    from batchgen_b200.config import get_model_config
    with pytest.raises(PreflightError, match="one GPU"):
        model_contract(get_model_config(str(tmp_path / "m")), 2, True)
