"""Nanurax kernels and models on the GPU against the plain implementation, in bf16 and in true fp32."""
import math

import pytest
import torch

import nanurax_models as nm
import nanurax_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-30))


def _gen(seed):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------- row operators
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("T,D", [(5, 100), (3, 2307), (70, 256), (1, 5)])
def test_residual_norm_with_every_addend(T, D, dtype):
    from batchgen_b200.ops import residual
    g = _gen(T + D)
    D4, cols, K = -(-D // 4) * 4, -(-D // 64) * 64, 3
    x, add = torch.randn(T, D4, generator=g), torch.randn(T, D4, generator=g)
    routed, pos = torch.randn(9, D4, generator=g), torch.randint(-1, 9, (T, K), generator=g).to(torch.int32)
    w = 1 + 0.2 * torch.randn(D, generator=g)
    xd = x.to(DEV)
    y = residual.residual_norm(xd, w.to(DEV), 1e-5, D, cols, dtype, add=add.to(DEV), routed=routed.to(DEV), pos=pos.to(DEV))
    want = x[:, :D] + add[:, :D]
    for t in range(T):
        for k in range(K):
            if pos[t, k] >= 0:
                want[t] += routed[pos[t, k], :D]
    assert torch.allclose(xd[:, :D].cpu(), want, atol=1e-5)
    assert _rel(y[:, :D], oracle.rms_norm(want, w, 1e-5)) < (5e-3 if dtype == torch.bfloat16 else 1e-6)
    assert float(y[:, D:].abs().sum()) == 0
    emb = torch.randn(11, D, generator=g).to(dtype)
    ids = torch.randint(0, 11, (T,), generator=g).to(torch.int32)
    y = residual.residual_norm(xd, w.to(DEV), 1e-5, D, cols, dtype, ids=ids.to(DEV), embed=emb.to(DEV), embed_scale=3.5)
    assert torch.allclose(xd[:, :D].cpu(), emb[ids.long()].float() * 3.5, atol=1e-6)
    rows = torch.tensor([T - 1, 0, T - 1])
    before = xd.clone()
    y = residual.residual_norm(xd, w.to(DEV), 1e-5, D, cols, dtype, add=add.to(DEV), rows=rows.to(DEV), keep=False)
    assert torch.equal(before, xd)
    assert _rel(y[:, :D], oracle.rms_norm((before.cpu() + add)[rows, :D], w, 1e-5)) < 5e-3


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_glu_cast_and_gather(dtype):
    from batchgen_b200.ops import residual
    g = _gen(1)
    T, F, Fo = 37, 44, 64
    z = 2.5 * torch.randn(T, 3 * F, generator=g)
    scale, gate = torch.rand(T, generator=g), torch.randn(T, 1, generator=g)
    tol = 5e-3 if dtype == torch.bfloat16 else 2e-6
    zd = z.to(DEV)
    out = torch.empty(T, Fo, dtype=dtype, device=DEV)
    residual.glu(zd[:, F:], F, "gelu_tanh", out=out)
    assert _rel(out[:, :F], oracle.gelu_tanh(z[:, F:2 * F]) * z[:, 2 * F:]) < tol and float(out[:, F:].abs().sum()) == 0
    residual.glu(zd[:, F:], F, "swiglu_oai", 0.9, row_scale=scale.to(DEV), gate=gate.to(DEV), out=out)
    s = scale.unsqueeze(-1)
    a, u = (s * z[:, F:2 * F]).clamp(max=0.9), (s * z[:, 2 * F:]).clamp(-0.9, 0.9)
    assert _rel(out[:, :F], a * torch.sigmoid(1.702 * a) * (u + 1) * torch.sigmoid(gate)) < tol
    c = residual.cast_act(zd[:, 3:20], 64, dtype, act="tanh")
    assert _rel(c[:, :17], torch.tanh(z[:, 3:20])) < tol and float(c[:, 17:].abs().sum()) == 0
    x = torch.randn(6, 64, generator=g).to(dtype)
    pos = torch.tensor([[4, 0], [1, -1], [2, 3], [5, 6], [-1, -1], [8, 7]], dtype=torch.int32)
    w = torch.rand(6, 2, generator=g)
    xs, ws = residual.moe_gather(x.to(DEV), pos.to(DEV), w.to(DEV), 12)
    for t in range(6):
        for k in range(2):
            if pos[t, k] >= 0:
                assert torch.equal(xs[pos[t, k]].cpu(), x[t]) and float(ws[pos[t, k]]) == float(w[t, k])


def test_f32_gemm_is_not_a_reduced_mode():
    from batchgen_b200.ops import gemm
    g = _gen(2)
    for M, N, K in ((1, 7, 5), (130, 97, 203), (64, 64, 64)):
        a, b = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g)
        assert _rel(gemm.rows_gemm(a.to(DEV), b.to(DEV)), a.double() @ b.double().T) < 1e-6
    counts = torch.tensor([5, 0, 70], dtype=torch.int32)
    off = torch.tensor([0, 8, 8, 80], dtype=torch.int32)
    x, w = torch.randn(80, 33, generator=g), torch.randn(3, 21, 33, generator=g)
    y = gemm.grouped_rows_gemm(x.to(DEV), w.to(DEV), off.to(DEV), counts.to(DEV), max_rows=70).cpu()
    for e in range(3):
        a, n = int(off[e]), int(counts[e])
        if n:
            assert _rel(y[a:a + n], x[a:a + n].double() @ w[e].double().T) < 1e-6


# ---------------------------------------------------------------- generalised delta rule
def _delta_case(T, H, d, seed):
    """Inputs of the op (padded heads, stacked columns with gaps) and the oracle's view of them."""
    from batchgen_b200.ops import delta
    g = _gen(seed)
    dp = -(-d // 8) * 8
    n = H * dp
    cols = [torch.randn(T, H, d, generator=g) for _ in range(5)]              # r, k, v, g, a
    low, w0, ab = torch.randn(T, H, d, generator=g), torch.randn(H, d, generator=g), torch.randn(H, d, generator=g)
    norm = 1 + 0.2 * torch.randn(H, d, generator=g)
    pad = lambda t: torch.nn.functional.pad(t, (0, dp - d)).reshape(*t.shape[:-2], n)      # noqa: E731
    z = torch.zeros(T, 5 * (n + 8))
    offs = tuple(i * (n + 8) for i in range(5))
    for o, t in zip(offs, cols):
        z[:, o:o + n] = pad(t)
    p = delta.DeltaParams(*(pad(t).to(DEV) for t in (w0, ab, norm)), heads=H, dim=d, dim_p=dp, decay_scale=math.exp(-0.5),
                          eps=1e-5)
    r, k, v, gate, a = (t.double() for t in cols)
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(low.double() + w0))
    args = (r, k, v, decay, k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6), torch.sigmoid(a + ab))

    def finish(o):
        return oracle.rms(o, 1e-5) * norm * torch.sigmoid(gate[: o.shape[0]])
    return z, offs, pad(low), p, args, gate, norm, dp


@pytest.mark.parametrize("H,d", [(3, 8), (2, 20), (5, 48), (2, 64), (3, 90), (2, 128), (1, 160), (1, 256), (1, 392)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_rule_prompts_continuations_and_decoding(H, d, dtype):
    from batchgen_b200.ops import delta
    lens = [37, 1, 2, 150]
    T = sum(lens)
    z, offs, low, p, args, gate, norm, dp = _delta_case(T, H, d, H * 1000 + d)
    cu = [0]
    for x in lens:
        cu.append(cu[-1] + x)
    S0 = torch.randn(H, d, d, generator=_gen(9))
    n = H * dp
    state = torch.full((6, n * dp + 8), 7.0)                                  # slots hold what others left there
    view = state[:, 8:]
    view[3].view(H, dp, dp).zero_()[:, :d, :d] = S0                           # the second sequence goes on from a state
    sd = state.to(DEV)
    out = torch.full((T, n + 64), 5.0, dtype=dtype, device=DEV)
    slots = torch.tensor([4, 3, 0, 1], dtype=torch.int32, device=DEV)
    init = torch.tensor([0, 1, 0, 0], dtype=torch.int32, device=DEV)
    delta.delta_forward(z.to(DEV), offs, low.to(DEV), p, sd[:, 8:], slots, out[:, :n],
                        torch.tensor(cu, dtype=torch.int32, device=DEV), cu, init)
    tol = 1e-2 if dtype == torch.bfloat16 else 3e-5
    ends = {}
    for i, slot in enumerate((4, 3, 0, 1)):
        part = [t[cu[i]:cu[i + 1]] for t in args]
        o, S = oracle.general_delta(*part, S=S0.double() if i == 1 else None)
        ends[slot] = S
        want = oracle.rms(o, 1e-5) * norm * torch.sigmoid(gate[cu[i]:cu[i + 1]].double())
        got = out[cu[i]:cu[i + 1], :n].view(-1, H, dp)[..., :d]
        assert _rel(got, want) < tol, i
        assert _rel(sd[slot, 8:].view(H, dp, dp)[:, :d, :d], S) < 3e-5, i
    assert float((sd[2] - 7).abs().sum()) == 0 and float((sd[:, :8] - 7).abs().sum()) == 0 and float((out[:, n:] - 5).abs().sum()) == 0
    # decoding from those states, with a padding row and rows in another order of slots
    z2, _, low2, p2, args2, gate2, norm2, _ = _delta_case(4, H, d, H * 1000 + d + 1)
    p2.w0, p2.ab, p2.norm_w = p.w0, p.ab, p.norm_w
    order = [1, -1, 4, 0]
    out2 = torch.full((4, n), 5.0, dtype=dtype, device=DEV)
    delta.delta_forward(z2.to(DEV), offs, low2.to(DEV), p2, sd[:, 8:], torch.tensor(order, dtype=torch.int32, device=DEV), out2)
    w0, ab = (t.cpu().view(H, dp)[:, :d].double() for t in (p.w0, p.ab))
    a2 = z2[:, offs[4]:offs[4] + n].view(4, H, dp)[..., :d].double()
    dec = torch.exp(-math.exp(-0.5) * torch.sigmoid(low2.view(4, H, dp)[..., :d].double() + w0))
    for t, slot in enumerate(order):
        if slot < 0:
            assert float(out2[t].abs().sum()) == 0
            continue
        one = [x[t:t + 1] for x in args2]
        one[3], one[5] = dec[t:t + 1], torch.sigmoid(a2[t:t + 1] + ab)
        o, S = oracle.general_delta(*one, S=ends[slot])
        want = oracle.rms(o, 1e-5) * norm * torch.sigmoid(gate2[t:t + 1].double())
        assert _rel(out2[t:t + 1].view(1, H, dp)[..., :d], want) < tol, t
        assert _rel(sd[slot, 8:].view(H, dp, dp)[:, :d, :d], S) < 3e-5, t


def test_delta_decode_over_many_rows_and_steps():
    """More (sequence, head) items than SMs, slots in any order, several steps: the ring of state buffers turns over."""
    from batchgen_b200.ops import delta
    B, H, d = 150, 3, 32
    z, offs, low, p, args, gate, norm, dp = _delta_case(B, H, d, 77)
    perm = torch.randperm(B, generator=_gen(4))
    slots = perm.to(torch.int32).to(DEV)
    slots[5], slots[149] = -1, -1
    st = torch.zeros(B, H * d * d, device=DEV)
    S = torch.zeros(B, H, d, d, dtype=torch.float64)
    out = torch.empty(B, H * d, device=DEV)
    zd, ld = z.to(DEV), low.to(DEV)
    for step in range(7):
        delta.delta_forward(zd, offs, ld, p, st, slots, out)
    r, k, v, w, u, a = args
    for _ in range(7):
        y = torch.einsum("bhk,bhkv->bhv", u, S)
        S = w.unsqueeze(-1) * S - (a * u).unsqueeze(-1) * y.unsqueeze(2) + k.unsqueeze(-1) * v.unsqueeze(2)
    o = torch.einsum("bhkv,bhk->bhv", S, r)
    live = [b for b in range(B) if b not in (5, 149)]
    assert _rel(st.view(B, H, d, d)[perm[live].to(DEV)], S[live]) < 1e-5
    want = oracle.rms(o, 1e-5) * norm * torch.sigmoid(gate)
    assert _rel(out.view(B, H, d)[live], want[live]) < 1e-5 and float(out[[5, 149]].abs().sum()) == 0


# ---------------------------------------------------------------- attention
def _paged(k, v, page, pages, seed, dtype, dp, dvp):
    """k [n, G, d], v [n, G, dv] of one sequence -> its pages written into ``pages`` (a pool), and the block-table row."""
    n, G, d = k.shape
    row = torch.cat([torch.nn.functional.pad(k, (0, dp - d)).reshape(n, -1),
                     torch.nn.functional.pad(v, (0, dvp - v.shape[-1])).reshape(n, -1)], -1)
    need = -(-n // page)
    ids = [pages["free"].pop() for _ in range(need)]
    for i, pg in enumerate(ids):
        part = row[i * page:(i + 1) * page]
        pages["pool"][pg, : part.shape[0]] = part.to(dtype)
    return ids


def _attention_case(lens, H, G, d, dv, page, chunk, dtype, seed=0, talk=True, edit=None):
    from batchgen_b200.ops import talking
    g = _gen(seed)
    dp, dvp = -(-d // 8) * 8, -(-dv // 8) * 8
    qs = [torch.randn(n, H, d, generator=g) for n in lens]
    ks = [torch.randn(n, G, d, generator=g) for n in lens]
    vs = [torch.randn(n, G, dv, generator=g) for n in lens]
    T = torch.eye(H) + 0.4 * torch.randn(H, H, generator=g) if talk else None
    if edit:
        edit(qs, ks, vs)
    if dtype == torch.bfloat16:
        ks, vs = [k.bfloat16().float() for k in ks], [v.bfloat16().float() for v in vs]
    n_pages = sum(-(-n // page) for n in lens) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    pool = {"pool": torch.randn(n_pages, page, G * (dp + dvp), generator=g).to(dtype), "free": order}
    tables = [_paged(k, v, page, pool, seed, dtype, dp, dvp) for k, v in zip(ks, vs)]
    bt = torch.zeros(len(lens), max(map(len, tables)) + 1, dtype=torch.int32)
    for i, t in enumerate(tables):
        bt[i, : len(t)] = torch.tensor(t)
    p = talking.TalkParams(H, G, dp, dvp, d ** -0.5, chunk, True, T.to(DEV) if talk else None)
    want = [oracle.talking_attention(q.double(), k.double(), v.double(), (T if talk else torch.eye(H)).double(), d ** -0.5,
                                     chunk or 1 << 30) for q, k, v in zip(qs, ks, vs)]
    q = torch.cat([torch.nn.functional.pad(x, (0, dp - d)).reshape(x.shape[0], -1) for x in qs])
    return q.to(DEV), p, pool["pool"].to(DEV), bt.to(DEV), want, dp, dvp


SHAPES = [(9, 3, 56, 48, 64, 100), (4, 4, 20, 36, 16, 37), (8, 1, 64, 128, 64, 0), (32, 8, 128, 128, 64, 160),
          (1, 1, 8, 8, 32, 16), (16, 2, 40, 200, 128, 64), (10, 2, 96, 24, 64, 1)]


@pytest.mark.parametrize("H,G,d,dv,page,chunk", SHAPES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_rows_and_tiles_match_the_oracle(H, G, d, dv, page, chunk, dtype, monkeypatch):
    from batchgen_b200.ops import _ext, talking
    lens = [150, 33, 1, 300]
    q, p, pool, bt, want, dp, dvp = _attention_case(lens, H, G, d, dv, page, chunk, dtype, seed=H + d)
    T = q.shape[0]
    pos = torch.cat([torch.arange(n) for n in lens])
    seq = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32).to(DEV)
    lens_t = (pos + 1).to(torch.int32).to(DEV)
    full = torch.cat(want)
    tol = 2e-2 if dtype == torch.bfloat16 else 2e-5

    def check(out, what, rows=slice(None)):
        got = out[:, : H * dvp].view(T, H, dvp)[..., :dv][rows]
        assert _rel(got, full[rows]) < tol, what
        worst = (got.double().cpu() - full[rows]).norm(dim=(-1, -2)) / full[rows].norm(dim=(-1, -2)).clamp_min(0.05 * float(full.norm(dim=(-1, -2)).mean()))
        assert float(worst.max()) < 8 * tol, (what, int(worst.argmax()))
    for splits in (1, 3):
        out = torch.full((T, H * dvp + 8), 5.0, dtype=dtype, device=DEV)
        talking.attend_rows(q, p, pool, bt, lens_t, out[:, : H * dvp], seq, num_splits=splits)
        check(out, splits)
        assert float((out[:, H * dvp:] - 5).abs().sum()) == 0
    # a padding row (length 0) is zero, a subset of rows leaves the others alone
    some = torch.tensor([3, 200, 180], dtype=torch.int32, device=DEV)
    lz = lens_t.clone()
    lz[200] = 0
    for splits in (1, 2):
        out = torch.full((T, H * dvp), 5.0, dtype=dtype, device=DEV)
        talking.attend_rows(q, p, pool, bt, lz, out, seq[some.long()].contiguous(), some, num_splits=splits)
        assert float(out[200].abs().sum()) == 0 and float((out[4] - 5).abs().sum()) == 0
        assert _rel(out[[3, 180]].view(2, H, dvp)[..., :dv], full[[3, 180]]) < tol
    if not talking.prefill_supported(p, dtype, page):
        return
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    out = torch.full((T, H * dvp), 5.0, dtype=dtype, device=DEV)
    talking.attend_prefill(q, p, pool, bt, out, talking.work_blocks(talking.prefill_work(cu, [0] * 4, chunk), T, DEV))
    check(out, "tiles")
    # mixed queries held for a few rows at a time (ranges that cut through tiles' alignment)
    monkeypatch.setattr(talking, "_FOLD_ROWS", 100)
    blocks = talking.work_blocks(talking.prefill_work(cu, [0] * 4, chunk), T, DEV)
    assert len(blocks) > 2
    out = torch.full((T, H * dvp), 5.0, dtype=dtype, device=DEV)
    talking.attend_prefill(q, p, pool, bt, out, blocks)
    check(out, "row ranges")
    # the last 70 queries of the long sequence as a piece of their own (cached keys before them)
    out = torch.full((T, H * dvp), 5.0, dtype=dtype, device=DEV)
    talking.attend_prefill(q, p, pool, bt[3:4].contiguous(), out,
                           talking.work_blocks([(T - 70, 70, 0, 230)], T, DEV))
    check(out, "piece", slice(T - 70, T))
    assert float((out[: T - 70] - 5).abs().sum()) == 0
    _ext.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunk", [64, 100, 190])
def test_one_outstanding_key_inside_and_outside_the_chunk(chunk, dtype):
    """The query asks for exactly one key (its score stands far out): first of its chunk, the one before it, page borders,
    itself.  A seen key's value comes out almost alone; an unseen one must leave no trace."""
    from batchgen_b200.ops import _ext, talking
    n, H, G, d, dv = 400, 4, 2, 16, 16
    i = 399 if chunk != 100 else 398
    first = i - i % chunk
    for j in sorted({first, first - 1, first + 1, i, i - 1, 64 * 5, 64 * 5 - 1, 64 * 5 + 63, first - chunk} & set(range(n))):
        if j > i:
            continue

        def edit(qs, ks, vs):
            qs[0][i] = 0.0
            qs[0][i, :, 3] = 6.0
            ks[0][:, :, 3] = 0.0
            ks[0][j, :, 3] = 12.0
            vs[0][j] += 50.0
        q, p, pool, bt, want, dp, dvp = _attention_case([n], H, G, d, dv, 64, chunk, dtype, seed=j, talk=False, edit=edit)
        lens_t = (torch.arange(n) + 1).to(torch.int32).to(DEV)
        seen = first <= j <= i
        ref = want[0][i]
        assert (float(ref.mean()) > 40) == seen
        outs = []
        for splits in (1, 4):
            out = torch.zeros(n, H * dvp, dtype=dtype, device=DEV)
            talking.attend_rows(q, p, pool, bt, lens_t, out, torch.zeros(n, dtype=torch.int32, device=DEV), num_splits=splits)
            outs.append(out)
        if dtype == torch.bfloat16:
            out = torch.zeros(n, H * dvp, dtype=dtype, device=DEV)
            talking.attend_prefill(q, p, pool, bt, out, talking.work_blocks(talking.prefill_work([0, n], [0], chunk), n, DEV))
            outs.append(out)
        for out in outs:
            assert _rel(out[i].view(H, dv), ref) < (3e-2 if dtype == torch.bfloat16 else 1e-4), (j, seen)
    _ext.check_status()


def test_the_sink_takes_its_share():
    """Scores far below 0 leave almost everything to the sink; equal scores of 0 leave it one part of n + 1."""
    from batchgen_b200.ops import talking
    n = 40

    def edit(qs, ks, vs):
        qs[0][:] = 0.0
        ks[0][:] = 0.0
        vs[0][:] = 1.0
        qs[0][20:, :, 0] = -8.0
        ks[0][:, :, 0] = 8.0
    q, p, pool, bt, want, dp, dvp = _attention_case([n], 2, 1, 16, 16, 64, 0, torch.bfloat16, talk=False, edit=edit)
    lens_t = (torch.arange(n) + 1).to(torch.int32).to(DEV)
    outs = [torch.zeros(n, 2 * dvp, dtype=torch.bfloat16, device=DEV) for _ in range(2)]
    talking.attend_rows(q, p, pool, bt, lens_t, outs[0], torch.zeros(n, dtype=torch.int32, device=DEV))
    talking.attend_prefill(q, p, pool, bt, outs[1], talking.work_blocks(talking.prefill_work([0, n], [0], 0), n, DEV))
    for out in outs:
        for t in range(20):
            assert abs(float(out[t].float().mean()) - (t + 1) / (t + 2)) < 5e-3
        assert float(out[20:].float().abs().max()) < 1e-4


# ---------------------------------------------------------------- models
@pytest.mark.parametrize("dtype,tol", [("fp32", 3e-5), ("bf16", 6e-2)])
@pytest.mark.parametrize("name", sorted(nm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name, dtype, tol):
    from batchgen_b200.ops import _ext
    d = nm.CONFIGS[name]
    w = nm.weights_of(d, seed=11)
    toks = nm.prompt(d, 230)
    want = oracle.forward(d, w, toks, torch.float64)
    eng = nm.engine(nm.build(d, w, DEV, dtype))
    for sizes in ([230], [2], [150, 1], [63, 1, 2, 40, 5], [64]):
        s = eng.open_sequence()
        got = nm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert nm.close(got, want, tol, d), (sizes, nm.error(got, want))
    _ext.check_status()
    assert eng.kv.alloc.num_used == 0


@pytest.mark.parametrize("dtype,tol", [("fp32", 3e-5), ("bf16", 6e-2)])
def test_mixed_batches_equal_each_request_alone(dtype, tol):
    d = nm.CONFIGS["odd"]
    w = nm.weights_of(d, seed=12)
    eng = nm.engine(nm.build(d, w, DEV, dtype), tokens=64 * 12)
    prompts = [nm.prompt(d, n, i) for i, n in enumerate((260, 41, 130, 64, 3, 90, 1))]
    want = [oracle.forward(d, w, p, torch.float64) for p in prompts]
    live, at, got, rng = {}, [0] * 7, [[] for _ in prompts], _gen(6)
    order = list(range(7))
    while order or live:
        while order and len(live) < 4:
            live[order[0]] = eng.open_sequence()
            order.pop(0)
        pieces = []
        for i, s in live.items():
            if torch.rand(1, generator=rng) < 0.2 and len(live) > 1:
                continue
            n = 1 if torch.rand(1, generator=rng) < 0.4 else int(torch.randint(2, 100, (1,), generator=rng))
            pieces.append((i, s, min(n, len(prompts[i]) - at[i])))
        if not pieces:
            continue
        out = eng.extend([(s, prompts[i][at[i]:at[i] + n], range(n)) for i, s, n in pieces]).cpu()
        for (i, s, n), rows in zip(pieces, out.split([x[2] for x in pieces])):
            got[i].append(rows)
            at[i] += n
            if at[i] == len(prompts[i]):
                eng.close_sequence(live.pop(i))
    for g, x in zip(got, want):
        assert nm.close(torch.cat(g), x, tol, d), nm.error(torch.cat(g), x)
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("dtype,tol", [("fp32", 1e-4), ("bf16", 6e-2)])
def test_a_long_prompt_over_many_pages_and_chunks(dtype, tol):
    d = nm.config(150, 64, [nm.delta(2, 32, nm.dense(64)), nm.attention(4, 2, 16, 24, 700, nm.moe(40, 3, 3, 1.2, 24))])
    w = nm.weights_of(d, seed=15)
    toks = nm.prompt(d, 1500)
    want = oracle.forward(d, w, toks, torch.float64)
    eng = nm.engine(nm.build(d, w, DEV, dtype), tokens=1536 + 64)
    for sizes in ([1500], [1390, 1], [333]):
        s = eng.open_sequence()
        got = nm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert nm.close(got, want, tol, d), (sizes, nm.error(got, want))


def test_greedy_generation_in_32_bit_and_long_decoding():
    from batchgen_b200.runtime.sequence import SamplingParams
    d = nm.CONFIGS["twice"]
    w = nm.weights_of(d, seed=13)
    prompts = [nm.prompt(d, n, i) for i, n in enumerate((90, 7, 40))]
    eng = nm.engine(nm.build(d, w, DEV, "fp32"), tokens=64 * 64)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=120, ignore_eos=True))
    for p, o in zip(prompts, outs):
        logits = oracle.forward(d, w, p + o, torch.float64)[len(p) - 1:-1]
        assert len(o) == 120 and logits.argmax(-1).tolist() == o


def test_captured_decode_steps_equal_eager_ones():
    from batchgen_b200.runtime.graphs import DecodeGraphRunner
    from batchgen_b200.runtime.sequence import SamplingParams
    d = nm.CONFIGS["twice"]
    w = nm.weights_of(d, seed=14)
    model = nm.build(d, w, DEV, "bf16")
    prompts = [nm.prompt(d, n, i) for i, n in enumerate((70, 9, 130, 33, 5))]
    params = SamplingParams(max_new_tokens=40, ignore_eos=True)
    eager = nm.engine(model, tokens=64 * 40, slots=8).generate(prompts, params)
    eng = nm.engine(model, tokens=64 * 40, slots=8)
    eng.graph_runner = DecodeGraphRunner(model, eng.kv, max_batch=8, max_pages_per_seq=40, num_buckets=2)
    eng.graph_runner.capture_all()
    outs = eng.generate(prompts, params)
    assert eng.graph_runner.replays > 0
    # summation orders differ with the batch: tokens agree until the first near-tie of the exact logits
    for p, a, b in zip(prompts, eager, outs):
        n = next((i for i, (x, y) in enumerate(zip(a, b)) if x != y), len(a))
        if n < len(a):
            row = oracle.forward(d, w, p + a[:n], torch.float64)[-1]
            assert float((row[a[n]] - row[b[n]]).abs()) < 0.1 * float(row.std()), n


def test_sampled_rows_and_server_style_engine_on_the_tiny_preset():
    from batchgen_b200.config import get_model_config
    from batchgen_b200.models import build_model
    from batchgen_b200.runtime.sequence import SamplingParams
    model = build_model(get_model_config("tiny-nanurax"), device=DEV, dtype="bf16", seed=1)
    eng = nm.engine(model, tokens=64 * 40, slots=4)
    outs = eng.generate([[1, 2, 3], [5] * 70], [SamplingParams(max_new_tokens=9, temperature=0.8, top_k=20),
                                               SamplingParams(max_new_tokens=5)])
    assert [len(o) for o in outs] == [9, 5]
