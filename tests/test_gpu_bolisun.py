"""Bolisun kernels and models on the GPU against the plain implementation, in bf16 and in true fp32."""
import pytest
import torch
import torch.nn.functional as F

import bolisun_models as bm
import bolisun_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-30))


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def _pad(t, w):
    return F.pad(t, (0, w - t.shape[-1]))


# ---------------------------------------------------------------- row operators
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,D,S", [(5, 99, 1), (3, 1030, 2), (300, 515, 2), (9, 2307, 3), (7, 260, 4), (2, 5001, 5), (2, 8192, 2),
                                   (1, 6, 9), (3, 130, 16)])
def test_streams_join_mix_and_are_read(T, D, S, dtype):
    from batchgen_b200.ops import residual
    g, K = _gen(T + D), 5
    D4, cols = -(-D // 4) * 4, -(-D // 64) * 64
    tol = 5e-3 if dtype == BF else 2e-6
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    x, add, bias, routed = _pad(r(T, S, D), D4), r(T, D4), r(D), r(11, D4)
    pos = torch.randint(-1, 11, (T, K), generator=g).to(torch.int32)
    rw, w, read = torch.rand(T, K, generator=g), 1 + 0.2 * r(D), r(S)
    hc = residual.Hyper(*(t.to(DEV) for t in (r(S), r(S, S), r(S))))
    mix, share = hc.mix.cpu().double(), hc.share.cpu().double()
    rows = torch.where((pos >= 0).unsqueeze(-1), routed[pos.clamp_min(0).long()], torch.zeros(1)).double()
    moe = (rw.double().unsqueeze(-1) * rows).sum(1)[:, :D]
    padded = _pad(bias, D4).to(DEV)
    for dense, more, y in ((add, dict(bias=padded), add[:, :D].double() + bias), (None, dict(bias=padded), bias.double().expand(T, D)),
                           (add, dict(routed=routed.to(DEV), pos=pos.to(DEV), route_w=rw.to(DEV)), add[:, :D].double() + moe),
                           (None, dict(routed=routed.to(DEV), pos=pos.to(DEV), route_w=rw.to(DEV)), moe)):
        want = torch.einsum("st,nsd->ntd", mix, x[..., :D].double()) + share.view(1, S, 1) * y.unsqueeze(1)
        xd = x.to(DEV)
        h = residual.hyper_norm(xd, _pad(w, D4).to(DEV), 1e-5, D, cols, dtype, read=read.to(DEV), hc=hc,
                                add=None if dense is None else dense.to(DEV), **more)
        assert _rel(xd[..., :D], want) < 2e-6 and float(xd[..., D:].abs().sum()) == 0
        u = torch.einsum("s,nsd->nd", read.double(), want)
        assert _rel(h[:, :D], oracle.rms(u, 1e-5) * w) < tol and float(h[:, D:].abs().sum()) == 0
    # picked rows, the plain sum, streams left alone
    some = torch.tensor([T - 1, 0, T - 1])
    before = x.to(DEV)
    h = residual.hyper_norm(before, _pad(w, D4).to(DEV), 1e-5, D, cols, dtype, hc=hc, add=add.to(DEV), rows=some.to(DEV), keep=False)
    want = (torch.einsum("st,nsd->ntd", mix, x[..., :D].double()) + share.view(1, S, 1) * add[:, :D].double().unsqueeze(1)).sum(1)
    assert torch.equal(before.cpu(), x) and _rel(h[:, :D], (oracle.rms(want, 1e-5) * w)[some]) < tol
    h = residual.hyper_norm(before, _pad(w, D4).to(DEV), 1e-5, D, cols, dtype)
    assert _rel(h[:, :D], oracle.rms(x[..., :D].double().sum(1), 1e-5) * w) < tol
    # the embedding fills every stream
    emb, ids = r(11, D).to(dtype), torch.randint(0, 11, (T,), generator=g).to(torch.int32)
    residual.hyper_norm(before, _pad(w, D4).to(DEV), 1e-5, D, cols, dtype, read=read.to(DEV), ids=ids.to(DEV), embed=emb.to(DEV),
                        embed_scale=2.5)
    assert torch.allclose(before[..., :D].cpu(), (emb[ids.long()].float() * 2.5).unsqueeze(1).expand(T, S, D))


def test_gated_silu():
    from batchgen_b200.ops import residual
    z = 3 * torch.randn(7, 88, generator=_gen(1))
    want = oracle.silu(z[:, 8:48].double()) * z[:, 48:88].double()
    for dtype, tol in ((BF, 5e-3), (F32, 1e-6)):
        y = torch.full((7, 64), 5.0, dtype=dtype, device=DEV)
        residual.glu(z.to(DEV)[:, 8:], 40, "silu", out=y)
        assert _rel(y[:, :40], want) < tol and float(y[:, 40:].abs().sum()) == 0


@pytest.mark.parametrize("E,top,groups", [(12, 3, (4, 2)), (12, 1, (3, 3)), (64, 8, (8, 4)), (30, 5, (10, 3)), (7, 2, None), (1, 1, None),
                                          (12, 1, (12, 1)), (160, 6, (32, 5))])
def test_router(E, top, groups):
    from batchgen_b200.ops import moe
    z, corr = torch.randn(50, E + 4, generator=_gen(E)), 0.2 * torch.randn(E, generator=_gen(3)) - 1.0
    idx, w = oracle.route(z[:, :E].double(), corr.double(), {"top": top, "scale": 1.3, "groups": groups and dict(zip(("count", "keep"), groups))})
    i2, w2 = moe.router_topk(z.to(DEV)[:, :E], corr.to(DEV), top, *(groups or (1, 1)), "always", 1.3, "softmax_all", None, "max")
    assert torch.equal(idx.sort(-1)[0], i2.cpu().long().sort(-1)[0])
    assert torch.allclose(w.sort(-1)[0], w2.cpu().double().sort(-1)[0], atol=1e-6)


@pytest.mark.parametrize("dtype,tol", [(F32, 2e-6), (BF, 1e-2)])
def test_experts_weighted_at_the_sum(dtype, tol):
    from batchgen_b200.ops import moe, residual
    g, D, Fe, E, T, top = _gen(9), 72, 40, 6, 37, 3
    w = {f"e{e}.{x}": (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype).float() for e in range(E)
         for x, s in (("gate", (Fe, D)), ("up", (Fe, D)), ("down", (D, Fe)))}
    h = torch.randn(T, D, generator=g).to(dtype).float()
    idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    rw = torch.rand(T, top, generator=g)
    want = torch.zeros(T, D, dtype=F64)
    for t in range(T):
        for k in range(top):
            want[t] += rw[t, k].double() * oracle.expert(h[t:t + 1].double(), {n: x.double() for n, x in w.items()}, f"e{idx[t, k]}.")[0]
    w13 = torch.stack([torch.cat([_pad(F.pad(w[f"e{e}.{x}"], (0, 0, 0, 24)), 128) for x in ("gate", "up")]) for e in range(E)])
    w2 = torch.stack([_pad(w[f"e{e}.down"], 64) for e in range(E)])
    ew = moe.ExpertWeights(w13.to(dtype).to(DEV), w2.to(dtype).to(DEV), activation="silu")
    rows, pos = moe.routed_rows(_pad(h, 128).to(dtype).to(DEV), idx.to(DEV), rw.to(DEV), ew, False)
    x, one = torch.zeros(T, 1, D, device=DEV), torch.ones(1, device=DEV)
    residual.hyper_norm(x, torch.ones(D, device=DEV), 1e-5, D, 128, dtype, hc=residual.Hyper(one, one.view(1, 1), one), routed=rows,
                        pos=pos, route_w=rw.to(DEV))
    assert _rel(x[:, 0], want) < tol


@pytest.mark.parametrize("sc", [None, bm.scaling(8.0, 3000, 32.0, 1.0), bm.scaling(2.5, 77, 5.0, 0.4)])
def test_rotary_tables_are_exact_far_away(sc):
    from batchgen_b200.ops.conv import Rotary
    for dims, base in ((2, 10.0), (20, 500.0), (128, 1e6)):
        r = Rotary.make(dims, base, DEV, True, tuple(sc[k] for k in ("factor", "original", "fast", "slow")) if sc else ())
        pos = torch.tensor([0, 1, 63, 64, 4095, 100_000, 3_000_000])
        got = r.table((pos + 1).to(torch.int32).to(DEV)).double().cpu()
        a = pos.double().unsqueeze(1) * torch.tensor(oracle.frequencies(dims, base, sc), dtype=F64)
        assert float((got - torch.cat([a.cos(), a.sin()], 1) * r.mult).abs().max()) < 1e-6


# ---------------------------------------------------------------- attention
class _Attention:
    """Random heads of several sequences through bias, norm, rotation and cache, and the plain form's outputs."""

    def __init__(self, lens, H, G, d, dv, rd, window, keep, page, dtype, seed=0, edit=None, sc=None, bias=True):
        from batchgen_b200.ops import talking
        from batchgen_b200.ops.conv import Rotary
        g = _gen(seed)
        r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
        dp, dvp = -(-d // 8) * 8, -(-dv // 8) * 8
        self.H, self.dv, self.T, self.lens = H, dv, sum(lens), lens
        self.p = p = talking.TalkParams(H, G, dp, dvp, (4.5 if edit else 1.1) * d ** -0.5, window=window, keep=keep, out_scale=0.7)
        qs, ks, vs = ([r(n, h, w) for n in lens] for h, w in ((H, d), (G, d), (G, dv)))
        b = [0.5 * r(h, w) * bias for h, w in ((H, d), (G, d), (G, dv))]
        wq, wk = 1 + 0.2 * r(d), 1 + 0.2 * r(d)
        if edit:
            edit(qs, ks, vs)
        self.prep = talking.HeadPrep(d, 1e-5, torch.cat([_pad(x, w).reshape(-1) for x, w in zip(b, (dp, dp, dvp))]).to(DEV),
                                     _pad(wq, dp).to(DEV), _pad(wk, dp).to(DEV), True)
        rot = Rotary.make(rd, 200.0, DEV, True, tuple(sc[k] for k in ("factor", "original", "fast", "slow")) if sc else ())
        self.pos = torch.cat([torch.arange(n) for n in lens])
        self.lens_t = (self.pos + 1).to(torch.int32).to(DEV)
        self.rope = rot.table(self.lens_t)
        n_pages = sum(-(-n // page) for n in lens) + 3
        order = torch.randperm(n_pages, generator=g).tolist()
        self.pool = r(n_pages, page, p.kv_row).to(dtype).to(DEV)
        bt = torch.zeros(len(lens), max(-(-n // page) for n in lens) + 1, dtype=torch.int32)
        slots, used = [], 0
        for i, n in enumerate(lens):
            need = -(-n // page)
            bt[i, :need] = torch.tensor(order[used:used + need])
            slots += [int(bt[i, t // page]) * page + t % page for t in range(n)]
            used += need
        self.bt, self.slots = bt.to(DEV), torch.tensor(slots, device=DEV)
        self.seq = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32).to(DEV)
        cat = lambda xs, w: torch.cat([_pad(x, w).reshape(x.shape[0], -1) for x in xs])      # noqa: E731
        self.z = torch.cat([torch.zeros(self.T, 8), cat(qs, dp), cat(ks, dp), cat(vs, dvp), torch.full((self.T, 4), 9.0)], 1)
        self.want, self.q = [], []
        for q, k, v in zip(qs, ks, vs):
            q, k, v = (x.double() + y for x, y in zip((q, k, v), b))
            q, k = (oracle.rotate(oracle.rms(x, 1e-5) * y, 200.0, rd, sc) for x, y in ((q, wq), (k, wk)))
            seen = oracle.visible(len(q), window or len(q), keep)
            self.want.append(oracle.attention(q, k, v, p.scale, seen) * 0.7)
            self.q.append(q)

    def prepare(self, operand, write_q=True):
        """The projections' columns as a step would have them; returns (queries' view, the prompt kernel's operand)."""
        from batchgen_b200.ops import talking
        z = self.z.to(DEV)
        n = self.H * self.p.dim_p
        qf = talking.prepare_heads(z[:, 8:], self.slots, self.pool, self.p, self.prep, self.rope, write_q, operand)
        assert float(z[:, :8].abs().sum()) == 0 and float((z[:, -4:] - 9).abs().sum()) == 0
        return z[:, 8:8 + n], qf

    def out(self, dtype):
        return torch.full((self.T, self.H * self.p.vdim_p), 5.0, dtype=dtype, device=DEV)

    def heads(self, out):
        return out.view(self.T, self.H, self.p.vdim_p)[..., :self.dv]


SHAPES = [(9, 3, 56, 48, 56, 64, 64), (4, 4, 20, 36, 6, 16, 33), (8, 1, 80, 128, 32, 64, 100), (32, 8, 128, 128, 128, 64, 128),
          (1, 1, 8, 8, 2, 32, 1), (16, 2, 40, 200, 24, 128, 17), (10, 2, 96, 24, 96, 64, 250), (6, 2, 136, 264, 60, 64, 90),
          (2, 1, 384, 40, 128, 64, 65), (12, 12, 8, 512, 8, 32, 40), (20, 4, 128, 64, 128, 64, 700),
          (20, 1, 120, 88, 64, 16, 75), (24, 2, 64, 56, 64, 64, 130)]


@pytest.mark.parametrize("H,G,d,dv,rd,page,window", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF])
def test_windowed_attention_rows_and_tiles(H, G, d, dv, rd, page, window, dtype):
    from batchgen_b200.ops import _ext, talking
    lens = [150, 33, 1, 500]
    tol = 2e-2 if dtype == BF else 2e-5
    for keep in (0, 7, 64, 140):
        sc = bm.scaling(4.0, 90, 8.0, 0.5) if keep else None
        a = _Attention(lens, H, G, d, dv, rd, window, keep, page, dtype, H + d + keep, sc=sc)
        p, full = a.p, torch.cat(a.want)
        tiles = talking.prefill_supported(p, dtype, page)
        q, qf = a.prepare(tiles)
        if qf is not None:
            want = torch.cat(a.q) * p.scale * 1.4426950408889634
            assert _rel(qf[..., :d], want) < 5e-3 and float(qf[..., d:].abs().sum()) == 0
        assert _rel(q.view(a.T, H, p.dim_p)[..., :d], torch.cat(a.q)) < 2e-6
        for splits in (1, 3, 0):
            out = a.out(dtype)
            talking.attend_rows(q, p, a.pool, a.bt, a.lens_t, out, a.seq, num_splits=splits)
            assert _rel(a.heads(out), full) < tol, (keep, splits)
        some = [3, 650, 180]
        out = a.out(dtype)
        talking.attend_rows(q, p, a.pool, a.bt, a.lens_t, out, a.seq[torch.tensor(some)].contiguous(), _i32(some), num_splits=2)
        assert _rel(a.heads(out)[some], full[some]) < tol and float((out[4] - 5).abs().sum()) == 0
        if not tiles:
            continue
        cu = [0, 150, 183, 184, 684]
        out = a.out(dtype)
        blocks = talking.work_blocks(talking.prefill_work(cu, [0] * 4, 0, 1, window), a.T, DEV)
        talking.attend_prefill(q, p, a.pool, a.bt, out, blocks, operand=qf)
        assert _rel(a.heads(out), full) < tol, keep
        for n in (1, 70, 260):                                        # pieces of their own, cached keys before them
            out = a.out(dtype)
            talking.attend_prefill(q, p, a.pool, a.bt[3:4].contiguous(), out, talking.work_blocks(
                [(a.T - n + i, min(128, n - i), 0, 500 - n + i) for i in range(0, n, 128)], a.T, DEV), operand=qf)
            assert _rel(a.heads(out)[-n:], full[-n:]) < tol and float((out[: a.T - n] - 5).abs().sum()) == 0
    _ext.check_status()


@pytest.mark.parametrize("H,G,d,dv", [(6, 2, 24, 40), (33, 1, 128, 128), (10, 1, 64, 8)])
def test_row_kernel_of_plain_heads_with_chunks_a_sink_and_gates(H, G, d, dv):
    """The parts of the row kernel that other designs use."""
    from batchgen_b200.ops import talking
    g, n, chunk = _gen(H), 200, 70
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    q, k, v, gate = r(n, H, d), r(n, G, d).to(BF).float(), r(n, G, dv).to(BF).float(), r(n, H)
    p = talking.TalkParams(H, G, d, dv, d ** -0.5, chunk, True, out_scale=1.5)
    pool = torch.zeros(4, 64, p.kv_row, dtype=BF, device=DEV)
    pool.view(256, -1)[:n] = torch.cat([k.reshape(n, -1), v.reshape(n, -1)], 1).to(DEV)
    i, j = torch.arange(n).view(-1, 1), torch.arange(n).view(1, -1)
    seen = torch.cat([(j <= i) & (j // chunk == i // chunk), torch.ones(n, 1, dtype=torch.bool)], 1)
    more = [torch.cat([x.double(), torch.zeros(1, *x.shape[1:], dtype=F64)]) for x in (k, v)]        # the sink: a score of 0, a value of 0
    want = oracle.attention(q.double(), *more, d ** -0.5, seen) * 1.5 * torch.sigmoid(gate.double()).unsqueeze(-1)
    lens = torch.arange(1, n + 1, dtype=torch.int32)
    lens[13] = 0
    for splits in (1, 2, 5):
        out = torch.full((n, H * dv), 5.0, dtype=BF, device=DEV)
        talking.attend_rows(q.reshape(n, -1).to(DEV), p, pool, _i32([[0, 1, 2, 3]]), lens.to(DEV), out, torch.zeros(n, dtype=torch.int32,
                            device=DEV), num_splits=splits, gate=gate.to(DEV))
        got = out.view(n, H, dv)
        assert float(got[13].abs().sum()) == 0
        keep = [t for t in range(n) if t != 13]
        assert _rel(got[keep], want[keep]) < 1e-2, splits


def test_heads_without_norms_turn_halves_too():
    """The same kernel for heads as other designs have them: no bias, no norm, pairs (i, i + half)."""
    from batchgen_b200.ops import talking
    from batchgen_b200.ops.conv import Rotary, rotate_ref
    for d, half in ((24, 12), (136, 50), (520, 200), (8, 1)):
        g = _gen(d)
        p = talking.TalkParams(3, 2, d, 16, 0.3)
        z = torch.randn(5, 3 * d + p.kv_row, generator=g)
        pool = torch.zeros(2, 16, p.kv_row, device=DEV)
        rope = Rotary.make(2 * half, 90.0, DEV).table(_i32([1, 5, 9, 40, 1000]))
        zd = z.to(DEV)
        qf = talking.prepare_heads(zd, torch.tensor([3, 30, -1, 7, 16], device=DEV), pool, p, talking.HeadPrep(d), rope, True, True)
        want = rotate_ref(z[:, :5 * d].view(5, 5, d), rope.cpu())
        assert _rel(zd[:, :3 * d].view(5, 3, d), want[:, :3]) < 2e-6 and _rel(qf[..., :d], want[:, :3] * 0.3 * 1.4426950408889634) < 5e-3
        flat = pool.view(32, -1).cpu()
        for t, s in ((0, 3), (1, 30), (3, 7), (4, 16)):
            assert _rel(flat[s], torch.cat([want[t, 3:].reshape(-1), z[t, 5 * d:]])) < 2e-6
        assert float(flat[[i for i in range(32) if i not in (3, 30, 7, 16)]].abs().sum()) == 0


@pytest.mark.parametrize("window,keep", [(70, 21), (64, 64), (50, 0), (1, 1), (130, 100), (300, 3)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_one_outstanding_key_at_every_kind_of_place(dtype, window, keep):
    """The query asks for exactly one key (its score stands far out): kept first tokens and the next ones, just inside and just
    outside the window, page borders, its neighbour, itself, the next token.  The channels that carry the score do not turn."""
    from batchgen_b200.ops import _ext, talking
    n, H, G, d, dv, i = 400, 4, 2, 16, 16, 390
    edge = i - window
    places = {0, 1, keep - 1, keep, keep + 1, edge - 1, edge, edge + 1, edge + 2, 63, 64, 319, 320, 383, 384, i - 1, i, i + 1}
    for j in sorted(x for x in places if 0 <= x < n):
        def edit(qs, ks, vs):
            qs[0][i] = 0.01
            qs[0][i, :, 12:] = 8.0
            ks[0][:, :, 12:] = 0.0
            ks[0][j] *= 0.01
            ks[0][j, :, 12:] = 14.0
            vs[0][j] += 50.0
        a = _Attention([n], H, G, d, dv, 8, window, keep, 64, dtype, j, edit, bias=False)
        seen = j <= i and (i - j < window or j < keep)
        assert (float(a.want[0][i].mean()) > 20) == seen, j
        q, qf = a.prepare(dtype == BF)
        outs = []
        for splits in (1, 4):
            outs.append(a.out(dtype))
            talking.attend_rows(q, a.p, a.pool, a.bt, a.lens_t, outs[-1], a.seq, num_splits=splits)
        if dtype == BF:
            for cut in ([0, n], [0, i - 1, n], [0, 257, n]):                # the query's place in its tile differs
                outs.append(a.out(dtype))
                work = [w for s, e in zip(cut, cut[1:]) for w in talking.prefill_work([0, e - s], [s], 0, 1, window)]
                at = [s for s, e in zip(cut, cut[1:]) for _ in talking.prefill_work([0, e - s], [s], 0, 1, window)]
                work = [(w[0] + s, w[1], 0, w[3]) for w, s in zip(work, at)]
                talking.attend_prefill(q, a.p, a.pool, a.bt, outs[-1], talking.work_blocks(work, n, DEV), operand=qf)
        for out in outs:
            assert _rel(a.heads(out)[i], a.want[0][i]) < (3e-2 if dtype == BF else 1e-4), (j, seen)
    _ext.check_status()


# ---------------------------------------------------------------- models
TOL = [("fp32", 1e-4), ("bf16", 6e-2)]


def _close(got, want, tol, d):
    """In 32 bits every row within ``tol``.  In 16 bits single rows stand out (a narrow head whose output nearly cancels is blown up
    by its norm), and a close choice of experts may flip, after which states carry the difference on."""
    e = bm.row_errors(got, want)
    if tol < 1e-3:
        return bool(e.max() < tol)
    if any((l["mlp"] or {}).get("kind") == "moe" for l in d["layers"]):
        return bool((e > tol).double().mean() <= 0.15 and e.median() < tol / 2)
    return bool(e.max() < 4 * tol and e.mean() < tol / 2)


def _weights(d, seed, dtype):
    return bm.weights_of(d, seed, settled=dtype == "bf16")


@pytest.mark.parametrize("dtype,tol", TOL)
@pytest.mark.parametrize("name", sorted(bm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name, dtype, tol):
    from batchgen_b200.ops import _ext
    d = bm.CONFIGS[name]
    w = _weights(d, 11, dtype)
    toks = bm.prompt(d, 230)
    want = oracle.forward(d, w, toks, F64)
    eng = bm.engine(bm.build(d, w, DEV, dtype))
    for sizes in ([230], [2], [150, 1], [63, 1, 2, 40, 5], [64]):
        s = eng.open_sequence()
        got = bm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert _close(got, want, tol, d), (sizes, bm.row_errors(got, want).sort()[0][-40:])
    _ext.check_status()
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("seed", range(10, 22))
def test_random_designs(seed):
    d = bm.random_config(seed)
    toks = bm.prompt(d, 140)
    for dtype, tol in TOL:
        w = _weights(d, seed, dtype)
        want = oracle.forward(d, w, toks, F64)
        eng = bm.engine(bm.build(d, w, DEV, dtype))
        for sizes in ([140], [37, 2, 1]):
            got = bm.run_pieces(eng, eng.open_sequence(), toks, sizes)
            assert _close(got, want, tol, d), (dtype, sizes, bm.row_errors(got, want).sort()[0][-40:])


@pytest.mark.parametrize("dtype,tol", TOL)
def test_mixed_batches_equal_each_request_alone(dtype, tol):
    d = bm.CONFIGS["odd"] if dtype == "fp32" else bm.without_choices(bm.CONFIGS["odd"])
    w = bm.weights_of(d, seed=12)
    eng = bm.engine(bm.build(d, w, DEV, dtype), tokens=64 * 12)
    prompts = [bm.prompt(d, n, i) for i, n in enumerate((260, 41, 130, 64, 3, 90, 1))]
    want = [oracle.forward(d, w, p, F64) for p in prompts]
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
    assert _close(torch.cat([torch.cat(g) for g in got]), torch.cat(want), tol, d)
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("dtype,tol", TOL)
def test_a_long_prompt_over_many_pages(dtype, tol):
    d = bm.config(150, 64, 2, [bm.layer((4, 2, 16, 24), (100, 70), (16, 1e4, bm.scaling(4.0, 300, 16.0, 1.0)), ((0.99, 0.999), 16, 16),
                                        bm.dense(64, 1.0)), bm.layer((3, 1, 24, 16), (700, 5), (8, 1e4, None), ((0.9,), 16, 24))])
    w = bm.weights_of(d, seed=15)
    toks = bm.prompt(d, 1200)
    want = oracle.forward(d, w, toks, F64)
    eng = bm.engine(bm.build(d, w, DEV, dtype), tokens=1216 + 64)
    for sizes in ([1200], [1100, 1], [333]):
        s = eng.open_sequence()
        got = bm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert _close(got, want, tol, d), (sizes, bm.error(got, want))


def test_greedy_generation_in_32_bit_and_long_decoding():
    from batchgen_b200.runtime.sequence import SamplingParams
    d = bm.CONFIGS["odd"]
    w = bm.weights_of(d, seed=13)
    prompts = [bm.prompt(d, n, i) for i, n in enumerate((90, 7, 40))]
    eng = bm.engine(bm.build(d, w, DEV, "fp32"), tokens=64 * 64)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=120, ignore_eos=True))
    for p, o in zip(prompts, outs):
        logits = oracle.forward(d, w, p + o, F64)[len(p) - 1:-1]
        assert len(o) == 120 and logits.argmax(-1).tolist() == o


@pytest.mark.parametrize("name", ["whole", "wide"])
def test_captured_decode_steps_equal_eager_ones(name):
    from batchgen_b200.runtime.graphs import DecodeGraphRunner
    from batchgen_b200.runtime.sequence import SamplingParams
    d = bm.CONFIGS[name]
    w = bm.weights_of(d, seed=14)
    model = bm.build(d, w, DEV, "bf16")
    prompts = [bm.prompt(d, n, i) for i, n in enumerate((70, 9, 130, 33, 5))]
    params = SamplingParams(max_new_tokens=40, ignore_eos=True)
    eager = bm.engine(model, tokens=64 * 40, slots=8).generate(prompts, params)
    eng = bm.engine(model, tokens=64 * 40, slots=8)
    eng.graph_runner = DecodeGraphRunner(model, eng.kv, max_batch=8, max_pages_per_seq=40, num_buckets=2)
    eng.graph_runner.capture_all()
    outs = eng.generate(prompts, params)
    assert eng.graph_runner.replays > 0
    # summation orders differ with the batch: tokens agree until the first near-tie of the exact logits
    for p, a, b in zip(prompts, eager, outs):
        n = next((i for i, (x, y) in enumerate(zip(a, b)) if x != y), len(a))
        if n < len(a):
            row = oracle.forward(d, w, p + a[:n], F64)[-1]
            assert float((row[a[n]] - row[b[n]]).abs()) < 0.15 * float(row.std()), n


def test_sampled_rows_and_server_style_engine_on_the_tiny_preset():
    from batchgen_b200.config import get_model_config
    from batchgen_b200.models import build_model
    from batchgen_b200.runtime.sequence import SamplingParams
    model = build_model(get_model_config("tiny-bolisun"), device=DEV, dtype="bf16", seed=1)
    eng = bm.engine(model, tokens=64 * 40, slots=4)
    outs = eng.generate([[1, 2, 3], [5] * 70], [SamplingParams(max_new_tokens=9, temperature=0.8, top_k=20),
                                               SamplingParams(max_new_tokens=5)])
    assert [len(o) for o in outs] == [9, 5]
