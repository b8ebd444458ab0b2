"""Pitudra kernels and models on the GPU against the plain implementation, in bf16 and in true fp32."""
import pytest
import torch
import torch.nn.functional as F

import pitudra_models as pm
import pitudra_oracle as oracle

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


def _up(n, m=8):
    return -(-n // m) * m


# ---------------------------------------------------------------- row operators
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,D,K", [(5, 99, 3), (3, 1030, 1), (300, 515, 8), (2, 5001, 16), (1, 6, 5), (7, 2304, 4), (2, 16384, 2)])
def test_outputs_join_behind_their_norm(T, D, K, dtype):
    from batchgen_b200.ops import residual
    g, D4, cols = _gen(T + D), _up(D, 4), _up(D, 64)
    tol = 5e-3 if dtype == BF else 2e-6
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    x, add, routed = _pad(r(T, D), D4), _pad(3 + r(T, D), D4), _pad(r(11, D), D4)
    pos = torch.randint(-1, 11, (T, K), generator=g).to(torch.int32)
    rw, w, b, mu = torch.rand(T, K, generator=g), 1 + 0.2 * r(D), r(D), torch.rand(D, generator=g)
    rows = torch.where((pos >= 0).unsqueeze(-1), routed[pos.clamp_min(0).long()], torch.zeros(1)).double()
    moe = (rw.double().unsqueeze(-1) * rows).sum(1)[:, :D]
    norm, plain = residual.Norm(_pad(w, D4).to(DEV), _pad(b, D4).to(DEV), True), residual.Norm(_pad(w, D4).to(DEV))
    for kw, want in ((dict(add=add.to(DEV), post=norm), oracle.layer_norm(add[:, :D].double(), w, b, 1e-5)),
                     (dict(add=add.to(DEV), post=plain), oracle.rms(add[:, :D].double(), 1e-5) * w),
                     (dict(routed=routed.to(DEV), pos=pos.to(DEV), route_w=rw.to(DEV), post=norm), oracle.layer_norm(moe, w, b, 1e-5))):
        want = want + x[:, :D].double()
        xd = x.to(DEV)
        h = residual.sandwich_norm(xd, None, 1e-5, D, cols, dtype, **kw)
        assert _rel(xd[:, :D], want) < 2e-6 and float(xd[:, D:].abs().sum()) == 0
        assert _rel(h[:, :D], want) < tol and float(h[:, D:].abs().sum()) == 0
        xd = x.to(DEV)
        assert residual.sandwich_norm(xd, None, 1e-5, D, cols, dtype, emit=False, **kw) is None and _rel(xd[:, :D], want) < 2e-6
        # the shift towards the previous token, whose row is in the slot (no slot: zeros, none kept)
        hist = torch.zeros(T + 2, D4 + 4, device=DEV)[:, :D4]
        old = r(T + 2, D4)
        hist.copy_(old)
        slots = torch.randperm(T + 2, generator=g)[:T].to(torch.int32)
        if T > 1:
            slots[1] = -1
        taps = torch.stack([_pad(mu, D4), -_pad(mu, D4)]).to(DEV)
        h = residual.sandwich_norm(x.to(DEV), None, 1e-5, D, cols, dtype, canon=residual.Canon(taps, hist, slots.to(DEV)), **kw)
        before = torch.where((slots >= 0).unsqueeze(-1), old[slots.clamp_min(0).long(), :D], torch.zeros(1)).double()
        assert _rel(h[:, :D], want + (before - want) * mu) < tol and float(h[:, D:].abs().sum()) == 0
        kept = hist.cpu()
        for t in range(T):
            if slots[t] >= 0:
                assert _rel(kept[int(slots[t]), :D], want[t]) < 2e-6
        # the final norm reads picked rows and leaves the residual alone
        some, xd = torch.tensor([T - 1, 0, T - 1]), x.to(DEV)
        h = residual.sandwich_norm(xd, norm, 1e-5, D, cols, dtype, rows=some.to(DEV), keep=False, **kw)
        assert torch.equal(xd.cpu(), x) and _rel(h[:, :D], oracle.layer_norm(want[some], w, b, 1e-5)) < tol


@pytest.mark.parametrize("n,layers,cols", [(11, 3, 64), (64, 1, 64), (130, 2, 192), (1, 5, 64)])
def test_side_rows(n, layers, cols):
    from batchgen_b200.ops import residual
    g = _gen(n)
    z, ids = 2 * torch.randn(9, _up(n), generator=g), torch.randint(0, 37, (9,), generator=g).to(torch.int32)
    for dtype, tol in ((BF, 5e-3), (F32, 1e-6)):
        table = torch.randn(37, layers * n, generator=g).to(dtype)
        i = layers - 1
        y = residual.token_side(z.to(DEV), table.to(DEV)[:, i * n:(i + 1) * n], ids.to(DEV), cols, dtype)
        want = oracle.gelu_tanh(z[:, :n].double()) * table[ids.long(), i * n:].double()
        assert _rel(y[:, :n], want) < tol and float(y[:, n:].abs().sum()) == 0


@pytest.mark.parametrize("dtype,tol", [(F32, 2e-6), (BF, 1e-2)])
@pytest.mark.parametrize("D,Fe,E,T,top", [(72, 40, 6, 37, 3), (128, 128, 4, 300, 2), (200, 96, 9, 3, 9), (64, 200, 1, 5, 1)])
def test_squared_relu_experts(D, Fe, E, T, top, dtype, tol):
    from batchgen_b200.ops import moe, residual
    g, Dp, Fp = _gen(D), _up(D, 64), _up(Fe, 64)
    w = {f"e{e}.{x}": (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype).float() for e in range(E) for x, s in (("up", (Fe, D)), ("down", (D, Fe)))}
    w["router"] = torch.randn(E, D, generator=g)
    h = torch.randn(T, D, generator=g).to(dtype).float()
    want = oracle.mixture(h.double(), {k: v.double() for k, v in w.items()}, "", {"router": {"experts": E, "top": top}})
    idx, rw = moe.router_topk((h @ w["router"].T).to(DEV), None, top, scoring="softmax")
    ew = moe.ExpertWeights(torch.stack([_pad(F.pad(w[f"e{e}.up"], (0, 0, 0, Fp - Fe)), Dp) for e in range(E)]).to(dtype).to(DEV),
                           torch.stack([_pad(w[f"e{e}.down"], Fp) for e in range(E)]).to(dtype).to(DEV), activation="relu2")
    rows, pos = moe.routed_rows(_pad(h, Dp).to(dtype).to(DEV), idx, rw, ew, False)
    got = (rw.unsqueeze(-1) * rows[pos.long()][..., :D]).sum(1)
    assert _rel(got, want) < tol


# ---------------------------------------------------------------- HGRN2
@pytest.mark.parametrize("heads,d,dv", [(3, 20, 28), (1, 128, 128), (2, 64, 64), (5, 8, 136), (2, 152, 40), (4, 32, 8), (1, 300, 72)])
def test_hgrn2_prompts_pieces_and_decoding(heads, d, dv):
    from batchgen_b200.ops import _ext, recurrent
    g = _gen(d + dv)
    dp, dvp = _up(d), _up(dv)
    lens = [37, 1, 90, 8]
    T = sum(lens)
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    q, z, v = 1.5 * r(T, heads, d), 4 * r(T, heads, d), r(T, heads, dv)
    bias, low, nw = r(heads, d), torch.rand(heads, d, generator=g), 1 + 0.2 * r(dv)
    low[0, 0], low[-1, -1] = 0.0, 0.9999                       # a channel that may forget at once, one that hardly forgets
    z[:, 0, 0] -= 30
    S0 = r(len(lens), heads, d, dv)
    want, S1 = [], []
    for i, (a, n) in enumerate(zip([0, 37, 38, 128], lens)):
        f = oracle.forget(z[a:a + n].double() + bias, low.double())
        o, S = oracle.hgrn2(oracle.silu(q[a:a + n].double()), f, v[a:a + n].double(), S0[i].double())
        want.append((oracle.rms(o, 1e-5) * nw).flatten(1))
        S1.append(S)
    want = torch.cat(want)
    head = lambda t, w: _pad(t, w).flatten(-2)      # noqa: E731
    vec = lambda t: head(t, dp).reshape(-1).contiguous().to(DEV)      # noqa: E731
    p = recurrent.RecurrentParams("hgrn2", heads, dp, dv, dvp, _pad(nw, dvp).repeat(heads).to(DEV), 1e-5, f_bias=vec(bias), f_lower=vec(low))
    cols = torch.cat([head(q, dp), head(z, dp), head(v, dvp)], 1).to(DEV)
    n = heads * dp
    slots = [4, 0, 2, 5]

    def pool():
        t = torch.zeros(7, heads * dp * dvp + 12, device=DEV)[:, :heads * dp * dvp]
        for i, s in enumerate(slots):
            t[s] = F.pad(S0[i], (0, dvp - dv, 0, dp - d)).reshape(-1).to(DEV)
        t[6] = 3.0
        return t

    def run(st, rows, cu, sl, init=None):
        x = cols[rows]
        out = torch.full((x.shape[0], heads * dvp), 5.0, device=DEV)
        recurrent.recurrent_forward(p, x[:, :n], x[:, n:2 * n], x[:, 2 * n:], None, {"S": st}, _i32(sl), out, cu, None, init)
        return out.view(-1, heads, dvp)[..., :dv].flatten(1)

    def states(st):
        return torch.stack([st[s].view(heads, dp, dvp)[:, :d, :dv] for s in slots])
    st = pool()
    got = run(st, torch.arange(T), _i32([0, 37, 38, 128, 136]), slots, _i32([1] * 4))
    assert _rel(got, want) < 2e-5 and _rel(states(st), torch.stack(S1)) < 2e-6 and float((st[6] - 3).abs().max()) == 0
    # pieces, then single tokens through the decode kernel, one row without a slot
    st = pool()
    outs = [[], [], [], []]
    first = [20, 0, 61, 2]
    rows = torch.cat([torch.arange(a, a + k) for a, k in zip((0, 37, 38, 128), first)])
    got = run(st, rows, _i32([0, 20, 20, 81, 83]), slots, _i32([1] * 4))
    for i, x in enumerate(got.split(first)):
        outs[i].append(x)
    at = list(first)
    while any(a < m for a, m in zip(at, lens)):
        live = [i for i in range(4) if at[i] < lens[i]]
        rows = torch.tensor([(0, 37, 38, 128)[i] + at[i] for i in live] + [0])
        got = run(st, rows, None, [slots[i] for i in live] + [-1])
        assert float(got[-1].abs().max()) == 0
        for k, i in enumerate(live):
            outs[i].append(got[k:k + 1])
            at[i] += 1
    assert _rel(torch.cat([torch.cat(o) for o in outs]), want) < 2e-5 and _rel(states(st), torch.stack(S1)) < 2e-6
    # a sequence that starts: what the slot held before does not count
    st = pool()
    got = run(st, torch.arange(37), _i32([0, 37]), [4], _i32([0]))
    f = oracle.forget(z[:37].double() + bias, low.double())
    o, _ = oracle.hgrn2(oracle.silu(q[:37].double()), f, v[:37].double())
    assert _rel(got, (oracle.rms(o, 1e-5) * nw).flatten(1)) < 2e-5
    _ext.check_status()


# ---------------------------------------------------------------- attention
class _Pages:
    """Cache pages of several sequences in a random order, with stale numbers in them."""

    def __init__(self, lens, page, row, dtype, g):
        self.T, self.lens = sum(lens), lens
        n_pages = sum(-(-n // page) for n in lens) + 3
        order = torch.randperm(n_pages, generator=g).tolist()
        self.pool = torch.randn(n_pages, page, row, generator=g).to(dtype).to(DEV)
        bt = torch.zeros(len(lens), max(-(-n // page) for n in lens) + 1, dtype=torch.int32)
        slots, used = [], 0
        for i, n in enumerate(lens):
            need = -(-n // page)
            bt[i, :need] = torch.tensor(order[used:used + need])
            slots += [int(bt[i, t // page]) * page + t % page for t in range(n)]
            used += need
        self.bt, self.slots = bt.to(DEV), torch.tensor(slots, device=DEV)
        self.seq = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32).to(DEV)
        self.pos = torch.cat([torch.arange(n) for n in lens])
        self.lens_t = (self.pos + 1).to(torch.int32).to(DEV)
        self.cu = [sum(lens[:i]) for i in range(len(lens) + 1)]


class _Attention(_Pages):
    """Random heads through bias, norm over all of them and cache, and the plain form's outputs."""

    def __init__(self, lens, H, G, d, dv, window, page, dtype, seed=0, edit=None, rot=0, interleaved=False):
        from batchgen_b200.ops import talking
        from batchgen_b200.ops.conv import Rotary, rotate_ref
        g = _gen(seed)
        r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
        dp, dvp = _up(d), _up(dv)
        super().__init__(lens, page, G * (dp + dvp), dtype, g)
        self.H, self.dv, self.sinks = H, dv, 2 * r(H)
        self.p = talking.TalkParams(H, G, dp, dvp, (4.5 if edit else 1.1) * d ** -0.5, window=window, sinks=self.sinks.to(DEV), gate_all=True)
        qs, ks, vs = ([r(n, h, w) for n in lens] for h, w in ((H, d), (G, d), (G, dv)))
        b = [0.5 * r(h, w) * (edit is None) for h, w in ((H, d), (G, d), (G, dv))]
        wq, wk = 1 + 0.2 * r(H, d), 1 + 0.2 * r(G, d)
        self.gates = [r(n, H, dv) for n in lens]
        if edit:
            edit(qs, ks, vs)
        flat = lambda *xs: torch.cat([_pad(x, _up(x.shape[-1])).flatten(-2) for x in xs], -1)      # noqa: E731
        self.prep = talking.HeadPrep(d, 1e-5, flat(*b).to(DEV), flat(wq).to(DEV), flat(wk).to(DEV), interleaved, True)
        self.rope = Rotary.make(rot, 200.0, DEV, interleaved).table(self.lens_t) if rot else None
        self.z = torch.cat([torch.zeros(self.T, 8), torch.cat([flat(*x) for x in zip(qs, ks, vs)]), torch.full((self.T, 4), 9.0)], 1)
        self.gate = torch.cat([flat(x) for x in self.gates]).to(DEV)
        self.want, self.q = [], []
        for i, (q, k, v) in enumerate(zip(qs, ks, vs)):
            q, k, v = (x.double() + y for x, y in zip((q, k, v), b))
            q, k = (oracle.rms(x.flatten(1), 1e-5).view_as(x) * y for x, y in ((q, wq), (k, wk)))
            if rot:
                tab = Rotary.make(rot, 200.0, "cpu", interleaved).table(torch.arange(1, len(q) + 1)).double()
                q, k = rotate_ref(q, tab, interleaved), rotate_ref(k, tab, interleaved)
            o = oracle.attention(q, k, v, self.p.scale, oracle.visible(len(q), window), self.sinks.double())
            self.want.append(o * torch.sigmoid(self.gates[i].double()))
            self.q.append(q)

    def prepare(self, operand, write_q=True):
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


SHAPES = [(9, 3, 56, 48, 64, 64), (4, 4, 20, 36, 16, 33), (8, 1, 80, 128, 64, 100), (32, 8, 128, 128, 64, 128), (1, 1, 8, 8, 32, 1),
          (16, 2, 40, 200, 128, 17), (10, 2, 96, 24, 64, 250), (6, 2, 136, 264, 64, 90), (2, 1, 384, 40, 64, 65), (12, 12, 8, 250, 32, 40),
          (20, 4, 128, 64, 64, 700), (40, 2, 120, 88, 16, 75), (24, 2, 64, 192, 64, 130)]


@pytest.mark.parametrize("H,G,d,dv,page,window", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF])
def test_attention_with_sinks_and_gates_per_element(H, G, d, dv, page, window, dtype):
    from batchgen_b200.ops import _ext, talking
    lens = [150, 33, 1, 300]
    tol = 2e-2 if dtype == BF else 2e-5
    a = _Attention(lens, H, G, d, dv, window, page, dtype, H + d)
    p, full = a.p, torch.cat(a.want)
    tiles = talking.prefill_supported(p, dtype, page)
    q, qf = a.prepare(tiles)
    if qf is not None:
        assert _rel(qf[..., :d], torch.cat(a.q) * p.scale * 1.4426950408889634) < 5e-3 and float(qf[..., d:].abs().sum()) == 0
    assert _rel(q.view(a.T, H, p.dim_p)[..., :d], torch.cat(a.q)) < 2e-6
    for splits in (1, 3, 0):
        out = a.out(dtype)
        talking.attend_rows(q, p, a.pool, a.bt, a.lens_t, out, a.seq, num_splits=splits, gate=a.gate)
        assert _rel(a.heads(out), full) < tol, splits
    some = [3, 450, 180]
    out = a.out(dtype)
    talking.attend_rows(q, p, a.pool, a.bt, a.lens_t, out, a.seq[torch.tensor(some)].contiguous(), _i32(some), num_splits=2, gate=a.gate)
    assert _rel(a.heads(out)[some], full[some]) < tol and float((out[4] - 5).abs().sum()) == 0
    if tiles:
        out = a.out(dtype)
        blocks = talking.work_blocks(talking.prefill_work(a.cu, [0] * 4, 0, 1, window), a.T, DEV)
        talking.attend_prefill(q, p, a.pool, a.bt, out, blocks, operand=qf, gate=a.gate)
        assert _rel(a.heads(out), full) < tol
        for n in (1, 70, 260):                                        # pieces of their own, cached keys before them
            out = a.out(dtype)
            talking.attend_prefill(q, p, a.pool, a.bt[3:4].contiguous(), out, talking.work_blocks(
                [(a.T - n + i, min(128, n - i), 0, 300 - n + i) for i in range(0, n, 128)], a.T, DEV), operand=qf, gate=a.gate)
            assert _rel(a.heads(out)[-n:], full[-n:]) < tol and float((out[: a.T - n] - 5).abs().sum()) == 0
    _ext.check_status()


@pytest.mark.parametrize("rot,interleaved", [(8, False), (8, True), (24, False), (24, True)])
def test_norms_over_all_heads_before_a_rotation(rot, interleaved):
    """The same kernel for heads as other designs may have them."""
    a = _Attention([40, 7], 5, 5, 24, 16, 0, 16, F32, 3, rot=rot, interleaved=interleaved)
    q, qf = a.prepare(True, False)
    assert _rel(q, a.z[:, 8:8 + 5 * 24]) == 0                        # left alone
    assert _rel(qf[..., :24], torch.cat(a.q) * a.p.scale * 1.4426950408889634) < 5e-3
    q, _ = a.prepare(False)
    assert _rel(q.view(-1, 5, 24), torch.cat(a.q)) < 2e-6


class _Latents(_Pages):
    """Random latents of several sequences and queries of their heads; the plain form's outputs."""

    def __init__(self, lens, H, d, rd, dv, rank, window, page, dtype, seed=0, edit=None, sinks=None):
        from batchgen_b200.config import ModelConfig, pitudra_config
        from batchgen_b200.models.mixers import build_mixer
        from batchgen_b200.models.weights import WeightSource
        g = _gen(seed)
        r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
        cfg = pitudra_config(pm.config(32, 64, [pm.latent(H, d, rd, dv, 24, rank, window, base=90.0, scale=(d + rd) ** -0.5)]))
        assert isinstance(cfg, ModelConfig)
        w = oracle.random_weights(pm.config(32, 64, [pm.latent(H, d, rd, dv, 24, rank, window)]), seed)
        if sinks is not None:
            w["l0.mix.sink"] = torch.full((H,), sinks)
        cq, z = [r(n, 24) for n in lens], [r(n, rank + rd) for n in lens]
        qs = [r(n, H, d + rd) for n in lens]
        if edit:
            edit(qs, z, w)
        self.mx = build_mixer(cfg.layer_specs[0].mixer, "l0.mix.", WeightSource(device=DEV, loader=lambda n, s: w.get(n)), cfg, dtype)
        self.p, self.H, self.dv = self.mx.lat, H, dv
        super().__init__(lens, page, self.p.row, dtype, g)
        self.rope = self.mx.rot.table(self.lens_t)
        parts = [torch.cat(x) for x in (cq, z)]
        self.z = torch.cat([torch.zeros(self.T, 8), parts[0], _pad(parts[1][:, :rank], _up(rank)), _pad(parts[1][:, rank:], _up(rd))], 1).to(DEV)
        self.cols = (8, 32, 32 + _up(rank))
        flat = torch.cat(qs)
        self.q = torch.cat([_pad(flat[..., d:], _up(rd)), _pad(flat[..., :d], _up(d))], -1).flatten(1).to(DEV)
        self.operand = torch.cat([oracle.rms(x.double(), 1e-5) * w["l0.mix.dq.norm"] for x in cq])
        self.rows, self.want = [], []
        wd = {k[7:]: v.double() for k, v in w.items()}
        for q, x in zip(qs, z):
            x = x.double()
            c, kr = oracle.rms(x[:, :rank], 1e-5) * wd["dkv.norm"], oracle.rotate(x[:, rank:], 90.0)
            n, q = len(x), q.double()
            q = torch.cat([q[..., :d], oracle.rotate(q[..., d:], 90.0)], -1)
            k = torch.cat([(c @ wd["uk"].T).view(n, H, d), kr.unsqueeze(1).expand(n, H, rd)], -1)
            v = (c @ wd["uv"].T).view(n, H, dv)
            self.rows.append(torch.cat([c, kr], 1))
            self.want.append(oracle.attention(q, k, v, (d + rd) ** -0.5, oracle.visible(n, window), wd["sink"]))

    def prepare(self, dtype):
        from batchgen_b200.ops import latent
        return latent.prepare(self.z, self.cols, self.slots, self.pool, self.p, self.rope, dtype)

    def in_latent_space(self, dtype, rows=None, splits=0):
        from batchgen_b200.ops import latent
        qa = latent.queries(self.q, self.p, self.rope, rows, dtype)
        lens, seq = (self.lens_t, self.seq) if rows is None else (self.lens_t[rows.long()], self.seq[rows.long()])
        o = latent.attend(qa, self.p, self.pool, self.bt, lens.contiguous(), seq.contiguous(), splits)
        out = torch.full((qa.shape[0], self.H * self.p.vdim_p + 8), 5.0, dtype=dtype, device=DEV)
        latent.head_product(o, self.p.w_uv, out[:, 8:].unflatten(1, (self.H, self.p.vdim_p)))
        assert float((out[:, :8] - 5).abs().sum()) == 0
        return out[:, 8:].unflatten(1, (self.H, self.p.vdim_p))[..., :self.dv]

    def expanded(self, cu, ctx, bt, first):
        """Pieces cu[i] .. cu[i + 1] of the rows from ``first`` on."""
        from batchgen_b200.ops import latent
        out = torch.full((self.T, self.H * self.p.vdim_p), 5.0, dtype=BF, device=DEV)
        groups = latent.expansions(cu, ctx, self.p.window, self.pool.shape[1], DEV)
        latent.attend_prompt(self.q[first:], self.p, self.pool, bt, self.rope[first:], out[first:], groups)
        return out.view(self.T, self.H, self.p.vdim_p)[..., :self.dv]


#          heads, dim, rotated, value, rank, window, page
LATENTS = [(5, 20, 6, 12, 50, 37, 64), (1, 8, 2, 8, 8, 1, 16), (32, 128, 64, 128, 512, 128, 64), (16, 16, 16, 24, 200, 100, 64),
           (17, 24, 8, 16, 96, 33, 16), (40, 16, 16, 32, 256, 300, 32), (3, 200, 56, 256, 120, 90, 64), (20, 32, 32, 40, 400, 200, 128),
           (35, 8, 72, 16, 584, 64, 64), (8, 300, 20, 264, 72, 50, 64), (64, 12, 126, 20, 510, 150, 64), (2, 9, 128, 9, 509, 0, 64)]


@pytest.mark.parametrize("H,d,rd,dv,rank,window,page", LATENTS)
@pytest.mark.parametrize("dtype", [F32, BF])
def test_latents_in_latent_space_and_expanded(H, d, rd, dv, rank, window, page, dtype):
    from batchgen_b200.ops import _ext, latent, talking
    lens = [150, 33, 1, 300]
    tol = 2e-2 if dtype == BF else 2e-5
    a = _Latents(lens, H, d, rd, dv, rank, window, page, dtype, H + d)
    p, full = a.p, torch.cat(a.want)
    op = a.prepare(dtype)
    assert _rel(op[:, :24], a.operand) < (5e-3 if dtype == BF else 2e-6) and float(op[:, 24:].abs().sum()) == 0
    got = a.pool.flatten(0, 1)[a.slots]
    assert _rel(torch.cat([got[:, :rank], got[:, p.rank_p:p.rank_p + rd]], 1), torch.cat(a.rows)) < (5e-3 if dtype == BF else 2e-6)
    assert float(got[:, rank:p.rank_p].abs().sum()) == 0 and float(got[:, p.rank_p + rd:].abs().sum()) == 0
    for splits in (1, 3, 0):
        assert _rel(a.in_latent_space(dtype, None, splits), full) < tol, splits
    some = [3, 450, 180, 0]
    assert _rel(a.in_latent_space(dtype, _i32(some), 2), full[some]) < tol
    if latent.prompt_supported(p, dtype, page):
        least = talking.PREFILL_MIN_TOKENS
        out = a.expanded(a.cu, [0] * 4, a.bt, 0)
        long = torch.cat([torch.full((n,), n >= least) for n in lens])
        assert _rel(out[long], full[long]) < tol and float((out[~long] - 5).abs().sum()) == 0
        for n in (32, 70, 260):                                       # pieces of their own, cached keys before them
            out = a.expanded([0, n], [300 - n], a.bt[3:4].contiguous(), a.T - n)
            assert _rel(out[-n:], full[-n:]) < tol, n
    _ext.check_status()


def test_a_group_of_expanded_pages_at_a_time(monkeypatch):
    from batchgen_b200.ops import latent
    a = _Latents([150, 40, 90, 300], 4, 24, 8, 32, 64, 70, 64, BF, 2)
    a.prepare(BF)
    for most, groups in ((1, 4), (300, 3), (10_000, 1)):
        monkeypatch.setattr(latent, "EXPAND_TOKENS", most)
        assert len(latent.expansions(a.cu, [0] * 4, 70, 64, DEV)) == groups
        assert _rel(a.expanded(a.cu, [0] * 4, a.bt, 0), torch.cat(a.want)) < 2e-2


@pytest.mark.parametrize("window", [70, 64, 1, 130, 300, 33])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_one_outstanding_key_at_every_kind_of_place(dtype, window):
    """The query asks for exactly one key (its score stands far out): the window's first key, the ones before and after it, page and
    tile borders, its neighbour, itself, the next token; plain heads and latents."""
    from batchgen_b200.ops import _ext, latent, talking
    n, H, G, d, dv, i = 330, 4, 2, 16, 16, 320
    edge = i - window
    for j in sorted(x for x in {0, 1, edge - 1, edge, edge + 1, edge + 2, 63, 64, 255, 256, 319, 320, i - 1, i, i + 1, i - 31, i - 32} if 0 <= x < n):
        def edit(qs, ks, vs):
            qs[0][i], ks[0][:, :, 12:] = 0.01, 0.0
            qs[0][i, :, 12:] = 8.0
            ks[0][j] *= 0.01
            ks[0][j, :, 12:] = 14.0
            vs[0][j] += 50.0
        seen = edge < j <= i
        a = _Attention([n], H, G, d, dv, window, 64, dtype, j, edit)
        # (a gate per element scales the answer: its spread tells)
        assert (float(a.want[0][i].abs().mean()) > 10) == seen, j
        q, qf = a.prepare(dtype == BF)
        outs = []
        for splits in (1, 4):
            outs.append(a.out(dtype))
            talking.attend_rows(q, a.p, a.pool, a.bt, a.lens_t, outs[-1], a.seq, num_splits=splits, gate=a.gate)
        if dtype == BF:
            for cut in ([0, n], [0, i - 1, n], [0, 257, n]):                # the query's place in its tile differs
                outs.append(a.out(dtype))
                work = [(w[0] + s, w[1], 0, w[3]) for s, e in zip(cut, cut[1:]) for w in talking.prefill_work([0, e - s], [s], 0, 1, window)]
                talking.attend_prefill(q, a.p, a.pool, a.bt, outs[-1], talking.work_blocks(work, n, DEV), operand=qf, gate=a.gate)
        for out in outs:
            assert _rel(a.heads(out)[i], a.want[0][i]) < (3e-2 if dtype == BF else 1e-4), (j, seen)

        def edit(qs, z, w):                                               # the first latent channel asks and answers
            w["l0.mix.uk"][:, 0] = 2.0
            w["l0.mix.uv"][:, 0] = 3.0
            w["l0.mix.dkv.norm"][0] = 1.0
            z[0][:, 0], z[0][j] = 0.0, 0.02 * z[0][j]
            z[0][j, 0] = 1.0
            qs[0][i, :, :16], qs[0][i, :, 16:] = 1.0, 0.0
        for sinks, answers in ((None, seen), (400.0, False)):
            b = _Latents([n], H, 16, 8, dv, 40, window, 64, dtype, j, edit, sinks)
            assert (float(b.want[0][i].mean()) > 10) == answers, (j, sinks)
            b.prepare(dtype)
            outs = [b.in_latent_space(dtype, None, s) for s in (1, 4)]
            if dtype == BF:
                for s in (0, i - 40, 257):
                    outs.append(b.expanded([0, n - s], [s], b.bt, s))
            for out in outs:
                diff = (out[i].double().cpu() - b.want[0][i]).abs().max()
                assert float(diff) < (0.03 if dtype == BF else 1e-4) * (1 + float(b.want[0][i].abs().max())), (j, sinks)
    _ext.check_status()


# ---------------------------------------------------------------- models
TOL = [("fp32", 1e-4), ("bf16", 6e-2)]


def _close(got, want, tol, d):
    """In 32 bits every row within ``tol``.  In 16 bits single rows stand out (a narrow head whose output nearly cancels is blown up
    by its norm), and a close choice of experts may flip, after which states carry the difference on."""
    e = pm.row_errors(got, want)
    if tol < 1e-3:
        return bool(e.max() < tol)
    if any(l["mlp"] and l["mlp"]["router"]["top"] < l["mlp"]["router"]["experts"] for l in d["layers"]):
        return bool((e > tol).double().mean() <= 0.15 and e.median() < tol / 2)
    return bool(e.max() < 4 * tol and e.mean() < tol / 2)


def _weights(d, seed, dtype):
    return pm.weights_of(d, seed, settled=dtype == "bf16")


@pytest.mark.parametrize("dtype,tol", TOL)
@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name, dtype, tol):
    from batchgen_b200.ops import _ext
    d = pm.CONFIGS[name]
    w = _weights(d, 11, dtype)
    toks = pm.prompt(d, 200)
    want = oracle.forward(d, w, toks, F64)
    eng = pm.engine(pm.build(d, w, DEV, dtype))
    for sizes in ([200], [2], [150, 1], [63, 1, 2, 40, 5], [64]):
        s = eng.open_sequence()
        got = pm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert _close(got, want, tol, d), (sizes, pm.row_errors(got, want).sort()[0][-40:])
    _ext.check_status()
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("seed", range(10, 26))
def test_random_designs(seed):
    d = pm.random_config(seed)
    toks = pm.prompt(d, 140)
    for dtype, tol in TOL:
        w = _weights(d, seed, dtype)
        want = oracle.forward(d, w, toks, F64)
        eng = pm.engine(pm.build(d, w, DEV, dtype))
        for sizes in ([140], [37, 2, 1]):
            got = pm.run_pieces(eng, eng.open_sequence(), toks, sizes)
            assert _close(got, want, tol, d), (dtype, sizes, pm.row_errors(got, want).sort()[0][-40:])


@pytest.mark.parametrize("dtype,tol", TOL)
def test_mixed_batches_equal_each_request_alone(dtype, tol):
    d = pm.CONFIGS["odd"] if dtype == "fp32" else pm.without_choices(pm.CONFIGS["odd"])
    w = pm.weights_of(d, seed=12)
    eng = pm.engine(pm.build(d, w, DEV, dtype), tokens=64 * 12)
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((260, 41, 130, 64, 3, 90, 1))]
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
    d = pm.config(150, 64, [pm.latent(4, 16, 8, 24, 32, 48, 700, pm.moe(32, 2, 2), 1e4), pm.hgrn2(2, 16, 16), pm.attention(4, 2, 16, 24, 100),
                            pm.latent(3, 24, 8, 16, 24, 48, 65, base=1e4, kv_from=0)], 16)
    w = pm.weights_of(d, seed=15)
    toks = pm.prompt(d, 1000)
    want = oracle.forward(d, w, toks, F64)
    eng = pm.engine(pm.build(d, w, DEV, dtype), tokens=1024 + 64)
    for sizes in ([1000], [930, 1], [333]):
        s = eng.open_sequence()
        got = pm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert _close(got, want, tol, d), (sizes, pm.error(got, want))


def test_greedy_generation_in_32_bit_and_long_decoding():
    from batchgen_b200.runtime.sequence import SamplingParams
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=13)
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((90, 7, 40))]
    eng = pm.engine(pm.build(d, w, DEV, "fp32"), tokens=64 * 64)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=120, ignore_eos=True))
    for p, o in zip(prompts, outs):
        logits = oracle.forward(d, w, p + o, F64)[len(p) - 1:-1]
        assert len(o) == 120 and logits.argmax(-1).tolist() == o


@pytest.mark.parametrize("name", ["whole", "latents"])
def test_captured_decode_steps_equal_eager_ones(name):
    from batchgen_b200.runtime.graphs import DecodeGraphRunner
    from batchgen_b200.runtime.sequence import SamplingParams
    d = pm.CONFIGS[name]
    w = pm.weights_of(d, seed=14)
    model = pm.build(d, w, DEV, "bf16")
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((70, 9, 130, 33, 5))]
    params = SamplingParams(max_new_tokens=40, ignore_eos=True)
    eager = pm.engine(model, tokens=64 * 40, slots=8).generate(prompts, params)
    eng = pm.engine(model, tokens=64 * 40, slots=8)
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
    model = build_model(get_model_config("tiny-pitudra"), device=DEV, dtype="bf16", seed=1)
    eng = pm.engine(model, tokens=64 * 40, slots=4)
    outs = eng.generate([[1, 2, 3], [5] * 70], [SamplingParams(max_new_tokens=9, temperature=0.8, top_k=20),
                                               SamplingParams(max_new_tokens=5)])
    assert [len(o) for o in outs] == [9, 5]
