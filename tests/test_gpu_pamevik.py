"""Pamevik kernels and models on the GPU against the plain implementation, in bf16 and in true fp32."""
import pytest
import torch
import torch.nn.functional as F

import pamevik_models as pm
import pamevik_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-30))


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------- row operators
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,D", [(5, 100), (3, 1030), (9, 2307), (2, 5001), (2, 8200), (1, 6)])
def test_sandwich_norm_with_every_addend(T, D, dtype):
    from batchgen_b200.ops import residual
    g = _gen(T + D)
    D4, cols = -(-D // 4) * 4, -(-D // 64) * 64
    tol = 5e-3 if dtype == BF else 2e-6

    def vec(mean=0.0):
        return mean + 0.2 * torch.randn(D, generator=g)
    x, a, b = (torch.randn(T, D4, generator=g) * s + 0.5 for s in (1.0, 3.0, 0.2))
    w1, b1, w2, b2, wa, wb = vec(1), vec(), vec(1), vec(), vec(1), vec(1)
    pad = lambda v: F.pad(v, (0, D4 - D)).to(DEV)      # noqa: E731
    n1, n2 = residual.Norm(pad(w1), pad(b1), True), residual.Norm(pad(w2), pad(b2), True)
    for second in (False, True):
        s = a[:, :D].double()
        if second:
            s = 0.5 * (oracle.rms(s, 1e-5) * wa + oracle.rms(b[:, :D].double(), 1e-5) * wb)
        want = x[:, :D].double() + oracle.layer_norm(s, w1, b1, 1e-5)
        xd = x.to(DEV)
        more = dict(add2=b.to(DEV), branch_w=(pad(wa), pad(wb))) if second else {}
        y = residual.sandwich_norm(xd, n2, 1e-5, D, cols, dtype, add=a.to(DEV), post=n1, **more)
        assert _rel(xd[:, :D], want) < 2e-6
        assert _rel(y[:, :D], oracle.layer_norm(want, w2, b2, 1e-5)) < tol and float(y[:, D:].abs().sum()) == 0
        raw = residual.sandwich_norm(xd, n2, 1e-5, D, cols, dtype, raw=True)
        assert raw.dtype == F32 and _rel(raw[:, :D], oracle.layer_norm(want, w2, b2, 1e-5)) < 2e-6
        assert float(raw[:, D:].abs().sum()) == 0
    emb = torch.randn(11, D, generator=g).to(dtype)
    ids = torch.randint(0, 11, (T,), generator=g).to(torch.int32)
    residual.sandwich_norm(xd, n2, 1e-5, D, cols, dtype, ids=ids.to(DEV), embed=emb.to(DEV))
    assert torch.equal(xd[:, :D].cpu(), emb[ids.long()].float())
    rows = torch.tensor([T - 1, 0, T - 1])
    before = xd.clone()
    rms_norm = residual.Norm(pad(w2))                        # neither mean nor bias
    y = residual.sandwich_norm(xd, rms_norm, 1e-5, D, cols, dtype, add=a.to(DEV), post=residual.Norm(pad(w1)), rows=rows.to(DEV),
                               keep=False)
    assert torch.equal(before, xd)
    want = before.cpu()[:, :D].double() + oracle.rms(a[:, :D].double(), 1e-5) * w1
    assert _rel(y[:, :D], (oracle.rms(want, 1e-5) * w2)[rows]) < tol


def test_squared_relu():
    from batchgen_b200.ops import residual
    z = torch.randn(7, 40, generator=_gen(1))
    for dtype, tol in ((BF, 5e-3), (F32, 1e-6)):
        y = residual.cast_act(z.to(DEV)[:, :37], 64, dtype, act="relu2")
        assert _rel(y[:, :37], z[:, :37].clamp_min(0) ** 2) < tol and float(y[:, 37:].abs().sum()) == 0


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 6, 9])
@pytest.mark.parametrize("C", [12, 516])
def test_convolution_pieces_steps_and_history(taps, C):
    """Three sequences in pieces of all sizes (shorter than the window too), beside one another, in slots that hold junk; then
    token by token; the decode norm folds the same convolution in."""
    from batchgen_b200.ops import residual
    from batchgen_b200.ops.conv import causal_conv
    g = _gen(taps * 1000 + C)
    n = (90, 41, 60)
    xs = [torch.randn(m, C, generator=g) for m in n]
    w = torch.randn(C, taps, generator=g)
    want = [oracle.causal_conv(x.double(), w.double()) for x in xs]
    wd = w.t().contiguous().to(DEV)
    stride = 8 + (taps - 1) * C
    pool = torch.full((5, stride), 7.0, device=DEV)
    hist = pool[:, 8:]
    slots, at, got = [3, 0, 4], [0, 0, 0], [[], [], []]
    steps = [(33, 1, 2), (1, 2, 1), (2, 5, 17), (3, 0, 1), (40, 20, 3)]
    for sizes in steps:
        live = [i for i in range(3) if sizes[i]]
        cu = [0]
        for i in live:
            cu.append(cu[-1] + sizes[i])
        x = torch.cat([xs[i][at[i]:at[i] + sizes[i]] for i in live]).to(DEV)
        seq = torch.repeat_interleave(torch.arange(len(live)), torch.tensor([sizes[i] for i in live])).to(torch.int32).to(DEV)
        init = _i32([int(at[i] > 0) for i in live])
        args = (_i32(cu), cu, seq, init)
        sl = _i32([slots[i] for i in live])
        kept = pool.clone()
        res = torch.full((cu[-1], C + 12), 5.0, device=DEV)
        causal_conv(x, wd, hist, sl, res[:, :C + 8], "residual", *args)
        assert float((res[:, C + 8:] - 5).abs().sum()) == 0 and float(res[:, C:C + 8].abs().sum()) == 0
        pool.copy_(kept)
        out = torch.empty(cu[-1], C, device=DEV)
        causal_conv(x, wd, hist, sl, out, "silu", *args)
        for j, i in enumerate(live):
            part = want[i][at[i]:at[i] + sizes[i]]
            assert _rel(out[cu[j]:cu[j + 1]], F.silu(part)) < 2e-6, (sizes, i)
            assert _rel(res[cu[j]:cu[j + 1], :C], xs[i][at[i]:at[i] + sizes[i]] + part) < 2e-6
            at[i] += sizes[i]
    norm = residual.Norm(torch.ones(C, device=DEV), torch.zeros(C, device=DEV), True)
    for _ in range(5):                                       # one token each, a padding row among them
        rows = torch.stack([xs[0][at[0]], torch.zeros(C), xs[1][at[1]], xs[2][at[2]]]).to(DEV)
        sl = _i32([slots[0], -1, slots[1], slots[2]])
        kept = pool.clone()
        out = torch.empty(4, C + 4, dtype=BF, device=DEV)
        causal_conv(rows, wd, hist, sl, out, "residual")
        for r, i in ((0, 0), (2, 1), (3, 2)):
            assert _rel(out[r, :C], xs[i][at[i]] + want[i][at[i]]) < 5e-3
        after = pool.clone()
        # the folded form, on inputs that the norm reproduces: its history holds normed rows, so start both from the same one
        pool.copy_(kept)
        y = residual.sandwich_norm(rows.clone(), norm, 1e-5, C, C, F32, canon=residual.Canon(wd, hist, sl))
        h = oracle.layer_norm(rows.double().cpu(), 1.0, 0.0, 1e-5)
        for r, s in ((0, slots[0]), (2, slots[1]), (3, slots[2])):
            past = kept[s, 8:].view(taps - 1, C).double().cpu()
            full = torch.cat([past, h[r:r + 1]])
            assert _rel(y[r], h[r] + (full * w.t().double()).sum(0)) < 2e-6
            if taps > 1:
                assert _rel(pool[s, 8:].view(taps - 1, C), full[1:]) < 2e-6
        pool.copy_(after)
        at = [a + 1 for a in at]
    assert float((pool[:, :8] - 7).abs().sum()) == 0 and float((pool[1] - 7).abs().sum()) == 0


def test_rotary_table_is_exact_far_away():
    from batchgen_b200.ops.conv import Rotary
    for dims, base in ((2, 10.0), (20, 500.0), (128, 1e6)):
        r = Rotary.make(dims, base, DEV)
        pos = torch.tensor([0, 1, 63, 64, 4095, 100_000, 3_000_000])
        got = r.table((pos + 1).to(torch.int32).to(DEV)).double().cpu()
        a = pos.double().unsqueeze(1) * torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
        assert float((got - torch.cat([a.cos(), a.sin()], 1)).abs().max()) < 1e-6


# ---------------------------------------------------------------- recurrences
RULE_SHAPES = [(3, 12, 20, 3), (6, 24, 40, 2), (2, 64, 24, 2), (2, 128, 128, 1), (3, 90, 60, 3), (4, 32, 128, 4), (2, 136, 48, 1),
               (1, 40, 200, 1), (2, 160, 136, 2), (1, 200, 264, 1), (1, 256, 8, 1), (2, 392, 24, 1), (1, 512, 40, 1)]


class _Case:
    """One recurrence's random inputs over ``T`` tokens: the op's padded columns and the plain form's view of them."""

    def __init__(self, rule, H, d, dv, G, T, seed, open_gates=False, const=None):
        from batchgen_b200.ops.conv import Rotary
        from batchgen_b200.ops.recurrent import RecurrentParams
        g = _gen(seed)
        self.rule, self.H, self.d, self.dv, self.G = rule, H, d, dv, G if rule == "channel_delta" else H
        G, dp, dvp = self.G, -(-d // 8) * 8, -(-dv // 8) * 8
        self.dp, self.dvp = dp, dvp
        r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
        self.q, self.k, self.v, self.gate = r(T, G, d), r(T, G, d), r(T, H, dv), r(T, H, dv)
        self.extra = (r(T, H, d) - 2, r(T, H)) if rule == "channel_delta" else (r(T, H), r(T, H) + 3) if rule == "mlstm" else ()
        if open_gates:                                    # states that hardly fade
            self.extra = ((self.extra[0] - 12, self.extra[1]) if rule == "channel_delta"
                          else (self.extra[0], self.extra[1] + 9) if rule == "mlstm" else ())
        c = const or dict(norm=1 + 0.2 * r(H, dv), A=0.5 * r(H), dt=0.5 * r(H, d), bi=0.5 * r(H), bf=0.5 * r(H),
                          decay=1 - 10 ** (-1 - 2 * torch.rand(H, generator=g)) * (1e-3 if open_gates else 1))
        self.c = c
        kw = dict(rule=rule, heads=H, dim_p=dp, vdim=dv, vdim_p=dvp, eps=1e-5, norm_w=self._pad(c["norm"], dvp).reshape(-1).to(DEV))
        if rule == "channel_delta":
            kw.update(q_scale=d ** -0.5, qk_heads=G, rate=c["A"].exp().to(DEV), dt_bias=self._pad(c["dt"], dp).reshape(-1).to(DEV))
        elif rule == "mlstm":
            kw.update(q_scale=d ** -0.5, gate_cap=6.0, i_bias=c["bi"].to(DEV), f_bias=c["bf"].to(DEV))
        else:
            kw.update(k_scale=d ** -0.5, gate="silu", decay=c["decay"].to(DEV))
        self.p = RecurrentParams(**kw)
        self.rot = Rotary.make(d // 4 * 2, 50.0, DEV) if rule == "retention" else None

    @staticmethod
    def _pad(t, w):
        return F.pad(t, (0, w - t.shape[-1]))

    def run(self, rows, pos, state, slots, out, **where):
        from batchgen_b200.ops.recurrent import recurrent_forward
        q, k = (self._pad(t[rows], self.dp).reshape(len(rows), -1) for t in (self.q, self.k))
        v, gate = (self._pad(t[rows], self.dvp).reshape(len(rows), -1) for t in (self.v, self.gate))
        z = torch.cat([q, k, v, gate], 1).to(DEV)          # one stacked projection, read through column views
        a, b, n = q.shape[1], q.shape[1] * 2, v.shape[1]
        more = {}
        if self.rule == "channel_delta":
            more = dict(low=self._pad(self.extra[0][rows], self.dp).reshape(len(rows), -1).to(DEV), beta=self.extra[1][rows].to(DEV))
        elif self.rule == "mlstm":
            more = dict(gate_i=self.extra[0][rows].to(DEV), gate_f=self.extra[1][rows].to(DEV))
        elif self.rot is not None:
            more = dict(rope=self.rot.table((torch.as_tensor(pos) + 1).to(torch.int32).to(DEV)))
        recurrent_forward(self.p, z[:, :a], z[:, a:b], z[:, b:b + n], z[:, b + n:], state, slots, out, **where, **more)

    def plain(self, rows, pos, state=None):
        """(gated outputs [n, H, dv], state) of rows at positions ``pos`` of one sequence."""
        D = torch.float64
        q, k, v = (t[rows].to(D) for t in (self.q, self.k, self.v))
        c = {n: t.to(D) for n, t in self.c.items()}
        act = torch.sigmoid
        if self.rule == "channel_delta":
            rep = self.H // self.G
            q, k = oracle.unit(q).repeat_interleave(rep, 1) * self.d ** -0.5, oracle.unit(k).repeat_interleave(rep, 1)
            g = torch.exp(-c["A"].exp().view(1, -1, 1) * F.softplus(self.extra[0][rows].to(D) + c["dt"]))
            o, state = oracle.gated_delta(q, k, v, g, torch.sigmoid(self.extra[1][rows].to(D)), state)
        elif self.rule == "mlstm":
            i = 6.0 * torch.tanh((self.extra[0][rows].to(D) + c["bi"]) / 6.0)
            f = F.logsigmoid(6.0 * torch.tanh((self.extra[1][rows].to(D) + c["bf"]) / 6.0))
            o, state = oracle.mlstm(q * self.d ** -0.5, k, v, i, f, state)
        else:
            # positions beside one another in the plain rotation: turn a whole sequence's worth and pick
            n = max(pos) + 1
            turn = lambda t: oracle.rotate(torch.zeros(n, *t.shape[1:], dtype=D).index_copy(0, torch.as_tensor(pos), t), 50.0,   # noqa: E731
                                           self.d // 4 * 2)[torch.as_tensor(pos)] if self.rot is not None else t
            o, state = oracle.retention(turn(q), turn(k) * self.d ** -0.5, v, c["decay"], state)
            act = F.silu
        return oracle.rms(o, 1e-5) * c["norm"] * act(self.gate[rows].to(D)), state

    def pools(self, slots):
        """Pools that hold what others left there, each with columns of something else in front."""
        shapes = {"S": self.H * self.dp * self.dvp}
        if self.rule == "mlstm":
            shapes.update(n=self.H * self.dp, m=self.H)
        row = sum(-(-x // 4) * 4 for x in shapes.values()) + 8
        pool, at, views = torch.full((slots, row), 7.0, device=DEV), 8, {}
        for name, x in shapes.items():
            views[name] = pool[:, at:at + x]
            at += -(-x // 4) * 4
        return pool, views

    def state_error(self, views, slot, state):
        if self.rule != "mlstm":
            return _rel(views["S"][slot].view(self.H, self.dp, self.dvp)[:, :self.d, :self.dv], state)
        S, n, m = state                                       # the running maximum's rounding scales S and n alike
        f = torch.exp(views["m"][slot].double().cpu() - m)
        assert float((f - 1).abs().max()) < 1e-4
        return max(_rel(views["S"][slot].view(self.H, self.dp, self.dvp)[:, :self.d, :self.dv].double().cpu() * f.view(-1, 1, 1), S),
                   _rel(views["n"][slot].view(self.H, self.dp)[:, :self.d].double().cpu() * f.view(-1, 1), n))


@pytest.mark.parametrize("H,d,dv,G", RULE_SHAPES)
@pytest.mark.parametrize("rule", ["channel_delta", "mlstm", "retention"])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_recurrences_prompts_continuations_and_decoding(rule, H, d, dv, G, dtype):
    lens = [37, 1, 2, 100]
    cu = [0, 37, 38, 40, 140]
    c = _Case(rule, H, d, dv, G, 160, H * 1000 + d)
    pool, state = c.pools(6)
    tol = 1e-2 if dtype == BF else 5e-5
    n = c.H * c.dvp
    order = [4, 3, 0, 1]
    pos = [p for m in lens for p in range(m)]
    rows = torch.arange(140)
    out = torch.full((140, n + 64), 5.0, dtype=dtype, device=DEV)
    init = _i32([0, 0, 0, 0])
    c.run(rows, pos, state, _i32(order), out[:, :n], cu=_i32(cu), cu_host=cu, has_initial=init)
    ends = {}
    for i, slot in enumerate(order):
        want, ends[slot] = c.plain(rows[cu[i]:cu[i + 1]], pos[cu[i]:cu[i + 1]])
        got = out[cu[i]:cu[i + 1], :n].view(-1, H, c.dvp)[..., :dv]
        assert _rel(got, want) < tol, i
        assert c.state_error(state, slot, ends[slot]) < 3e-5, i
    assert float((pool[2] - 7).abs().sum()) == 0 and float((pool[:, :8] - 7).abs().sum()) == 0 and float((out[:, n:] - 5).abs().sum()) == 0
    # two sequences go on by a piece while a third has none and a skipped one yields zeros
    cu2 = [0, 3, 5, 5, 9]
    rows2, pos2 = torch.arange(140, 149), [37, 38, 39, 0, 1, 100, 101, 102, 103]
    out2 = torch.full((9, n), 5.0, dtype=dtype, device=DEV)
    c.run(rows2, pos2, state, _i32([4, -1, 0, 1]), out2, cu=_i32(cu2), cu_host=cu2, has_initial=_i32([1, 1, 1, 1]))
    for a, b, slot in ((0, 3, 4), (5, 9, 1)):
        want, ends[slot] = c.plain(rows2[a:b], pos2[a:b], ends[slot])
        assert _rel(out2[a:b].view(-1, H, c.dvp)[..., :dv], want) < tol
        assert c.state_error(state, slot, ends[slot]) < 3e-5
    assert float(out2[3:5].abs().sum()) == 0
    # decoding from there, slots in another order, a padding row
    at = {4: 40, 3: 1, 0: 2, 1: 104}
    for step in range(3):
        slots = [1, -1, 4, 0]
        rows3 = torch.tensor([149 + step * 3, 0, 150 + step * 3, 151 + step * 3])
        pos3 = [at[1], 0, at[4], at[0]]
        out3 = torch.full((4, n), 5.0, dtype=dtype, device=DEV)
        c.run(rows3, pos3, state, _i32(slots), out3)
        for r, slot in enumerate(slots):
            if slot < 0:
                assert float(out3[r].abs().sum()) == 0
                continue
            want, ends[slot] = c.plain(rows3[r:r + 1], [pos3[r]], ends[slot])
            assert _rel(out3[r:r + 1].view(1, H, c.dvp)[..., :dv], want) < tol, (step, r)
            assert c.state_error(state, slot, ends[slot]) < 3e-5
            at[slot] += 1


@pytest.mark.parametrize("rule", ["channel_delta", "mlstm", "retention"])
def test_decoding_over_many_rows_and_steps(rule):
    """More (sequence, head) items than SMs, slots in any order, several steps: the ring of state buffers turns over."""
    B, H, d, dv = 150, 4, 32, 40
    c = _Case(rule, H, d, dv, 2, B, 77)
    perm = torch.randperm(B, generator=_gen(4))
    slots = perm.to(torch.int32)
    slots[5], slots[149] = -1, -1
    pool, state = c.pools(B)
    pool.zero_()
    out = torch.empty(B, H * dv, device=DEV)
    for step in range(5):
        c.run(torch.arange(B), [step] * B, state, slots.to(DEV), out)
    for b in (0, 1, 6, 70, 148):
        rows = torch.full((5,), b)
        want, S = c.plain(rows, list(range(5)))
        assert _rel(out[b].view(H, dv), want[-1]) < 2e-5 and c.state_error(state, int(perm[b]), S) < 1e-5
    assert float(out[[5, 149]].abs().sum()) == 0


@pytest.mark.parametrize("rule", ["channel_delta", "mlstm", "retention"])
def test_a_write_far_back_still_answers(rule):
    """One token writes 50 times more than the others and the states hardly fade; a query for its key 250 tokens later finds it,
    whichever way the tokens were cut."""
    T, H, d, dv, at = 300, 2, 16, 24, 40
    c = _Case(rule, H, d, dv, 2, T, 5, open_gates=True)
    c.rot = None if rule == "retention" else c.rot           # equal keys stay equal
    c.v[at] *= 50.0
    c.q[290] = c.k[at]
    if rule == "channel_delta":
        c.k[at + 1:, :, 0] = 0.0                             # later corrections leave the key's own direction alone
        c.k[at] = 0.0
        c.k[at, :, 0] = 1.0
        c.q[290] = c.k[at]
    want, _ = c.plain(torch.arange(T), list(range(T)))
    c.v[at] /= 50.0
    without, _ = c.plain(torch.arange(T), list(range(T)))
    c.v[at] *= 50.0
    assert _rel(without[290], want[290]) > 0.3
    for cut in ([T], [at + 1, 1, 2, 246, 1], [at, 250], [2] * 150):
        pool, state = c.pools(1)
        out, a = torch.empty(T, H * dv, device=DEV), 0
        for n in cut + [1] * T:
            n = min(n, T - a)
            if n <= 0:
                break
            one = n == 1 and a > 0
            where = {} if one else dict(cu=_i32([0, n]), cu_host=[0, n], has_initial=_i32([int(a > 0)]))
            c.run(torch.arange(a, a + n), list(range(a, a + n)), state, _i32([0]), out[a:a + n], **where)
            a += n
        assert _rel(out[290].view(H, dv), want[290]) < 1e-4 and _rel(out.view(T, H, dv), want) < 5e-5, cut


def test_mlstm_gates_far_from_zero():
    """Input gates that rise and fall over the cap's whole range: the running maximum climbs, holds and decays."""
    T, H = 200, 3
    c = _Case("mlstm", H, 16, 16, 3, T, 8)
    ramp = torch.cat([torch.linspace(-30, 30, 80), torch.linspace(30, -30, 80), torch.full((40,), -30.0)])
    c.extra = (ramp.view(-1, 1) + c.extra[0], 10 * c.extra[1] - 30)
    want, end = c.plain(torch.arange(T), list(range(T)))
    pool, state = c.pools(1)
    out = torch.empty(T, H * 16, device=DEV)
    c.run(torch.arange(150), list(range(150)), state, _i32([0]), out[:150], cu=_i32([0, 150]), cu_host=[0, 150], has_initial=_i32([0]))
    for t in range(150, T):
        c.run(torch.tensor([t]), [t], state, _i32([0]), out[t:t + 1])
    assert _rel(out.view(T, H, 16), want) < 5e-5 and c.state_error(state, 0, end) < 5e-5


# ---------------------------------------------------------------- attention
def _attention_case(lens, H, G, d, dv, rd, page, dtype, seed=0, edit=None):
    from batchgen_b200.ops import talking
    from batchgen_b200.ops.conv import Rotary
    g = _gen(seed)
    dp, dvp = -(-d // 8) * 8, -(-dv // 8) * 8
    pad = lambda t, w: F.pad(t, (0, w - t.shape[-1])).reshape(t.shape[0], -1)      # noqa: E731
    qs, ks, vs = ([torch.randn(n, h, w, generator=g) for n in lens] for h, w in ((H, d), (G, d), (G, dv)))
    gates = [torch.randn(n, H, generator=g) for n in lens]
    if edit:
        edit(qs, ks, vs)
    p = talking.TalkParams(H, G, dp, dvp, 0.9 * d ** -0.5)
    rot = Rotary.make(rd, 200.0, DEV)
    T = sum(lens)
    pos = torch.cat([torch.arange(n) for n in lens])
    rope = rot.table((pos + 1).to(torch.int32).to(DEV))
    n_pages = sum(-(-n // page) for n in lens) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    pool = torch.randn(n_pages, page, p.kv_row + 16, generator=g).to(dtype).to(DEV)[:, :, :p.kv_row].contiguous()
    bt = torch.zeros(len(lens), max(-(-n // page) for n in lens) + 1, dtype=torch.int32)
    slots, used = [], 0
    for i, n in enumerate(lens):
        need = -(-n // page)
        bt[i, :need] = torch.tensor(order[used:used + need])
        slots += [int(bt[i, t // page]) * page + t % page for t in range(n)]
        used += need
    kv = torch.cat([torch.cat([pad(k, dp), pad(v, dvp)], 1) for k, v in zip(ks, vs)]).to(DEV)
    talking.kv_write(kv, torch.tensor(slots, device=DEV), pool, p, rope)
    want = []
    for q, k, v, gt in zip(qs, ks, vs, gates):
        o = oracle.attention(oracle.rotate(q.double(), 200.0, rd), oracle.rotate(k.double(), 200.0, rd), v.double(), p.scale)
        want.append(o * torch.sigmoid(gt.double()).unsqueeze(-1))
    q = torch.cat([pad(x, dp) for x in qs]).to(DEV)
    seq = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32).to(DEV)
    return q, p, pool, bt.to(DEV), want, dict(rope=rope, gate=torch.cat(gates).to(DEV)), (pos + 1).to(torch.int32).to(DEV), seq, T


SHAPES = [(9, 3, 56, 48, 56, 64), (4, 4, 20, 36, 6, 16), (8, 1, 80, 128, 32, 64), (32, 8, 128, 128, 128, 64), (1, 1, 8, 8, 2, 32),
          (16, 2, 40, 200, 24, 128), (10, 2, 96, 24, 96, 64), (6, 2, 136, 264, 60, 64), (2, 1, 384, 40, 128, 64), (12, 12, 8, 512, 8, 32)]


@pytest.mark.parametrize("H,G,d,dv,rd,page", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF])
def test_rotary_gated_attention_rows_and_tiles(H, G, d, dv, rd, page, dtype):
    from batchgen_b200.ops import _ext, talking
    lens = [150, 33, 1, 300]
    q, p, pool, bt, want, more, lens_t, seq, T = _attention_case(lens, H, G, d, dv, rd, page, dtype, seed=H + d)
    full = torch.cat(want)
    tol = 2e-2 if dtype == BF else 2e-5

    def check(out, what, rows=slice(None)):
        got = out[:, : H * p.vdim_p].view(T, H, p.vdim_p)[..., :dv][rows]
        assert _rel(got, full[rows]) < tol, what
    for splits in (1, 3):
        out = torch.full((T, H * p.vdim_p + 8), 5.0, dtype=dtype, device=DEV)
        talking.attend_rows(q, p, pool, bt, lens_t, out[:, : H * p.vdim_p], seq, num_splits=splits, **more)
        check(out, splits)
        assert float((out[:, H * p.vdim_p:] - 5).abs().sum()) == 0
    some = _i32([3, 200, 180])
    out = torch.full((T, H * p.vdim_p), 5.0, dtype=dtype, device=DEV)
    talking.attend_rows(q, p, pool, bt, lens_t, out, seq[some.long()].contiguous(), some, num_splits=2, **more)
    check(out, "subset", [3, 200, 180])
    assert float((out[4] - 5).abs().sum()) == 0
    if not talking.prefill_supported(p, dtype, page):
        return
    cu = [0, 150, 183, 184, 484]
    out = torch.full((T, H * p.vdim_p), 5.0, dtype=dtype, device=DEV)
    talking.attend_prefill(q, p, pool, bt, out, talking.work_blocks(talking.prefill_work(cu, [0] * 4, 0), T, DEV), **more)
    check(out, "tiles")
    out = torch.full((T, H * p.vdim_p), 5.0, dtype=dtype, device=DEV)      # a piece of its own, cached keys before it
    talking.attend_prefill(q, p, pool, bt[3:4].contiguous(), out, talking.work_blocks([(T - 70, 70, 0, 230)], T, DEV), **more)
    check(out, "piece", slice(T - 70, T))
    assert float((out[: T - 70] - 5).abs().sum()) == 0
    _ext.check_status()


@pytest.mark.parametrize("dtype", [F32, BF])
def test_one_outstanding_key_at_every_kind_of_place(dtype):
    """The query asks for exactly one key (its score stands far out): the first token, page borders, its neighbour, itself.  The
    channel that carries the score does not turn."""
    from batchgen_b200.ops import _ext, talking
    n, H, G, d, dv, i = 400, 4, 2, 16, 16, 398
    for j in (0, 1, 63, 64, 127, 128, 319, 320, 383, 384, 397, 398, 399):
        def edit(qs, ks, vs):
            qs[0][i] = 0.0
            qs[0][i, :, 12] = 8.0
            ks[0][:, :, 12] = 0.0
            ks[0][j, :, 12] = 14.0
            vs[0][j] += 50.0
        q, p, pool, bt, want, more, lens_t, seq, T = _attention_case([n], H, G, d, dv, 8, 64, dtype, seed=j, edit=edit)
        seen = j <= i
        assert (float((want[0][i] / torch.sigmoid(more["gate"][i].double().cpu()).unsqueeze(-1)).mean()) > 40) == seen
        outs = []
        for splits in (1, 4):
            out = torch.zeros(n, H * dv, dtype=dtype, device=DEV)
            talking.attend_rows(q, p, pool, bt, lens_t, out, seq, num_splits=splits, **more)
            outs.append(out)
        if dtype == BF:
            out = torch.zeros(n, H * dv, dtype=dtype, device=DEV)
            talking.attend_prefill(q, p, pool, bt, out, talking.work_blocks(talking.prefill_work([0, n], [0], 0), n, DEV), **more)
            outs.append(out)
        for out in outs:
            assert _rel(out[i].view(H, dv), want[0][i]) < (3e-2 if dtype == BF else 1e-4), (j, seen)
    _ext.check_status()


# ---------------------------------------------------------------- models
# worst row; the mean row has to be far better.  A head whose output nearly cancels is blown up by its norm, the smaller the head
# the likelier, so in 16 bits single rows stand out.
TOL = [("fp32", 1e-4), ("bf16", 2e-1)]


@pytest.mark.parametrize("dtype,tol", TOL)
@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_prompts_pieces_and_decoding_match_the_oracle(name, dtype, tol):
    from batchgen_b200.ops import _ext
    d = pm.CONFIGS[name]
    w = pm.weights_of(d, seed=11)
    toks = pm.prompt(d, 230)
    want = oracle.forward(d, w, toks, torch.float64)
    eng = pm.engine(pm.build(d, w, DEV, dtype))
    for sizes in ([230], [2], [150, 1], [63, 1, 2, 40, 5], [64]):
        s = eng.open_sequence()
        got = pm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert pm.error(got, want) < tol and float(pm.row_errors(got, want).mean()) < tol / 6, (sizes, pm.error(got, want))
    _ext.check_status()
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("dtype,tol", TOL)
def test_mixed_batches_equal_each_request_alone(dtype, tol):
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=12)
    eng = pm.engine(pm.build(d, w, DEV, dtype), tokens=64 * 12)
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((260, 41, 130, 64, 3, 90, 1))]
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
        assert pm.error(torch.cat(g), x) < tol
    assert eng.kv.alloc.num_used == 0 and eng.kv.state.num_free == 4


@pytest.mark.parametrize("dtype,tol", [("fp32", 2e-4), ("bf16", 1e-1)])
def test_a_long_prompt_over_many_pages(dtype, tol):
    d = pm.config(150, 64, [pm.channel_delta(2, 1, 16, 24, 4), pm.parallel((4, 2, 16, 24, 16, 1e4), ([0.99, 0.999], 16, 16, 16, 1e4),
                                                                          pm.dense(64)), pm.mlstm(2, 16, 16, 8.0)])
    w = pm.weights_of(d, seed=15)
    toks = pm.prompt(d, 1200)
    want = oracle.forward(d, w, toks, torch.float64)
    eng = pm.engine(pm.build(d, w, DEV, dtype), tokens=1216 + 64)
    for sizes in ([1200], [1100, 1], [333]):
        s = eng.open_sequence()
        got = pm.run_pieces(eng, s, toks, sizes)
        eng.close_sequence(s)
        assert pm.error(got, want) < tol, (sizes, pm.error(got, want))


def test_greedy_generation_in_32_bit_and_long_decoding():
    from batchgen_b200.runtime.sequence import SamplingParams
    d = pm.CONFIGS["odd"]
    w = pm.weights_of(d, seed=13)
    prompts = [pm.prompt(d, n, i) for i, n in enumerate((90, 7, 40))]
    eng = pm.engine(pm.build(d, w, DEV, "fp32"), tokens=64 * 64)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=120, ignore_eos=True))
    for p, o in zip(prompts, outs):
        logits = oracle.forward(d, w, p + o, torch.float64)[len(p) - 1:-1]
        assert len(o) == 120 and logits.argmax(-1).tolist() == o


@pytest.mark.parametrize("name", ["whole", "wide"])
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
            row = oracle.forward(d, w, p + a[:n], torch.float64)[-1]
            assert float((row[a[n]] - row[b[n]]).abs()) < 0.1 * float(row.std()), n


def test_sampled_rows_and_server_style_engine_on_the_tiny_preset():
    from batchgen_b200.config import get_model_config
    from batchgen_b200.models import build_model
    from batchgen_b200.runtime.sequence import SamplingParams
    model = build_model(get_model_config("tiny-pamevik"), device=DEV, dtype="bf16", seed=1)
    eng = pm.engine(model, tokens=64 * 40, slots=4)
    outs = eng.generate([[1, 2, 3], [5] * 70], [SamplingParams(max_new_tokens=9, temperature=0.8, top_k=20),
                                               SamplingParams(max_new_tokens=5)])
    assert [len(o) for o in outs] == [9, 5]
