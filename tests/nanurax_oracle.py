"""Plain, slow implementation of the Nanurax design: one function per mechanism, float64 or float32 torch on the
CPU, whole sequences at once and no cache.  It shares no code with the package; the tests compare the two.

``cfg`` is the parsed config.json, ``w`` a dict name -> tensor (any float dtype; promoted to ``dt``).
"""
import math

import torch


def rms(x, eps):
    """x divided by the root of (mean of squares + eps), over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_mlp(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def clamped_expert(x, gate, up, down, limit):
    """g is bounded from above only, u on both sides; y = g sigmoid(1.702 g) (u + 1)."""
    g = (x @ gate.T).clamp(max=limit)
    u = (x @ up.T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, router, top):
    """-> (chosen [n, top], their sigmoid scores [n, top]); the scores are not renormalised."""
    s = torch.sigmoid(h @ router.T)
    val, idx = torch.topk(s, top, dim=-1)
    return idx, val


def moe(h, w, p, mlp):
    """Routed experts on (weight * h), plus the shared expert gated by one sigmoid per token."""
    idx, val = route(h, w[p + "router"], mlp["router"]["top"])
    lim = mlp["expert"]["limit"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            e = f"{p}e{int(idx[t, j])}."
            out[t] += clamped_expert(val[t, j] * h[t], w[e + "gate"], w[e + "up"], w[e + "down"], lim)
    if mlp.get("shared"):
        s = p + "shared."
        y = clamped_expert(h, w[s + "gate"], w[s + "up"], w[s + "down"], mlp["shared"]["limit"])
        out = out + y * torch.sigmoid(h @ w[s + "sg"].T)
    return out


def visible_chunk(n, size):
    """[n, n] bool: j is seen by i when j <= i and both lie in the same chunk (counted from position 0)."""
    i = torch.arange(n)
    same = (i[:, None] // size) == (i[None, :] // size)
    return same & (i[None, :] <= i[:, None])


def sink_softmax(s, seen):
    """exp(s) / (1 + sum exp(s)) over the visible places of the last axis."""
    s = s.masked_fill(~seen, -math.inf)
    m = s.amax(-1, keepdim=True).clamp(min=0)            # the sink's score is 0
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def talking_attention(q, k, v, talk, scale, chunk):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; scores of the heads are mixed by talk [H, H] before the softmax."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    kk, vv = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    s = torch.einsum("hg,gij->hij", talk, s)
    p = sink_softmax(s, visible_chunk(n, chunk))
    return torch.einsum("hij,jhv->ihv", p, vv)


def attention_mixer(h, w, p, m, eps):
    H, G = m["heads"], m["kv_heads"]
    n = h.shape[0]
    q = (h @ w[p + "q"].T).view(n, H, m["dim"])
    k = (h @ w[p + "k"].T).view(n, G, m["dim"])
    v = (h @ w[p + "v"].T).view(n, G, m["vdim"])
    o = talking_attention(q, k, v, w[p + "talk"], m["scale"], m["mask"]["size"])
    return o.reshape(n, -1) @ w[p + "o"].T


def delta_inputs(h, w, p, H, d):
    """(r, k, v, decay, unit key, removal) of every token, [n, H, d] each."""
    n = h.shape[0]
    r, k, v = ((h @ w[p + x].T).view(n, H, d) for x in "rkv")
    low = torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(low)).view(n, H, d)
    a = torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).view(n, H, d)
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    return r, k, v, decay, u, a


def general_delta(r, k, v, decay, u, a, S=None):
    """S [H, key, value]; -> (o [n, H, d], last state)."""
    n, H, d = r.shape
    if S is None:
        S = torch.zeros(H, d, v.shape[-1], dtype=r.dtype)
    out = []
    for t in range(n):
        read = torch.einsum("hk,hkv->hv", u[t], S)
        S = (decay[t].unsqueeze(-1) * S - (a[t] * u[t]).unsqueeze(-1) * read.unsqueeze(1)
             + k[t].unsqueeze(-1) * v[t].unsqueeze(1))
        out.append(torch.einsum("hkv,hk->hv", S, r[t]))
    return torch.stack(out), S


def delta_mixer(h, w, p, m, eps):
    H, d = m["heads"], m["dim"]
    o, _ = general_delta(*delta_inputs(h, w, p, H, d))
    y = rms(o, eps).reshape(h.shape[0], -1) * w[p + "norm"]
    return (y * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"general_delta": delta_mixer, "attention": attention_mixer}


def forward(cfg, weights, tokens, dt=torch.float64, trace=None):
    """Logits [n, vocab] of one sequence.  ``trace``: list that receives the residual stream after every layer."""
    w = {k: (t.to(dt) if t.is_floating_point() else t) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens).long()] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        h = rms_norm(x, w[f"l{i}.norm1"], eps)
        y = MIXERS[layer["type"]](h, w, f"l{i}.mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp:
            p = f"l{i}.mlp."
            if mlp["kind"] == "dense":
                y = y + dense_mlp(h, w[p + "gate"], w[p + "up"], w[p + "down"])
            else:
                y = y + moe(h, w, p, mlp)
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


# ------------------------------------------------------------------ random models for the tests
def tensor_shapes(cfg, rank=None):
    """name -> shape of every tensor of a config (``rank``: width of the low-rank decay projection)."""
    D, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        out[f"l{i}.norm1"] = (D,)
        if layer["type"] == "general_delta":
            n, r = m["heads"] * m["dim"], rank or 12
            for x in ("r", "k", "v", "g", "a"):
                out[p + x] = (n, D)
            out.update({p + "a.b": (n,), p + "w0": (n,), p + "norm": (n,), p + "w1": (r, D), p + "w2": (n, r),
                        p + "o": (D, n)})
        else:
            H, G = m["heads"], m["kv_heads"]
            out.update({p + "q": (H * m["dim"], D), p + "k": (G * m["dim"], D), p + "v": (G * m["vdim"], D),
                        p + "talk": (H, H), p + "o": (D, H * m["vdim"])})
        mlp, p = layer.get("mlp"), f"l{i}.mlp."

        def ff(prefix, n):
            out.update({prefix + "gate": (n, D), prefix + "up": (n, D), prefix + "down": (D, n)})
        if mlp and mlp["kind"] == "dense":
            ff(p, mlp["ff"])
        elif mlp:
            out[p + "router"] = (mlp["router"]["experts"], D)
            for e in range(mlp["router"]["experts"]):
                ff(f"{p}e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                ff(p + "shared.", mlp["shared"]["ff"])
                out[p + "shared.sg"] = (1, D)
    return out


def random_weights(cfg, seed=0, rank=None):
    """bfloat16 weights that keep every mechanism visible: heads mix strongly, experts differ, gates are not flat."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        t = torch.randn(shape, generator=g)
        if name.endswith("norm") or name.endswith("norm1"):
            t = 1 + 0.2 * t
        elif name.endswith("talk"):
            t = 0.6 * torch.eye(shape[0]) + 0.5 * t / math.sqrt(shape[0])
        elif len(shape) == 1:
            t = 0.7 * t
        elif name == "embed":
            t = t / cfg["embedding"]["scale"]
        else:
            t = t * (1.2 / math.sqrt(shape[1]))
        out[name] = t.to(torch.bfloat16)
    return out
