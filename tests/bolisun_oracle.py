"""Plain, slow implementation of the Bolisun design: one function per mechanism, float64 or float32 torch on the CPU, whole
sequences at once and no cache.  It shares no code with the package; the tests compare the two.

``cfg`` is the parsed config.json, ``w`` a dict name -> tensor (any float dtype; promoted to ``dt``).
"""
import math

import torch


# ---------------------------------------------------------------- norms, rotation
def rms(x, eps):
    """x divided by the root of (mean of squares + eps), over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def frequencies(dims, base, scaling=None):
    """Angle per position of every pair.  With ``scaling`` the slow pairs are divided by ``factor``; a ramp over the pair's
    number lies between the pairs that turn ``fast`` and ``slow`` times within ``original`` positions."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f

    def pair_turning(times):
        return dims * math.log(scaling["original"] / (2 * math.pi * times)) / (2 * math.log(base))
    lo = max(math.floor(pair_turning(scaling["fast"])), 0)
    hi = min(math.ceil(pair_turning(scaling["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / scaling["factor"] * ramp + x * (1 - ramp))
    return out


def rotate(x, base, dims, scaling=None):
    """x [n, heads, d] at positions 0 .. n - 1: dimension 2 i turns with dimension 2 i + 1; dimensions from ``dims`` on stay."""
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    mult = 1.0 if scaling is None else 0.1 * math.log(scaling["factor"]) + 1.0
    out = x.clone()
    for i, f in enumerate(frequencies(dims, base, scaling)):
        c, s = ((fn(pos * f) * mult).to(x.dtype).view(-1, 1) for fn in (torch.cos, torch.sin))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---------------------------------------------------------------- mixers
def visible(n, size, keep_first):
    """[n, n] bool: position i sees j."""
    i, j = torch.arange(n).view(-1, 1), torch.arange(n).view(1, -1)
    return (j <= i) & ((i - j < size) | (j < keep_first))


def attention(q, k, v, scale, seen):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; head h reads key head h // (H / G); softmax over the seen keys -> [n, H, dv]."""
    H = q.shape[1]
    rep = H // k.shape[1]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T * scale).masked_fill(~seen, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, h // rep])
    return torch.stack(out, 1)


def retention(q, k, v, decay, S=None):
    """S <- decay_h S + k v^T, o = S^T q.  q, k [n, H, d], v [n, H, dv], decay [H] -> (o [n, H, dv], S)."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    out = []
    for t in range(n):
        S = decay.view(H, 1, 1) * S + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def mix_attention(h, w, p, m, eps):
    n = h.shape[0]
    q, k, v = (h @ w[p + x].T + w[p + x + ".b"] for x in "qkv")
    q = rms(q.view(n, m["heads"], m["dim"]), eps) * w[p + "q.norm"]
    k = rms(k.view(n, m["kv_heads"], m["dim"]), eps) * w[p + "k.norm"]
    r = m["rot"]
    q, k = (rotate(x, r["base"], r["dims"], r.get("scaling")) for x in (q, k))
    seen = visible(n, m["mask"]["size"], m["mask"]["keep_first"])
    o = attention(q, k, v.view(n, m["kv_heads"], m["vdim"]), m["scale"], seen)
    return o.reshape(n, -1) @ w[p + "o"].T + w[p + "o.b"]


def silu(z):
    return z * torch.sigmoid(z)


def mix_retention(h, w, p, m, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    q, k = ((h @ w[p + x].T).view(n, H, d) for x in "qk")
    o, _ = retention(q, k * d ** -0.5, (h @ w[p + "v"].T).view(n, H, m["vdim"]), torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o, eps).reshape(n, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mix_parallel(h, w, p, m, eps):
    return (m["left_scale"] * mix_attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * mix_retention(h, w, p + "right.", m["right"], eps))


# ---------------------------------------------------------------- feed-forwards
def dense(h, w, p, limit):
    g = (h @ w[p + "gate"].T).clamp(max=limit)
    u = (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, router):
    """z [n, experts] -> (experts [n, top], weights [n, top])."""
    s = torch.softmax(z, -1)
    choice = s + correction
    g = router.get("groups")
    if g:
        n, size = z.shape[0], z.shape[1] // g["count"]
        for t in range(n):
            best = [float(choice[t, i * size:(i + 1) * size].max()) for i in range(g["count"])]
            kept = sorted(range(g["count"]), key=lambda i: -best[i])[:g["keep"]]
            for i in range(g["count"]):
                if i not in kept:
                    choice[t, i * size:(i + 1) * size] = -math.inf
    idx = torch.topk(choice, router["top"], -1).indices
    p = s.gather(-1, idx)
    return idx, p / (p.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def mixture(h, w, p, f):
    idx, weight = route(h @ w[p + "router"].T, w[p + "correction"], f["router"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, k = torch.nonzero(idx == e, as_tuple=True)
        if len(t):
            out[t] += weight[t, k].unsqueeze(1) * expert(h[t], w, f"{p}e{e}.")
    return out + expert(h, w, p + "shared.") if f.get("shared") else out


# ---------------------------------------------------------------- the model
def hyper_step(xs, w, p, norm, fn, eps):
    """One sublayer around streams xs [s, n, width]: read a weighted sum, mix the old streams, add the output to each."""
    u = sum(w[p + "in"][s] * xs[s] for s in range(len(xs)))
    y = fn(rms(u, eps) * norm)
    return torch.stack([sum(w[p + "mix"][s, t] * xs[s] for s in range(len(xs))) + w[p + "out"][t] * y for t in range(len(xs))])


def source(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, ids, dt=torch.float64, trace=None):
    """Logits [n, vocab] of one sequence; ``trace`` (a list) collects the summed streams after every layer."""
    w = {k: t.to(dt) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids)] * cfg["embedding"]["scale"]
    xs = torch.stack([x] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        l, f = f"l{source(cfg, i)}.", layer.get("mlp")
        xs = hyper_step(xs, w, l + "hc1.", w[l + "norm1"], lambda h: mix_parallel(h, w, l + "mix.", layer["mixer"], eps), eps)
        if f:
            ff = (lambda h: dense(h, w, l + "mlp.", f["limit"])) if f["kind"] == "dense" else (lambda h: mixture(h, w, l + "mlp.", f))
            xs = hyper_step(xs, w, l + "hc2.", w[l + "norm2"], ff, eps)
        if trace is not None:
            trace.append(xs.sum(0))
    return rms(xs.sum(0), eps) * w["final.norm"] @ w["embed"].T


# ---------------------------------------------------------------- random weights for the tests
def tensor_shapes(cfg):
    D, s = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        l, a, r, f = f"l{i}.", layer["mixer"]["left"], layer["mixer"]["right"], layer.get("mlp")
        for q in "12" if f else "1":
            out.update({f"{l}norm{q}": (D,), f"{l}hc{q}.in": (s,), f"{l}hc{q}.out": (s,), f"{l}hc{q}.mix": (s, s)})
        p = l + "mix.left."
        for x, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
            out[p + x], out[p + x + ".b"] = (n, D), (n,)
        out.update({p + "q.norm": (a["dim"],), p + "k.norm": (a["dim"],), p + "o": (D, a["heads"] * a["vdim"]), p + "o.b": (D,)})
        p, qk, n = l + "mix.right.", r["heads"] * r["dim"], r["heads"] * r["vdim"]
        out.update({p + "q": (qk, D), p + "k": (qk, D), p + "v": (n, D), p + "g": (n, D), p + "o": (D, n)})

        def ff(p, n):
            out.update({p + "gate": (n, D), p + "up": (n, D), p + "down": (D, n)})
        if f and f["kind"] == "dense":
            ff(l + "mlp.", f["ff"])
        elif f:
            E = f["router"]["experts"]
            out.update({l + "mlp.router": (E, D), l + "mlp.correction": (E,)})
            for e in range(E):
                ff(f"{l}mlp.e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                ff(l + "mlp.shared.", f["shared"]["ff"])
    return out


def random_weights(cfg, seed=0, settled=False):
    """Weights with every mechanism in play: gains near 1, biases of visible size, streams that differ, router corrections that
    make choice scores of both signs.  ``settled``: corrections far apart, so that few choices are close.  Values are representable
    in bf16."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        t = torch.randn(shape, generator=g)
        leaf = name.split(".")[-1]
        if leaf == "b":
            t = 0.3 * t
        elif "norm" in leaf:
            t = 1 + 0.2 * t
        elif leaf == "in":
            t = (1 + 0.4 * t) / shape[0]
        elif leaf == "out":
            t = 1 + 0.4 * t
        elif leaf == "mix":
            t = 0.8 * torch.eye(shape[0]) + 0.2 * t / shape[0] ** 0.5
        elif leaf == "correction":
            t = (1.0 if settled else 0.1) * t - 0.15
        elif leaf != "embed":
            t = t * (2.5 if leaf == "router" else 1.3) * shape[1] ** -0.5
        w[name] = t.bfloat16().float()
    return w
