"""Plain, slow implementation of the Pitudra design: one function per mechanism, float64 or float32 torch on the CPU, whole
sequences at once and no cache.  It shares no code with the package; the tests compare the two.

``cfg`` is the parsed config.json, ``w`` a dict name -> tensor (any float dtype; promoted to ``dt``).
"""
import math

import torch


# ---------------------------------------------------------------- norms, shift, rotation
def rms(x, eps):
    """x divided by the root of (mean of squares + eps), over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def token_shift(h, mu):
    """Every token's row moves towards the one before it (zeros before the first), channel by channel."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def rotate(x, base):
    """x [n, ..., d] at positions 0 .. n - 1: dimension i turns with dimension i + d / 2."""
    n, half = x.shape[0], x.shape[-1] // 2
    out = x.clone()
    for i in range(half):
        a = torch.arange(n, dtype=torch.float64) * base ** (-2.0 * i / (2 * half))
        c, s = (f(a).to(x.dtype).view(n, *[1] * (x.dim() - 2)) for f in (torch.cos, torch.sin))
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


# ---------------------------------------------------------------- attention
def visible(n, size=None):
    """[n, n] bool: position i sees j."""
    i, j = torch.arange(n).view(-1, 1), torch.arange(n).view(1, -1)
    return (j <= i) & (i - j < (size or n))


def sink_softmax(s, seen, sink):
    """Weights of one head: the denominator has one more term, exp(sink), that belongs to no key."""
    s = s.masked_fill(~seen, -math.inf)
    m = torch.maximum(s.amax(-1, keepdim=True), sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def attention(q, k, v, scale, seen, sink):
    """q [n, H, d], k [n, G, d], v [n, G, dv], sink [H]; head h reads key head h // (H / G) -> [n, H, dv]."""
    H = q.shape[1]
    rep = H // k.shape[1]
    return torch.stack([sink_softmax(q[:, h] @ k[:, h // rep].T * scale, seen, sink[h]) @ v[:, h // rep] for h in range(H)], 1)


def mix_attention(h, w, p, m, eps):
    """Norms run over all heads' rows of the projection at once; an element-wise gate scales the heads."""
    n = h.shape[0]
    q, k, v = (h @ w[p + x].T + w[p + x + ".b"] for x in "qkv")
    q, k = rms(q, eps) * w[p + "q.norm"], rms(k, eps) * w[p + "k.norm"]
    q, k, v = (t.view(n, -1, d) for t, d in ((q, m["dim"]), (k, m["dim"]), (v, m["vdim"])))
    o = attention(q, k, v, m["scale"], visible(n, (m.get("mask") or {}).get("size")), w[p + "sink"])
    return (o.reshape(n, -1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def latent(h, w, p, m, eps):
    """What a latent layer keeps of its tokens: the normed latent and the rotated key part all heads share."""
    r = m["kv_rank"]
    z = h @ w[p + "dkv"].T
    return rms(z[:, :r], eps) * w[p + "dkv.norm"], rotate(z[:, r:], m["rot"]["base"])


def mix_latent(h, w, p, m, eps, kept):
    """``kept``: (latent, rotated key part) of this layer or of the one it borrows from."""
    n, H, d = h.shape[0], m["heads"], m["dim"]
    c, kr = kept
    q = (rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T
    q = q.view(n, H, d + m["rot_dim"])
    q = torch.cat([q[..., :d], rotate(q[..., d:], m["rot"]["base"])], -1)
    k = torch.cat([(c @ w[p + "uk"].T).view(n, H, d), kr.unsqueeze(1).expand(n, H, m["rot_dim"])], -1)
    v = (c @ w[p + "uv"].T).view(n, H, m["vdim"])
    o = attention(q, k, v, m["scale"], visible(n, (m.get("mask") or {}).get("size")), w[p + "sink"])
    return o.reshape(n, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- recurrence
def silu(z):
    return z * torch.sigmoid(z)


def hgrn2(q, f, v, S=None):
    """S <- diag(f) S + (1 - f) v^T, o = S^T q.  q, f [n, H, d], v [n, H, dv] -> (o [n, H, dv], S)."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    out = []
    for t in range(n):
        S = f[t].unsqueeze(2) * S + (1 - f[t]).unsqueeze(2) * v[t].unsqueeze(1)
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def forget(z, low):
    return low + (1 - low) * torch.sigmoid(z)


def mix_hgrn2(h, w, p, m, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    f = forget(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"])
    o, _ = hgrn2(silu(h @ w[p + "q"].T).view(n, H, d), f.view(n, H, d), (h @ w[p + "v"].T).view(n, H, m["vdim"]))
    return (rms(o, eps) * w[p + "norm"]).reshape(n, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward, token side input
def expert(h, w, p):
    return (h @ w[p + "up"].T).clamp(min=0) ** 2 @ w[p + "down"].T


def route(z, top):
    """z [n, experts] -> (experts [n, top], weights [n, top]): softmax over the chosen logits alone."""
    v, idx = torch.topk(z, top, -1)
    return idx, torch.softmax(v, -1)


def mixture(h, w, p, f):
    idx, weight = route(h @ w[p + "router"].T, f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, k = torch.nonzero(idx == e, as_tuple=True)
        if len(t):
            out[t] += weight[t, k].unsqueeze(1) * expert(h[t], w, f"{p}e{e}.")
    return out


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def side_input(x, e, w, p, eps):
    """What the token's own row of the layer's side table adds to the residual."""
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return rms(y, eps) * w[p + "side.norm"]


# ---------------------------------------------------------------- the model
def forward(cfg, w, ids, dt=torch.float64, trace=None):
    """Logits [n, vocab] of one sequence; ``trace`` (a list) collects the residual stream after every layer."""
    w = {k: t.to(dt) for k, t in w.items()}
    eps, ids = cfg["norm"]["eps"], torch.as_tensor(ids)
    x = w["embed"][ids]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        l, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        h = token_shift(x, w[l + "shift"])
        if kind == "attention":
            y = mix_attention(h, w, l + "mix.", m, eps)
        elif kind == "hgrn2":
            y = mix_hgrn2(h, w, l + "mix.", m, eps)
        else:
            j = m.get("kv_from")
            kept[i] = latent(h, w, l + "mix.", m, eps) if j is None else kept[j]
            y = mix_latent(h, w, l + "mix.", m, eps, kept[i])
        x = x + layer_norm(y, w[l + "norm1"], w[l + "norm1.b"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(mixture(x, w, l + "mlp.", layer["mlp"]), w[l + "norm2"], w[l + "norm2.b"], eps)
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            x = x + side_input(x, w["side.embed"][ids][:, i * n:(i + 1) * n], w, l, eps)
        if trace is not None:
            trace.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


# ---------------------------------------------------------------- random weights for the tests
def tensor_shapes(cfg):
    D, L = cfg["width"], len(cfg["layers"])
    out = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D), "final.norm": (D,), "final.norm.b": (D,)}
    side = (cfg.get("token_side") or {}).get("dim", 0)
    if side:
        out["side.embed"] = (cfg["vocab"], L * side)
    for i, layer in enumerate(cfg["layers"]):
        l, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        p, H, d, dv = l + "mix.", m["heads"], m["dim"], m["vdim"]
        out[l + "shift"] = (D,)
        for q in "12" if f else "1":
            out.update({f"{l}norm{q}": (D,), f"{l}norm{q}.b": (D,)})
        out[p + "o"] = (D, H * dv)
        if layer["type"] == "attention":
            G = m["kv_heads"]
            for x, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
                out[p + x], out[p + x + ".b"] = (n, D), (n,)
            out.update({p + "q.norm": (H * d,), p + "k.norm": (G * d,), p + "sink": (H,), p + "g": (H * dv, D)})
        elif layer["type"] == "hgrn2":
            out.update({p + "q": (H * d, D), p + "f": (H * d, D), p + "f.b": (H * d,), p + "lower": (H * d,), p + "v": (H * dv, D),
                        p + "norm": (dv,)})
        else:
            r, qr = m["kv_rank"], m["q_rank"]
            out.update({p + "dq": (qr, D), p + "dq.norm": (qr,), p + "uq": (H * (d + m["rot_dim"]), qr), p + "uk": (H * d, r),
                        p + "uv": (H * dv, r), p + "sink": (H,)})
            if m.get("kv_from") is None:
                out.update({p + "dkv": (r + m["rot_dim"], D), p + "dkv.norm": (r,)})
        if f:
            out[l + "mlp.router"] = (f["router"]["experts"], D)
            for e in range(f["router"]["experts"]):
                out.update({f"{l}mlp.e{e}.up": (f["expert"]["ff"], D), f"{l}mlp.e{e}.down": (D, f["expert"]["ff"])})
        if side:
            out.update({l + "side.gate": (side, D), l + "side.proj": (D, side), l + "side.norm": (D,)})
    return out


def random_weights(cfg, seed=0, settled=False):
    """Weights with every mechanism in play: gains near 1, biases, sinks and shifts of visible size, lower bounds all over (0, 1).
    ``settled``: routers with large logits, so that few choices are close.  Values are representable in bf16."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        t = torch.randn(shape, generator=g)
        leaf = name.split(".")[-1]
        if leaf == "b":
            t = 0.3 * t
        elif leaf.startswith("norm"):
            t = 1 + 0.2 * t
        elif leaf == "lower":
            t = torch.sigmoid(2 * t)
        elif leaf == "shift":
            t = torch.sigmoid(1.5 * t)
        elif leaf == "sink":
            t = 1.5 * t
        elif leaf != "embed":
            t = t * ((6.0 if settled else 2.0) if leaf == "router" else 1.3) * shape[1] ** -0.5
        w[name] = t.bfloat16().float()
    return w
