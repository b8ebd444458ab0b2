"""Plain, slow implementation of the Pamevik design: one function per mechanism, float64 or float32 torch on the CPU, whole
sequences at once and no cache.  It shares no code with the package; the tests compare the two.

``cfg`` is the parsed config.json, ``w`` a dict name -> tensor (any float dtype; promoted to ``dt``).
"""
import math

import torch
import torch.nn.functional as F


# ---------------------------------------------------------------- norms, convolution, rotation, activations
def layer_norm(x, weight, bias, eps):
    mean = x.mean(-1, keepdim=True)
    dev = x - mean
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * weight + bias


def rms(x, eps):
    """x divided by the root of (mean of squares + eps), over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(x, weight):
    """x [n, C], weight [C, taps]: y_t = sum_j weight[:, j] x_(t - taps + 1 + j), zeros before the first token."""
    n, taps = x.shape[0], weight.shape[1]
    y = torch.zeros_like(x)
    for t in range(n):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] = y[t] + weight[:, j] * x[s]
    return y


def rotate(x, base, dims):
    """x [n, heads, d] at positions 0 .. n - 1: dimension i (i < dims / 2) turns with dimension i + dims / 2 by the angle
    position * base^(-2 i / dims); dimensions from ``dims`` on stay."""
    half = dims // 2
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    out = x.clone()
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype).view(-1, 1), torch.sin(a).to(x.dtype).view(-1, 1)
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def squared_relu_mlp(h, up, down):
    return (h @ up.T).clamp_min(0).pow(2) @ down.T


# ---------------------------------------------------------------- mixers' cores
def attention(q, k, v, scale):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; head h reads key head h // (H / G); causal softmax -> [n, H, dv]."""
    n, H = q.shape[:2]
    rep = H // k.shape[1]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].T * scale
        s = s.masked_fill(torch.triu(torch.ones(n, n, dtype=torch.bool), 1), -math.inf)
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


def mlstm(q, k, v, i, f, state=None):
    """i, f [n, H]: log input and log forget gates.  -> (o [n, H, dv], (S, normaliser, running maximum))."""
    n, H, d = q.shape
    if state is None:
        state = (torch.zeros(H, d, v.shape[2], dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    S, nrm, m = state
    out = []
    for t in range(n):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep.view(H, 1, 1) * S + put.view(H, 1, 1) * k[t].unsqueeze(2) * v[t].unsqueeze(1)
        nrm = keep.view(H, 1) * nrm + put.view(H, 1) * k[t]
        m = new
        den = torch.maximum((nrm * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hkv,hk->hv", S, q[t]) / den.unsqueeze(1))
    return torch.stack(out), (S, nrm, m)


def gated_delta(q, k, v, g, beta, S=None):
    """q, k, g [n, H, d], v [n, H, dv], beta [n, H]: decay the rows, correct the value, write, read."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    out = []
    for t in range(n):
        S = g[t].unsqueeze(2) * S
        u = beta[t].unsqueeze(1) * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t].unsqueeze(2) * u.unsqueeze(1)
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


# ---------------------------------------------------------------- mixers
def mix_attention(h, w, p, m):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).view(n, H, m["dim"])
    k = (h @ w[p + "k"].T).view(n, G, m["dim"])
    v = (h @ w[p + "v"].T).view(n, G, m["vdim"])
    q, k = (rotate(x, m["rot"]["base"], m["rot"]["dims"]) for x in (q, k))
    o = attention(q, k, v, m["scale"]) * torch.sigmoid(h @ w[p + "g"].T).unsqueeze(2)
    return o.reshape(n, -1) @ w[p + "o"].T


def mix_retention(h, w, p, m, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    q, k = (rotate((h @ w[p + x].T).view(n, H, d), m["rot"]["base"], m["rot"]["dims"]) for x in ("q", "k"))
    v = (h @ w[p + "v"].T).view(n, H, m["vdim"])
    o, _ = retention(q, k * d ** -0.5, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o, eps).reshape(n, -1) * F.silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mix_mlstm(h, w, p, m, eps):
    n, H, d, cap = h.shape[0], m["heads"], m["dim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(n, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(n, H, d)
    v = (h @ w[p + "v"].T).view(n, H, m["vdim"])
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = F.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o, _ = mlstm(q, k, v, i, f)
    return (rms(o, eps).reshape(n, -1) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mix_channel_delta(h, w, p, m, eps):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (F.silu(causal_conv(h @ w[p + x].T, w[p + x + ".conv"])) for x in ("q", "k", "v"))
    q = unit(q.view(n, G, d)).repeat_interleave(H // G, 1) * d ** -0.5
    k = unit(k.view(n, G, d)).repeat_interleave(H // G, 1)
    low = (h @ w[p + "a1"].T) @ w[p + "a2"].T
    g = torch.exp(-torch.exp(w[p + "A_log"]).view(1, H, 1) * F.softplus(low + w[p + "dt_bias"]).view(n, H, d))
    o, _ = gated_delta(q, k, v.view(n, H, dv), g, torch.sigmoid(h @ w[p + "b"].T))
    o = rms(o, eps) * w[p + "norm"]
    return (o.reshape(n, -1) * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)) @ w[p + "o"].T


def mix_parallel(h, w, p, m, eps):
    a = rms(mix_attention(h, w, p + "left.", m["left"]), eps) * w[p + "left.out"]
    b = rms(mix_retention(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (a + b)


# ---------------------------------------------------------------- the model
def forward(cfg, w, ids, dt=torch.float64, trace=None):
    """Logits [n, vocab] of one sequence; ``trace`` (a list) collects the residual stream after every layer."""
    w = {k: t.to(dt) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids)]

    def ln(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)
    mixers = {"mlstm": mix_mlstm, "channel_delta": mix_channel_delta, "parallel": mix_parallel}
    for i, layer in enumerate(cfg["layers"]):
        l = f"l{i}."
        h = ln(x, l + "norm1")
        h = h + causal_conv(h, w[l + "canon1"])
        x = x + ln(mixers[layer["type"]](h, w, l + "mix.", layer["mixer"], eps), l + "norm1b")
        if layer.get("mlp"):
            h = ln(x, l + "norm2")
            h = h + causal_conv(h, w[l + "canon2"])
            x = x + ln(squared_relu_mlp(h, w[l + "mlp.up"], w[l + "mlp.down"]), l + "norm2b")
        if trace is not None:
            trace.append(x)
    return ln(x, "final.norm") @ w["head"].T


# ---------------------------------------------------------------- random weights for the tests
def tensor_shapes(cfg, ranks):
    """name -> shape; ``ranks`` = (decay rank, gate rank) of the low-rank projections."""
    D, taps = cfg["width"], cfg["canon"]["taps"]
    out = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D), "final.norm": (D,), "final.norm.b": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        for s in (["1", "2"] if layer.get("mlp") else ["1"]):
            for n in ("norm" + s, "norm" + s + "b"):
                out[l + n] = out[l + n + ".b"] = (D,)
            out[l + "canon" + s] = (D, taps)
        if layer.get("mlp"):
            out[l + "mlp.up"], out[l + "mlp.down"] = (layer["mlp"]["ff"], D), (D, layer["mlp"]["ff"])
        p = l + "mix."

        def lin(prefix, **rows):
            out.update({prefix + k: (r, D) for k, r in rows.items()})
        if layer["type"] == "mlstm":
            qk, n, H = m["heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"]
            lin(p, q=qk, k=qk, v=n, g=n, i=H, f=H)
            out.update({p + "i.b": (H,), p + "f.b": (H,), p + "norm": (n,), p + "o": (D, n)})
        elif layer["type"] == "channel_delta":
            H, G, d, n = m["heads"], m["kv_heads"], m["dim"], m["heads"] * m["vdim"]
            lin(p, q=G * d, k=G * d, v=n, b=H, a1=ranks[0], g1=ranks[1])
            out.update({p + x + ".conv": (out[p + x][0], m["conv"]) for x in ("q", "k", "v")})
            out.update({p + "a2": (H * d, ranks[0]), p + "g2": (n, ranks[1]), p + "A_log": (H,), p + "dt_bias": (H * d,),
                        p + "norm": (m["vdim"],), p + "o": (D, n)})
        else:
            a, r = m["left"], m["right"]
            lin(p + "left.", q=a["heads"] * a["dim"], k=a["kv_heads"] * a["dim"], v=a["kv_heads"] * a["vdim"], g=a["heads"])
            out[p + "left.o"] = (D, a["heads"] * a["vdim"])
            n = r["heads"] * r["vdim"]
            lin(p + "right.", q=r["heads"] * r["dim"], k=r["heads"] * r["dim"], v=n, g=n)
            out[p + "right.o"] = (D, n)
            out[p + "left.out"] = out[p + "right.out"] = (D,)
    return out


def random_weights(cfg, seed=0, ranks=(11, 9)):
    """Weights with every mechanism in play: gains near 1, biases of visible size, forget gates mostly open, decays from slow
    to fast, scores of order 1.  Values are representable in bf16."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in sorted(tensor_shapes(cfg, ranks).items()):
        t = torch.randn(shape, generator=g)
        leaf = name.split(".")[-1]
        if name.endswith((".i.b", ".f.b")):
            t = 0.5 * t + (2.0 if name.endswith(".f.b") else 0.0)
        elif leaf == "b" and len(shape) == 1:
            t = 0.2 * t
        elif leaf in ("A_log", "dt_bias"):
            t = 0.5 * t - (1.5 if leaf == "dt_bias" else 0.0)
        elif leaf in ("norm", "out") or leaf.startswith("norm"):
            t = 1 + 0.2 * t
        elif leaf.startswith("canon") or leaf == "conv":
            t = 0.5 * t
            if leaf == "conv":
                t[:, -1] += 1
        elif leaf in ("embed", "head"):
            t = t if leaf == "embed" else t * shape[1] ** -0.5
        else:
            t = t * 1.3 * shape[1] ** -0.5
        w[name] = t.bfloat16().float()
    return w
