"""Vifirax in plain, slow PyTorch: the statement the engine is held against.

One function per mechanism, whole sequences only, no cache, no batching, nothing shared with the package.  `cfg` is
the raw config.json dictionary, `w` maps tensor names to tensors; everything runs in the type of the weights it is
given (the tests pass float32 or float64 copies).

    embedding     x[p] = embed[token]
    layer         x += norm1(mixer(x));  x += norm2(ff(x));  norm(y) = y / sqrt(mean(y^2) + eps) * (1 + w)
    attention     q, k, v with biases; q and k normed over their whole rows (all heads at once) with plain gains; the first
                  rot.dims elements of every head turned, element i with i + dims/2, by p * f_i with the stretched frequencies
                  below; every earlier key visible; p_j = exp(s_j) / (1 + sum exp(s)); the head's output times
                  sigmoid(g x)_h; output projection with a bias.  A layer with `kv_from` reads that layer's keys and values
    turn          f_i = base^(-2i/dims);  at(t) = dims ln(original / (2 pi t)) / (2 ln base);  ramp_i goes from 0 at
                  max(floor(at(fast)), 0) to 1 at min(ceil(at(slow)), dims - 1);  f_i <- f_i ((1 - ramp_i) + ramp_i / factor);
                  cos and sin times 1 + 0.1 ln(factor)
    mamba2        z | x | B | C | dt = in(h);  x, B, C through a causal convolution per channel with a bias, and silu;
                  dt = softplus(dt + dt_bias);  per head (group h // (heads / groups)):
                  S = exp(-exp(A_log) dt) S + dt B x^T;  y = S^T C + D x;  y silu(z) in norm_groups equal parts, each over its own
                  root mean square, times a gain; output projection
    channel_delta q, k, v through a causal convolution over time per channel and silu; q and k heads made unit vectors (q also
                  times dim^-1/2); per value head a state S [dim, vdim]:  S = diag(g) S;  u = beta (v - S^T k);  S += k u^T;
                  o = S^T q;  g = exp(-exp(A_log_h) softplus(a2 (a1 x) + dt_bias)), beta = sigmoid(b x);
                  o over its root mean square per head, times a gain and sigmoid(g2 (g1 x)); output projection
    feed-forward  dense: down(silu(gate x) * up x);  experts: z = router x + bias, the `top` largest chosen, weights the softmax
                  over the chosen z, the output the weighted sum of the chosen experts' (dense, gated) outputs
    head          final norm, logits = (embed x) * logit_scale
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gain_norm(x, gain, eps):
    return rms(x, eps) * gain


def layer_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def frequencies(rot):
    """(frequencies as a list of Python floats, factor on cos and sin)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def at(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(float(sc["fast"]))), 0), min(math.ceil(at(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def turn(x, rot):
    """x [n, heads, dim], row i at position i."""
    if rot is None or int(rot["dims"]) == 0:
        return x
    dims = int(rot["dims"])
    f, m = frequencies(rot)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
    c, s = (torch.cos(a) * m).to(x.dtype)[:, None, :], (torch.sin(a) * m).to(x.dtype)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def sink_softmax(scores, visible):
    """Rows of exp(s_j) / (1 + sum over the visible of exp(s))."""
    scores = scores.masked_fill(~visible, float("-inf"))
    m = scores.max(dim=-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(scores - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention(m, w, p, h, eps, kv):
    """Returns (output, (keys, values) that the layer attended to)."""
    n, H, D = h.shape[0], m["heads"], m["dim"]
    G = m.get("kv_heads", H)
    V = m.get("vdim", D)
    q = gain_norm(h @ w[p + "q"].T + w[p + "q.b"], w[p + "q.norm"], eps).view(n, H, D)
    q = turn(q, m.get("rot"))
    if m.get("kv_from") is None:
        k = gain_norm(h @ w[p + "k"].T + w[p + "k.b"], w[p + "k.norm"], eps).view(n, G, D)
        k = turn(k, m.get("rot"))
        v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, V)
    else:
        k, v = kv[m["kv_from"]]
    scale = float(m.get("scale", D ** -0.5))
    visible = torch.arange(n)[None, :] <= torch.arange(n)[:, None]
    gate = torch.sigmoid(h @ w[p + "g"].T)
    out = []
    for a in range(H):
        g = a // (H // G)
        out.append((sink_softmax((q[:, a] @ k[:, g].T) * scale, visible) @ v[:, g]) * gate[:, a:a + 1])
    return torch.cat(out, dim=-1) @ w[p + "o"].T + w[p + "o.b"], (k, v)


def short_conv(x, taps, bias=None):
    """x [n, channels], taps [channels, T]: y[t] = bias + sum_i taps[:, T - 1 - i] * x[t - i], zeros before the start."""
    n, T = x.shape[0], taps.shape[1]
    padded = torch.cat([x.new_zeros((T - 1, x.shape[1])), x], dim=0)
    y = torch.zeros_like(x) if bias is None else bias.expand_as(x).clone()
    for i in range(T):
        y = y + padded[T - 1 - i:T - 1 - i + n] * taps[:, T - 1 - i]
    return y


def ssd(x, B, C, dt, a, D):
    """The recurrence alone: x [n, heads, vdim], B, C [n, groups, state], dt [n, heads], a (negative) and D [heads]."""
    n, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    y = torch.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        S = x.new_zeros((N, V))
        for t in range(n):
            S = torch.exp(a[h] * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + D[h] * x[t, h]
    return y


def mamba2(m, w, p, h, eps):
    n, H, V, N = h.shape[0], m["heads"], m["vdim"], m["state"]
    G, parts = m.get("groups", 1), m.get("norm_groups", 1)
    inner = H * V
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    dt = softplus(dt + w[p + "dt_bias"])
    y = ssd(x.reshape(n, H, V), B.reshape(n, G, N), C.reshape(n, G, N), dt, -torch.exp(w[p + "A_log"]), w[p + "D"])
    y = y.reshape(n, inner) * silu(z)
    y = rms(y.view(n, parts, inner // parts), eps).reshape(n, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_steps(q, k, v, beta, g):
    """The recurrence alone: q, k [n, kv heads, dim], v [n, heads, vdim], beta [n, heads], g [n, heads, dim]."""
    n, H, V = v.shape
    G, D = k.shape[1], k.shape[2]
    out = torch.zeros_like(v)
    for a in range(H):
        b = a // (H // G)
        S = v.new_zeros((D, V))
        for t in range(n):
            S = g[t, a][:, None] * S
            u = beta[t, a] * (v[t, a] - S.T @ k[t, b])
            S = S + torch.outer(k[t, b], u)
            out[t, a] = S.T @ q[t, b]
    return out


def channel_delta(m, w, p, h, eps):
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads", H)
    q = unit(silu(short_conv(h @ w[p + "q"].T, w[p + "q.conv"])).view(n, G, D)) * D ** -0.5
    k = unit(silu(short_conv(h @ w[p + "k"].T, w[p + "k.conv"])).view(n, G, D))
    v = silu(short_conv(h @ w[p + "v"].T, w[p + "v.conv"])).view(n, H, V)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(n, H, D)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z))
    o = rms(delta_steps(q, k, v, beta, g), eps) * w[p + "norm"]
    o = o.reshape(n, H * V) * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return o @ w[p + "o"].T


def gated_ff(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(mlp, w, p, h):
    """(chosen [n, top], their weights [n, top])."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    val, idx = torch.topk(z, int(mlp["router"]["top"]), dim=-1)
    return idx, torch.softmax(val, dim=-1)


def experts_ff(mlp, w, p, h):
    idx, weight = route(mlp, w, p, h)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        rows, rank = (idx == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weight[rows, rank][:, None] * gated_ff(w, f"{p}e{e}.", h[rows])
    return out


def forward(cfg, w, tokens, layers_out=None):
    """Logits [n, vocab] of one whole sequence; `layers_out`, a list, receives the residual after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kv = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "attention":
            y, kv[i] = attention(m, w, p, x, eps, kv)
        elif layer["type"] == "mamba2":
            y = mamba2(m, w, p, x, eps)
        else:
            y = channel_delta(m, w, p, x, eps)
        x = x + layer_norm(y, w[f"l{i}.norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = gated_ff(w, f"l{i}.mlp.", x) if mlp["kind"] == "dense" else experts_ff(mlp, w, f"l{i}.mlp.", x)
            x = x + layer_norm(y, w[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return (layer_norm(x, w["final.norm"], eps) @ w["embed"].T) * float(cfg.get("logit_scale", 1.0))
