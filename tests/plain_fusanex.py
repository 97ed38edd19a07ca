"""Fusanex in plain, slow PyTorch: the statement the engine is held against.

One function per mechanism, whole sequences only, no cache, no batching, nothing shared with the package.  `cfg` is
the raw config.json dictionary, `w` maps tensor names to tensors; everything runs in the type of the weights it is
given (the tests pass float32 or float64 copies).

    embedding        x = embed[token] * embedding.scale
    layer            x += mixer(n1(x)) + ff(n2(x)), both norms of the same x; n(y): y in norm.groups equal parts, every part
                     divided by its own sqrt(mean(part^2) + eps), the whole times a gain
    rglru            y = gelu_tanh(W_y h + b_y);  u = conv(W_x h + b_x) + b_c over time, channel by channel;  u in `blocks` equal
                     parts: r = sigmoid(R_b u_b + ..), i = sigmoid(I_b u_b + ..);  log a = -8 r softplus(lam);
                     S <- a S + sqrt(1 - a^2) i u;  output W_o (S * y)
    parallel         left_scale * left(h) + right_scale * right(h)
      left           grouped heads; q and k divided by their root mean square head by head and gained; q also times
                     1 + coef * ln(floor((p + 1) / every) + 1); values divided by their root mean square; softmax of scale * q.k
                     over every earlier key and the token's own
      right          five blends of the token's h and the one before it (zeros in front of the sequence), h + (h' - h) mu_s;
                     r, k, v, gate = silu(.), decay exp(-exp(W_2 tanh(W_1 .) + w0));  o = (S + diag(u) k v^T)^T r;
                     S <- diag(w) S + k v^T;  o divided by its root mean square per head, gained as a whole row, gated, projected
    feed-forward     scores softmax(router h) over experts and identity experts; the `top` largest of scores + correction; weights
                     the chosen scores over their sum; expert e: down(g sigmoid(1.702 g) (u + 1)), g = min(gate h, limit),
                     u = clamp(up h, -limit, limit); an identity expert gives h; a shared expert of the same form is added
    head             final norm, logits = head x
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, gain, groups, eps):
    n, width = x.shape
    return rms(x.view(n, groups, width // groups), eps).reshape(n, width) * gain


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def short_conv(x, taps, bias):
    """x [n, channels], taps [channels, T]: y[t] = bias + sum_i taps[:, T - 1 - i] * x[t - i], zeros before the start."""
    n, T = x.shape[0], taps.shape[1]
    padded = torch.cat([x.new_zeros((T - 1, x.shape[1])), x], dim=0)
    y = bias.expand(n, -1).clone()
    for i in range(T):
        y = y + padded[T - 1 - i:T - 1 - i + n] * taps[:, T - 1 - i]
    return y


def block_gate(u, mats, bias):
    """sigmoid of a block-diagonal map: mats [B, s, s] ([out, in]), bias [B, s], u [n, B * s]."""
    B, s, _ = mats.shape
    parts = [u[:, b * s:(b + 1) * s] @ mats[b].T + bias[b] for b in range(B)]
    return torch.sigmoid(torch.cat(parts, dim=-1))


def lru(u, r, i, lam):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u from S = 0; all rows."""
    log_a = -8.0 * r * torch.nn.functional.softplus(lam)
    a = torch.exp(log_a)
    add = torch.sqrt(-torch.expm1(2 * log_a)) * i * u
    S = torch.zeros_like(u[0])
    out = torch.empty_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + add[t]
        out[t] = S
    return out


def rglru(m, w, p, h):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = short_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = block_gate(u, w[p + "ra"], w[p + "ra.b"])
    i = block_gate(u, w[p + "ri"], w[p + "ri.b"])
    return (lru(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


def temperature(positions, every, coef, dtype):
    steps = torch.div(positions + 1, every, rounding_mode="floor").to(dtype)
    return 1 + coef * torch.log(steps + 1)


def attention(m, w, p, h, eps):
    n, H, D = h.shape[0], m["heads"], m["dim"]
    G, V, scale = m.get("kv_heads", H), m.get("vdim", D), float(m.get("scale", D ** -0.5))
    q = rms((h @ w[p + "q"].T).view(n, H, D), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T).view(n, G, D), eps) * w[p + "k.norm"]
    v = rms((h @ w[p + "v"].T).view(n, G, V), eps)
    if m.get("q_temp"):
        q = q * temperature(torch.arange(n), int(m["q_temp"]["every"]), float(m["q_temp"]["coef"]), h.dtype)[:, None, None]
    seen = torch.arange(n)[:, None] >= torch.arange(n)[None, :]
    out = []
    for a in range(H):
        s = (q[:, a] @ k[:, a // (H // G)].T) * scale
        out.append(torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, a // (H // G)])
    return torch.cat(out, dim=-1) @ w[p + "o"].T


def time_mix(r, k, v, decay, u):
    """r, k, decay [n, H, D], v [n, H, V], u [H, D]: the recurrence with a bonus for the token's own key and value."""
    n, H, D = r.shape
    out = torch.empty(n, H, v.shape[-1], dtype=r.dtype)
    for a in range(H):
        S = r.new_zeros((D, v.shape[-1]))
        for t in range(n):
            kv = torch.outer(k[t, a], v[t, a])
            out[t, a] = (S + u[a][:, None] * kv).T @ r[t, a]
            S = decay[t, a][:, None] * S + kv
    return out


def time_mixing(m, w, p, h, eps):
    n, H, D = h.shape[0], m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)

    def blend(s):
        return h + (before - h) * w[p + "mu." + s]
    r = (blend("r") @ w[p + "r"].T).view(n, H, D)
    k = (blend("k") @ w[p + "k"].T).view(n, H, D)
    v = (blend("v") @ w[p + "v"].T).view(n, H, D)
    gate = silu(blend("g") @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(blend("w") @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(n, H, D)
    o = rms(time_mix(r, k, v, decay, w[p + "u"]), eps).reshape(n, H * D)
    return (o * w[p + "norm"] * gate) @ w[p + "o"].T


def parallel(m, w, p, h, eps):
    return float(m.get("left_scale", 1.0)) * attention(m["left"], w, p + "left.", h, eps) + \
        float(m.get("right_scale", 1.0)) * time_mixing(m["right"], w, p + "right.", h, eps)


def expert(w, p, h, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(mlp, w, p, h):
    """(chosen [n, top], their weights [n, top])."""
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    idx = torch.topk(s + w[p + "correction"], int(mlp["router"]["top"]), dim=-1).indices
    val = torch.gather(s, 1, idx)
    return idx, val / (val.sum(-1, keepdim=True) + 1e-20)


def experts_ff(mlp, w, p, h):
    idx, val = route(mlp, w, p, h)
    E, limit = int(mlp["router"]["experts"]), float(mlp["expert"]["limit"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(idx[t].tolist(), val[t]):
            out[t] = out[t] + s * (h[t] if e >= E else expert(w, f"{p}e{e}.", h[t][None], limit)[0])
    if mlp.get("shared"):
        out = out + expert(w, p + "shared.", h, float(mlp["shared"]["limit"]))
    return out


def forward(cfg, w, tokens, layers_out=None):
    """Logits [n, vocab] of one whole sequence; `layers_out`, a list, receives the residual after every layer."""
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"].get("groups", 1))
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][tokens] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        h = group_norm(x, w[f"l{i}.norm1"], groups, eps)
        add = rglru(m, w, p, h) if layer["type"] == "rglru" else parallel(m, w, p, h, eps)
        if layer.get("mlp") is not None:
            add = add + experts_ff(layer["mlp"], w, f"l{i}.mlp.", group_norm(x, w[f"l{i}.norm2"], groups, eps))
        x = x + add
        if layers_out is not None:
            layers_out.append(x.clone())
    return group_norm(x, w["final.norm"], groups, eps) @ w["head"].T
