"""Plain CPU restatement of the Gopunex decoder: one function per mechanism, whole sequences, no cache, no chunking.

Test infrastructure only (imported by tests/, never by the package). Everything runs in the dtype of the tensors it is given
(float32 or float64), token by token where the mechanism is a recurrence and with full score matrices where it is attention,
so that no block, window, portion or reuse of state exists here that could hide a fault of the product path.

A model is (cfg, W): cfg the parsed configuration dictionary, W a dictionary of tensors by their stored names.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


def mlp_dense(h, W, p):
    return squared_relu(h @ W[p + "up"].T) @ W[p + "down"].T


def causal_conv(x, taps):
    """x [T, C], taps [C, n]: y_t = sum_i taps[:, n - 1 - i] x_{t - i}, zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for i in range(n):
            if t - i >= 0:
                y[t] = y[t] + taps[:, n - 1 - i] * x[t - i]
    return y


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def decayed_linear_attention(q, k, v, decay):
    """One head: q, k [T, dk], v [T, dv], scalar decay. S <- decay S + k v^T, o = S^T q."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay * S + k[t][:, None] * v[t][None, :]
        out.append(S.T @ q[t])
    return torch.stack(out)


def lightning(h, W, p, mc, eps):
    H, dk, dv = mc["heads"], mc["dim"], mc["vdim"]
    q, k, v = (silu(h @ W[p + n].T) for n in ("q", "k", "v"))
    o = [decayed_linear_attention(q[:, i * dk:(i + 1) * dk], k[:, i * dk:(i + 1) * dk], v[:, i * dv:(i + 1) * dv], mc["decay"][i])
         for i in range(H)]
    o = rms(torch.cat(o, -1), eps) * W[p + "norm"]
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def channel_decay(h, W, p, heads, dim):
    """g [T, heads, dim] in (0, 1): the factor on every key channel of the state."""
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]
    a = torch.exp(W[p + "A_log"])
    return torch.exp(-a[None, :, None] * softplus(z).view(-1, heads, dim))


def gated_delta(q, k, v, g, beta):
    """One head: decay the rows of S, write beta (v - S^T k) along k, read with q."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + k[t][:, None] * u[None, :]
        out.append(S.T @ q[t])
    return torch.stack(out)


def channel_delta(h, W, p, mc, eps):
    H, G, dk, dv = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
    T = h.shape[0]
    q, k, v = (silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.view(T, G, dk)) * dk ** -0.5
    k = unit(k.view(T, G, dk))
    v = v.view(T, H, dv)
    beta = sigmoid(h @ W[p + "b"].T)
    g = channel_decay(h, W, p, H, dk)
    gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T).view(T, H, dv)
    o = torch.stack([gated_delta(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i], beta[:, i]) for i in range(H)], 1)
    o = rms(o, eps) * W[p + "norm"] * gate
    return o.reshape(T, H * dv) @ W[p + "o"].T


def distance_bucket(n, B, D):
    half = B // 2
    if n < half:
        return n
    return min(B - 1, half + math.floor(math.log(n / half) / math.log(D / half) * (B - half)))


def distance_bias(rel, D, T):
    """bias [H, T, T] for query i, key j <= i (0 elsewhere) from the table rel [B, H]."""
    B = rel.shape[0]
    row = torch.tensor([distance_bucket(n, B, D) for n in range(T)])
    i = torch.arange(T)
    dist = (i[:, None] - i[None, :]).clamp(min=0)
    return rel[row[dist]].permute(2, 0, 1)


def softmax_off_by_one(s, mask):
    """Softmax whose denominator has one added (a sink of score 0 without a value)."""
    s = s.masked_fill(~mask, float("-inf"))
    m = torch.clamp(s.max(-1, keepdim=True).values, min=0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention(h, W, p, mc, eps, v_first):
    """Returns (output, values of this layer after mixing, or the unmixed ones if it is the first mixing layer)."""
    H, G, dk, dv = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
    T = h.shape[0]
    q, k, v = (h @ W[p + n].T + W[p + n + ".b"] for n in ("q", "k", "v"))
    q = (rms(q, eps) * W[p + "q.norm"]).view(T, H, dk)
    k = (rms(k, eps) * W[p + "k.norm"]).view(T, G, dk)
    if mc.get("v_mix") and v_first is not None:
        lam = W[p + "vmix"]
        v = (1 - lam) * v + lam * v_first
    vh = v.view(T, G, dv)
    bias = distance_bias(W[p + "rel"], mc["bias_max"], T)
    i = torch.arange(T)
    mask = i[:, None] >= i[None, :]
    out = []
    for a in range(H):
        b = a // (H // G)
        s = (q[:, a] @ k[:, b].T) * mc["scale"] + bias[a]
        out.append(softmax_off_by_one(s, mask) @ vh[:, b])
    return torch.cat(out, -1) @ W[p + "o"].T, v


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab]; appends the residual stream after every layer to layers_out if given."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    v_first = None
    for i, L in enumerate(cfg["layers"]):
        p, mc = f"l{i}.", L["mixer"]
        if L["type"] == "lightning":
            y = lightning(x, W, p + "mix.", mc, eps)
        elif L["type"] == "channel_delta":
            y = channel_delta(x, W, p + "mix.", mc, eps)
        else:
            y, v = attention(x, W, p + "mix.", mc, eps, v_first)
            if mc.get("v_mix") and v_first is None:
                v_first = v
        x = x + m * rms(y, eps) * (1 + W[p + "norm1"])
        if L["mlp"] is not None:
            x = x + m * rms(mlp_dense(x, W, p + "mlp."), eps) * (1 + W[p + "norm2"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * (1 + W["final.norm"])) @ W["head"].T
