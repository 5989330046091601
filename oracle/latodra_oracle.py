"""Plain CPU restatement of the Latodra decoder: one function per mechanism, whole sequences, no cache, no latent-space shortcut.

Test infrastructure only (imported by tests/, never by the package). Everything runs in the dtype of the tensors it is given (float32 or
float64) with full score matrices: keys and values of every head are formed from the latents, every query meets every key, so that no tile,
portion, absorbed projection or reuse of state exists here that could hide a fault of the product path.

A model is (cfg, W): cfg the parsed configuration dictionary, W a dictionary of tensors by their stored names.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def mlp_dense(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def yarn_frequencies(rot):
    """(frequencies of the dims / 2 pairs, factor on cos and sin) of a rotation entry; without 'scaling' the plain ones and 1."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return f, 1.0

    def place(turns):       # the (fractional) dimension whose pair makes `turns` turns over the original length
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(place(sc["fast"])), 0), min(math.ceil(place(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, ..., D]: pairs (2 i, 2 i + 1) of the first `dims` of D turned by position * frequency, the rest unchanged."""
    f, m = yarn_frequencies(rot)
    y = x.clone()
    for t, p in enumerate(positions):
        for i, fi in enumerate(f):
            c, s = m * math.cos(p * fi), m * math.sin(p * fi)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            y[t, ..., 2 * i] = u * c - v * s
            y[t, ..., 2 * i + 1] = v * c + u * s
    return y


def causal_softmax(s, sink=None):
    """Rows of s [T, T] over the keys j <= i; the sink is one more term of the denominator."""
    T = s.shape[0]
    s = s.masked_fill(~torch.tril(torch.ones(T, T, dtype=torch.bool)), float("-inf"))
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink)
    e = torch.exp(s - m)
    d = e.sum(-1, keepdim=True)
    if sink is not None:
        d = d + torch.exp(sink - m)
    return e / d


def latent_attention(h, W, p, mc, eps):
    """Both kinds: a rotated part if the entry has 'rot_dim', a sink and an output gate if the tensors are there."""
    H, dn, dr, dv, R = mc["heads"], mc["dim"], mc.get("rot_dim", 0), mc["vdim"], mc["kv_rank"]
    T = h.shape[0]
    q = ((rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, dn + dr)
    low = h @ W[p + "dkv"].T
    c = rms(low[:, :R], eps) * W[p + "dkv.norm"]
    k = (c @ W[p + "uk"].T).view(T, H, dn)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    if dr:
        at = range(T)
        qr, kr = rotate(q[:, :, dn:], at, mc["rot"]), rotate(low[:, R:], at, mc["rot"])
    out = []
    for a in range(H):
        s = q[:, a, :dn] @ k[:, a].T
        if dr:
            s = s + qr[:, a] @ kr.T
        sink = W[p + "sink"][a] if p + "sink" in W else None
        out.append(causal_softmax(s * mc["scale"], sink) @ v[:, a])
    o = torch.cat(out, -1)
    if p + "g" in W:
        o = o * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def layer(x, W, p, L, eps):
    y = latent_attention(rms(x, eps) * W[p + "norm1"], W, p + "mix.", L["mixer"], eps)
    x = x + rms(y, eps) * W[p + "norm1b"] * W[p + "ls1"]
    if L["mlp"] is not None:
        y = mlp_dense(rms(x, eps) * W[p + "norm2"], W, p + "mlp.")
        x = x + rms(y, eps) * W[p + "norm2b"] * W[p + "ls2"]
    return x


def layer_runs(cfg):
    """[(layer, pass or None if this run opens no pass)] in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab]; appends the residual stream after every layer run to layers_out if given."""
    eps = cfg["norm"]["eps"]
    e = rms(W["embed"][torch.as_tensor(tokens, dtype=torch.long)], eps) * W["embed.norm"]
    x = e
    for i, t in layer_runs(cfg):
        if t is not None:
            if t > 0:
                x = x + e
            x = x + W["loop.step"][t]
        x = layer(x, W, f"l{i}.", cfg["layers"][i], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * W["final.norm"]) @ W["embed"].T
