"""Small model configurations and weights for the hybrid-decoder tests, and the plain implementation's answers for them."""
import torch


def lightning(heads=2, dim=24, vdim=16, decay=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.35 + 0.6 * i / heads for i in range(heads)]}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=3):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads=6, kv_heads=2, dim=24, vdim=16, scale=0.31, bias_max=70, v_mix=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "v_mix": v_mix}}


def config(layers, width=56, vocab=73, ff=88, eps=3e-5, scale=1.7, mult=0.6):
    out = []
    for L in layers:
        L = dict(L)
        L.setdefault("mlp", {"kind": "dense", "ff": ff})
        out.append(L)
    return {"architecture": "Gopunex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "residual_mult": mult,
            "layers": out}


CONFIGS = {
    "all": config([lightning(), delta(), attention(), delta(heads=3, kv_heads=3), attention(), lightning(heads=1)]),
    "attention_first": config([attention(v_mix=False), attention(heads=4, kv_heads=4, dim=40), attention(heads=2, kv_heads=2, dim=8, vdim=32), attention(vdim=32)], width=64),
    "no_mlp": config([dict(delta(conv=1), mlp=None), lightning(heads=3, dim=8, vdim=40), dict(attention(heads=1, kv_heads=1), mlp=None)], width=48, mult=1.0, scale=1.0),
    "odd_sizes": config([attention(heads=3, kv_heads=1, dim=10, vdim=7), delta(heads=2, kv_heads=1, dim=5, vdim=9, conv=4), lightning(heads=3, dim=6, vdim=11)],
                        width=30, vocab=41, ff=34),
    "wide_heads": config([delta(heads=2, kv_heads=2, dim=72, vdim=136, conv=2), attention(heads=9, kv_heads=1, dim=136, vdim=96, bias_max=300),
                          lightning(heads=2, dim=160, vdim=48)], width=72),
    "narrow_window": config([attention(heads=2, kv_heads=1, dim=16, vdim=16, bias_max=9), delta(heads=1, kv_heads=1, dim=32, vdim=32, conv=6)], width=32),
}


def weights(cfg, seed=0, buckets=12, rank=11):
    """bf16 tensors whose gates, decays, biases and mixing factors are far from trivial."""
    import mixers
    g = torch.Generator().manual_seed(seed)
    from hybrid_model import tensor_shapes
    shapes = tensor_shapes(cfg)
    for i, L in enumerate(cfg["layers"]):
        mc, p = L["mixer"], f"l{i}.mix."
        if L["type"] == "channel_delta":
            shapes.update({p + k: s for k, s in mixers.ChannelDelta.shapes(mc, cfg["width"], rank).items()})
        if L["type"] == "attention":
            shapes.update({p + k: s for k, s in mixers.BiasAttention.shapes(mc, cfg["width"], buckets).items()})
    out = {}
    for name, shape in shapes.items():
        t = torch.randn(shape, generator=g)
        if name.endswith((".mix.norm", ".q.norm", ".k.norm")):
            t = 1 + 0.3 * t
        elif name.endswith("A_log"):
            t = torch.rand(shape, generator=g) * 3 - 2
        elif name.endswith("vmix"):
            t = torch.rand(shape, generator=g) * 0.6 + 0.2
        elif name.endswith((".rel", "dt_bias")):
            t = 1.5 * t
        elif name.endswith(".conv"):
            t = 0.7 * t
        elif len(shape) == 2 and name != "embed":
            t = 1.5 * t * shape[1] ** -0.5
        elif len(shape) == 1:
            t = 0.3 * t
        out[name] = t.to(torch.bfloat16)
    return out


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist()


def expected(cfg, W, toks, layers_out=None):
    import gopunex_oracle as O
    return O.forward(cfg, {k: v.double() for k, v in W.items()}, toks, layers_out)


def error(got, want):
    """Largest row difference (means removed), in units of the spread of the expected logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt().max() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()).item()


TOL = {torch.float32: 3e-5, torch.bfloat16: 0.06}
