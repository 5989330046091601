"""Small Latodra configurations and weights for the tests, and the plain implementation's answers for them."""
import torch

from hybrid_cases import TOL, error, tokens  # noqa: F401


def rot(dims, base=200.0, scaling=(3.0, 24, 5.0, 0.6)):
    out = {"base": base, "dims": dims}
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def turned(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=72, q_rank=56, scale=0.21, turn=None, **kw):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                  "scale": scale, "rot": turn or rot(rot_dim)}, **kw}


def plain(heads=5, dim=40, vdim=16, kv_rank=48, q_rank=24, scale=0.19, **kw):
    return {"type": "latent_attention_2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}, **kw}


def config(layers, width=64, vocab=83, ff=96, eps=2e-4, loop=None):
    out = [{"mlp": {"kind": "dense", "ff": ff}, **L} for L in layers]
    c = {"architecture": "Latodra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": out}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    "loop_inside": config([plain(), turned(), plain(heads=2, mlp=None), turned(heads=1)], loop=(1, 3, 3)),
    "loop_first": config([turned(turn=rot(16, 1e4, None)), plain(heads=16, dim=8)], width=48, loop=(0, 1, 2)),
    "one_pass": config([turned(heads=8, rot_dim=32, dim=8), turned(q_rank=8)], width=40, loop=(0, 2, 1)),
    "no_loop": config([turned(mlp=None), plain(mlp=None), plain(mlp={"kind": "dense", "ff": 40})], width=88, vocab=45),
    "odd_sizes": config([turned(dim=10, rot_dim=6, vdim=7, kv_rank=21, q_rank=13), plain(heads=3, dim=5, vdim=9, kv_rank=11, q_rank=17)], width=30, ff=34, vocab=41, loop=(1, 2, 2)),
    "part_turned": config([turned(heads=2, rot_dim=24, turn=rot(10, 50.0))], width=32),
    "large_heads": config([turned(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=96, scale=0.06), plain(heads=20, dim=64, vdim=64, kv_rank=320, q_rank=40, scale=0.11)], width=72, loop=(0, 2, 2)),
    "wide_heads": config([turned(heads=2, dim=200, rot_dim=40, vdim=144, kv_rank=136, scale=0.07), plain(heads=1, dim=16, vdim=96, kv_rank=640)], width=56),
}


def weights(cfg, seed=0):
    """bf16 tensors whose norms, gates, sinks and scales are far from trivial."""
    from hybrid_model import tensor_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if "norm" in name:
            t = 1 + 0.3 * t
        elif name.endswith((".ls1", ".ls2")):
            t = 0.6 + 0.3 * t
        elif name.endswith(".sink"):
            t = 1.5 * t
        elif name == "loop.step":
            t = 0.7 * t
        elif name.endswith((".uk", ".uq", ".g")):
            t = 1.5 * t * shape[1] ** -0.5
        elif name != "embed":
            t = t * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    out["embed"] = out["embed"] * 0.3
    return out


def expected(cfg, W, toks, layers_out=None):
    import latodra_oracle as O
    return O.forward(cfg, {k: v.double() for k, v in W.items()}, toks, layers_out)


def one_key_counts(marked):
    """(config, weights) of one layer whose queries look for the token `marked` alone: its score is about 12, all others are near 0."""
    cfg = config([turned(heads=1, dim=16, rot_dim=8, vdim=16, kv_rank=16, q_rank=16, scale=1.0)], width=32, vocab=40)
    W = weights(cfg, 5)
    for k in ("embed.norm", "l0.norm1", "l0.mix.dq.norm", "l0.mix.dkv.norm"):
        W[k] = torch.ones_like(W[k])
    E = W["embed"]
    E[:, 0] = 0
    E[marked] = 0
    E[marked, 0] = 6
    E[:, 1] = 1
    for k in ("dkv", "uk", "dq", "uq"):             # column / row 0 carries the mark, or the constant that queries it
        m = W["l0.mix." + k]
        m[1:] *= 0.3
        m[0] = 0
        m[0, 1 if k == "dq" else 0] = 1
        if k == "dkv":
            m[1:, 0] = 0
    W["l0.mix.sink"] = torch.full_like(W["l0.mix.sink"], -30)
    return cfg, W
