"""Token mixers and feed-forwards of the hybrid decoders. Each mixer is built from its configuration entry and the stored tensors of one
layer, declares the per-sequence state it keeps, and runs a portion of n tokens for B sequences from that state. The kernels are
sequence-length agnostic, so one code path serves whole prompts, portions of prompts and single tokens.

    MIXERS['lightning']       decayed linear attention, RMS norm over all heads, sigmoid gate
    MIXERS['channel_delta']   gated delta rule with one decay per head and key channel, short convolutions on q, k, v
    MIXERS['attention']       softmax attention with a learned bias by distance, a sink, whole-projection q / k norm and value mixing
    MIXERS['latent_attention']    attention over a cached low-rank latent per token, rotary positions on a part of every head, learned sinks
    MIXERS['latent_attention_2']  the same without positions and sinks, with an output gate
    MLPS['relu2']             W_down relu(W_up x)^2
    MLPS['gated_gelu']        W_down (gelu_tanh(W_gate x) * W_up x)
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

import seq_ops as S


@dataclass
class StepContext:
    """What the mixers of one step share."""
    B: int
    n: int
    pos: torch.Tensor              # int32 [1], position of the first token (device)
    host_pos: int                  # the same on the host; -1 in a step that is captured for replay
    eps: float
    v_first: torch.Tensor | None = None    # values of the first mixing layer, [B * n, width]


@dataclass
class StateSpec:
    """A tensor a layer keeps per sequence: shape without the leading batch; 'T_max' stands for the cache capacity. Tensors that must
    start at zero are cleared when a sequence starts."""
    shape: tuple
    fp32: bool = False
    zero: bool = False


class Loader:
    """Tensors of one layer by short name, moved to the device in the requested type."""

    def __init__(self, tensors, prefix: str, dtype: torch.dtype, device):
        self.t, self.prefix, self.dtype, self.device = tensors, prefix, dtype, device

    def has(self, name: str) -> bool:
        return self.prefix + name in self.t

    def raw(self, name: str, shape=None) -> torch.Tensor:
        t = self.t[self.prefix + name]
        if shape is not None and tuple(t.shape) != tuple(shape):
            raise ValueError(f"tensor {self.prefix + name}: shape {tuple(t.shape)}, expected {tuple(shape)}")
        return t

    def mat(self, name: str, shape=None) -> torch.Tensor:
        return self.raw(name, shape).to(self.device, self.dtype).contiguous()

    def f32(self, name: str, shape=None) -> torch.Tensor:
        return self.raw(name, shape).to(self.device, torch.float32).contiguous()

    def stack(self, names, shapes, biases: bool = False):
        """The named matrices one under the other (stack_rows). Returns (weight, bias or None, first row of each)."""
        w, offs = stack_rows([self.mat(name, shape) for name, shape in zip(names, shapes)])
        if not biases:
            return w, None, offs
        b = torch.zeros(w.shape[0], dtype=self.dtype, device=self.device)
        for name, shape, o in zip(names, shapes, offs):
            b[o:o + shape[0]] = self.mat(name + ".b", (shape[0],))
        return w, b, offs


def stack_rows(mats):
    """Matrices one under the other, each starting at a multiple of eight rows (zero rows between), so that one Linear serves all of them
    and every slice of its output starts on 16 bytes. Returns (weight, first row of each)."""
    offs, at = [], 0
    for m in mats:
        offs.append(at)
        at += (m.shape[0] + 7) // 8 * 8
    w = torch.zeros(at, mats[0].shape[1], dtype=mats[0].dtype, device=mats[0].device)
    for m, o in zip(mats, offs):
        w[o:o + m.shape[0]] = m
    return w, offs


CHUNK_FROM = 64     # portions of at least this many tokens take the chunked recurrence (bf16 models)


def _chunked(x: torch.Tensor, n: int) -> bool:
    return n >= CHUNK_FROM and x.dtype == torch.bfloat16


class Lightning:
    """Per head S <- decay S + k v^T, o = S^T q, with q, k, v = silu of their projections."""

    def __init__(self, mc: dict, L: Loader, width: int):
        self.H, self.dk, self.dv = mc["heads"], mc["dim"], mc["vdim"]
        if len(mc["decay"]) != self.H:
            raise ValueError(f"{len(mc['decay'])} decays for {self.H} heads")
        qk, v = self.H * self.dk, self.H * self.dv
        self.w_in, _, self.off = L.stack(("q", "k", "v", "g"), ((qk, width), (qk, width), (v, width), (v, width)))
        self.w_out, self.norm = L.mat("o", (width, v)), L.f32("norm", (v,))
        self.decay = torch.tensor(mc["decay"], dtype=torch.float32, device=L.device)

    @staticmethod
    def shapes(mc: dict, width: int) -> dict:
        qk, v = mc["heads"] * mc["dim"], mc["heads"] * mc["vdim"]
        return {"q": (qk, width), "k": (qk, width), "v": (v, width), "g": (v, width), "o": (width, v), "norm": (v,)}

    def state_spec(self):
        return {"S": StateSpec((self.H, self.dk, self.dv), fp32=True, zero=True)}

    def forward(self, x: torch.Tensor, st: dict, ctx: StepContext) -> torch.Tensor:
        qk, v, (oq, ok, ov, og) = self.H * self.dk, self.H * self.dv, self.off
        p = S.linear(x, self.w_in)
        o = S.decay_attention(p[:, oq:oq + qk], p[:, ok:ok + qk], p[:, ov:ov + v], self.decay, st["S"], ctx.B, ctx.n, self.H, self.dk, self.dv,
                              _chunked(x, ctx.n))
        return S.linear(S.norm_gate(o, p[:, og:og + v], self.norm, ctx.eps, 1), self.w_out)


class ChannelDelta:
    """Gated delta rule; the decay is a vector over the key channels of every head."""

    def __init__(self, mc: dict, L: Loader, width: int):
        self.H, self.G, self.dk, self.dv = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
        self.taps = mc["conv"]
        if self.H % self.G:
            raise ValueError(f"{self.H} heads over {self.G} key heads")
        qk, v = self.G * self.dk, self.H * self.dv
        ra, rg = L.raw("a1").shape[0], L.raw("g1").shape[0]
        self.w_in, _, self.off = L.stack(("q", "k", "v", "b", "a1", "g1"), ((qk, width), (qk, width), (v, width), (self.H, width), (ra, width), (rg, width)))
        self.ra, self.rg = ra, rg
        self.w_a2, self.w_g2 = L.mat("a2", (self.H * self.dk, ra)), L.mat("g2", (v, rg))
        self.conv = torch.cat([L.f32(n + ".conv", (c, self.taps)) for n, c in (("q", qk), ("k", qk), ("v", v))]).contiguous()
        self.A_log, self.dt_bias = L.f32("A_log", (self.H,)), L.f32("dt_bias", (self.H * self.dk,))
        self.norm, self.w_out = L.f32("norm", (self.dv,)), L.mat("o", (width, v))

    @staticmethod
    def shapes(mc: dict, width: int, rank: int | None = None) -> dict:
        H, dk, dv = mc["heads"], mc["dim"], mc["vdim"]
        qk, v, r = mc["kv_heads"] * dk, H * dv, rank or dv
        out = {"q": (qk, width), "k": (qk, width), "v": (v, width), "b": (H, width), "A_log": (H,), "norm": (dv,), "a1": (r, width),
               "a2": (H * dk, r), "dt_bias": (H * dk,), "g1": (r, width), "g2": (v, r), "o": (width, v)}
        out.update({n + ".conv": (out[n][0], mc["conv"]) for n in ("q", "k", "v")})
        return out

    def state_spec(self):
        spec = {"S": StateSpec((self.H, self.dk, self.dv), fp32=True, zero=True)}
        if self.taps > 1:
            spec["conv"] = StateSpec((self.taps - 1, self.conv.shape[0]), zero=True)
        return spec

    def forward(self, x: torch.Tensor, st: dict, ctx: StepContext) -> torch.Tensor:
        oq, ok, ov, ob, oa, og = self.off
        p = S.linear(x, self.w_in)
        a = S.linear(p[:, oa:oa + self.ra], self.w_a2)
        gate = S.linear(p[:, og:og + self.rg], self.w_g2)
        q, k, v, logg, beta = S.delta_prep(p, (oq, ok, ov, ob), a, self.conv, self.A_log, self.dt_bias, st.get("conv"), ctx.B, ctx.n, self.H, self.G,
                                           self.dk, self.dv, self.dk ** -0.5)
        o = S.delta_rule(q, k, v, logg, beta, st["S"], ctx.B, ctx.n, self.H, self.G, self.dk, self.dv, _chunked(x, ctx.n))
        return S.linear(S.norm_gate(o, gate, self.norm, ctx.eps, self.H), self.w_out)


def distance_bucket(n: int, buckets: int, bias_max: int) -> int:
    """Bucket of distance n: the first half of the buckets one distance each, the rest spaced evenly in the logarithm up to bias_max."""
    half = buckets // 2
    if n < half:
        return n
    if half < 1 or bias_max <= half:
        return buckets - 1
    at = math.log(n / half) / math.log(bias_max / half) * (buckets - half)
    return min(buckets - 1, half + math.floor(at + 1e-9))     # a distance on a bucket's border belongs to the bucket it opens


def distance_table(rel: torch.Tensor, bias_max: int) -> torch.Tensor:
    """rel [buckets, H] -> fp32 [H, D]: the bias of distances 0 .. D - 1, the last entry holding for all beyond."""
    B = rel.shape[0]
    row = [distance_bucket(0, B, bias_max)]
    while row[-1] < B - 1:
        row.append(distance_bucket(len(row), B, bias_max))
    return rel.float()[torch.tensor(row, device=rel.device)].T.contiguous()


class BiasAttention:
    """Softmax attention with positions only in a learned bias by distance."""

    def __init__(self, mc: dict, L: Loader, width: int):
        self.H, self.G, self.dk, self.dv, self.scale = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"], mc["scale"]
        if self.H % self.G:
            raise ValueError(f"{self.H} heads over {self.G} key / value heads")
        q, k, v = self.H * self.dk, self.G * self.dk, self.G * self.dv
        self.w_in, self.b_in, self.off = L.stack(("q", "k", "v"), ((q, width), (k, width), (v, width)), biases=True)
        self.wq, self.wk = L.f32("q.norm", (q,)), L.f32("k.norm", (k,))
        self.bias = S.DistanceBias.from_distances(distance_table(L.f32("rel"), mc["bias_max"]))
        if self.bias.top.numel() != self.H:
            raise ValueError(f"{L.prefix}rel holds {self.bias.top.numel()} heads, expected {self.H}")
        self.v_mix = bool(mc.get("v_mix", False))
        self.mix = L.f32("vmix").reshape(1) if self.v_mix and L.has("vmix") else None
        self.w_out = L.mat("o", (width, self.H * self.dv))

    @staticmethod
    def shapes(mc: dict, width: int, buckets: int = 32) -> dict:
        q, k, v = mc["heads"] * mc["dim"], mc["kv_heads"] * mc["dim"], mc["kv_heads"] * mc["vdim"]
        return {"q": (q, width), "q.b": (q,), "k": (k, width), "k.b": (k,), "v": (v, width), "v.b": (v,), "q.norm": (q,), "k.norm": (k,),
                "rel": (buckets, mc["heads"]), "vmix": (), "o": (width, mc["heads"] * mc["vdim"])}

    def state_spec(self):
        return {"k": StateSpec(("T_max", self.G * self.dk)), "v": StateSpec(("T_max", self.G * self.dv))}

    def forward(self, x: torch.Tensor, st: dict, ctx: StepContext) -> torch.Tensor:
        p = S.linear(x, self.w_in, self.b_in)
        first = self.v_mix and ctx.v_first is None
        if first:
            ctx.v_first = torch.empty(ctx.B * ctx.n, self.G * self.dv, dtype=p.dtype, device=p.device)
        elif self.v_mix and (self.mix is None or ctx.v_first.shape[1] != self.G * self.dv):
            raise ValueError("value mixing needs the weight 'vmix' and the value width of the first mixing layer")
        q = S.attn_prep(p, self.off, self.wq, self.wk, self.mix if self.v_mix and not first else None, ctx.v_first if self.v_mix else None, first,
                        st["k"], st["v"], ctx.pos, ctx.B, ctx.n, ctx.eps)
        o = S.attention_bias(q, st["k"], st["v"], self.bias, ctx.pos, ctx.host_pos, ctx.B, ctx.n, self.H, self.G, self.dk, self.dv, self.scale, True)
        return S.linear(o, self.w_out)


def rotary_frequencies(rot: dict):
    """(frequency of every pair, factor on cos and sin) of a rotation entry: base^(-2 i / dims), and with 'scaling' (YaRN) a blend of
    that and the same over 'factor', by how often a pair turns over the 'original' length: all of it kept above 'fast' turns, all divided
    below 'slow'."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    if dims % 2:
        raise ValueError(f"rotation of {dims} dimensions")
    freq = [math.pow(base, -2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return freq, 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), dims - 1)
    for i, f in enumerate(freq):
        slow = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freq[i] = f * (slow / sc["factor"] + 1.0 - slow)
    return freq, 0.1 * math.log(sc["factor"]) + 1.0


class LatentAttention:
    """Attention whose keys and values are products of one normed latent per token, which is all the cache holds (beside one rotated key
    part that the heads share). Queries pass through a latent of their own.

    Two forms give the same result. *Absorbed*: the key matrix is applied to the queries and the value matrix to the output, and all heads
    attend to the cached rows themselves: the work of a token grows with the latent's size, nothing is formed per cached token. It serves
    single tokens and short portions. *Expanded*: keys and values of all cached tokens are formed once per portion and ordinary attention
    runs on them: fewer products per pair of tokens, for long portions."""
    ROTATED, SINK, GATE = True, True, False

    def __init__(self, mc: dict, L: Loader, width: int):
        self.H, self.dn, self.dv = mc["heads"], mc["dim"], mc["vdim"]
        self.dr = mc["rot_dim"] if self.ROTATED else 0
        self.rq, self.R, self.scale = mc["q_rank"], mc["kv_rank"], mc["scale"]
        H, dn, dr, dv, R = self.H, self.dn, self.dr, self.dv, self.R
        # the latent and the key part are separate slices of the projection, so that each starts on 16 bytes
        dkv = L.mat("dkv", (R + dr, width))
        parts = {"dq": L.mat("dq", (self.rq, width)), "c": dkv[:R], "r": dkv[R:]}
        if self.GATE:
            parts["g"] = L.mat("g", (H * dv, width))
        self.w_in, at = stack_rows(list(parts.values()))
        self.off = dict(zip(parts, at))
        self.wq, self.wc = L.f32("dq.norm", (self.rq,)), L.f32("dkv.norm", (R,))
        self.w_uq = L.mat("uq", (H * (dn + dr), self.rq))
        uk, uv = L.mat("uk", (H * dn, R)), L.mat("uv", (H * dv, R))
        self.w_kv, (_, self.off_v) = stack_rows([uk, uv])                        # expanded: keys and values of a latent
        self.w_qk = uk.view(H, dn, R).transpose(1, 2).contiguous()               # absorbed: per head, queries -> latent space
        self.w_ov = uv.view(H, dv, R)                                            #           per head, latent space -> values
        self.w_out = L.mat("o", (width, H * dv))
        self.sinks = L.f32("sink", (H,)) if self.SINK else None
        self.rot = None
        if dr:
            freq, m = rotary_frequencies(mc["rot"])
            if 2 * len(freq) > dr:
                raise ValueError(f"rotation of {2 * len(freq)} dimensions in a part of {dr}")
            self.rot = S.Rotation(torch.tensor(freq, dtype=torch.float64, device=L.device), m)

    @classmethod
    def shapes(cls, mc: dict, width: int) -> dict:
        H, dn, dv, R, rq = mc["heads"], mc["dim"], mc["vdim"], mc["kv_rank"], mc["q_rank"]
        dr = mc["rot_dim"] if cls.ROTATED else 0
        out = {"dq": (rq, width), "dq.norm": (rq,), "uq": (H * (dn + dr), rq), "dkv": (R + dr, width), "dkv.norm": (R,), "uk": (H * dn, R),
               "uv": (H * dv, R), "o": (width, H * dv)}
        if cls.SINK:
            out["sink"] = (H,)
        if cls.GATE:
            out["g"] = (H * dv, width)
        return out

    def state_spec(self):
        spec = {"c": StateSpec(("T_max", self.R))}
        if self.dr:
            spec["kr"] = StateSpec(("T_max", self.dr))
        return spec

    def decode_weights(self):
        """Matrices that a one-token step reads."""
        return [self.w_in, self.w_uq, self.w_qk, self.w_ov, self.w_out]

    def _absorb(self, ctx: StepContext) -> bool:
        """Fewer multiplications per head (those of the absorbed attention count twice: its tiles are narrower)."""
        if ctx.n == 1 or self.dn + self.dr > 512 or self.dv > 256:        # heads larger than the ordinary attention kernels take
            return True
        n, pos = ctx.n, ctx.host_pos
        pairs, per = n * (pos + 0.5 * n), self.R * (self.dn + self.dv)
        return n * per + 2 * pairs * (2 * self.R + self.dr) < (pos + n) * per + pairs * (self.dn + self.dr + self.dv)

    def forward(self, x: torch.Tensor, st: dict, ctx: StepContext) -> torch.Tensor:
        B, n, H, dn, dr, dv, R, off = ctx.B, ctx.n, self.H, self.dn, self.dr, self.dv, self.R, self.off
        p = S.linear(x, self.w_in)
        kr = st.get("kr")
        cq = S.latent_prep(p, (off["dq"], off["c"], off["r"]), self.wq, self.wc, st["c"], kr, self.rot, ctx.pos, B, n, ctx.eps)
        gate = p[:, off["g"]:off["g"] + H * dv] if self.GATE else None
        q = S.linear(cq, self.w_uq)
        q_rot = q.view(B * n, H, dn + dr)[:, :, dn:]
        if self._absorb(ctx):
            qa = torch.empty(B * n, H, R + dr, dtype=q.dtype, device=q.device)
            S.head_linear(q, dn + dr, self.w_qk, qa[:, :, :R])
            if dr:
                S.rotate(q_rot, qa[:, :, R:], self.rot, ctx.pos, B, n)
            o = S.latent_attention(qa, st["c"], kr, self.sinks, ctx.pos, ctx.host_pos, B, n, self.scale)
            o = S.head_linear(o.view(B * n, H * R), R, self.w_ov, gate=gate).view(B * n, H * dv)
        else:
            if dr:
                S.rotate(q_rot, q_rot, self.rot, ctx.pos, B, n)
            T = ctx.host_pos + n
            kv = torch.empty(B, T, self.w_kv.shape[0], dtype=q.dtype, device=q.device)
            for b in range(B):
                S.linear(st["c"][b, :T], self.w_kv, out=kv[b])
            o = S.attention_bias(q, kv, kv[:, :, self.off_v:], None, ctx.pos, ctx.host_pos, B, n, H, H, dn + dr, dv, self.scale, self.SINK, self.sinks, kr,
                                 gate)
        return S.linear(o, self.w_out)


class GatedLatentAttention(LatentAttention):
    """Without positions (no rotated part) and sinks; the concatenated heads are multiplied by a sigmoid of a projection of the input."""
    ROTATED, SINK, GATE = False, False, True


class DenseMlp:
    def __init__(self, fc: dict, L: Loader, width: int):
        self.up, self.down = L.mat("up", (fc["ff"], width)), L.mat("down", (width, fc["ff"]))

    @staticmethod
    def shapes(fc: dict, width: int) -> dict:
        return {"up": (fc["ff"], width), "down": (width, fc["ff"])}

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return S.linear(S.linear(x, self.up, act=S.ACT_RELU2), self.down)


class GatedMlp:
    def __init__(self, fc: dict, L: Loader, width: int):
        pair = (L.mat("gate", (fc["ff"], width)), L.mat("up", (fc["ff"], width)))
        self.gate_up = torch.stack(pair, 1).view(2 * fc["ff"], width)        # rows alternate, the Linear's epilogue joins each pair
        self.down = L.mat("down", (width, fc["ff"]))

    @staticmethod
    def shapes(fc: dict, width: int) -> dict:
        return {"gate": (fc["ff"], width), "up": (fc["ff"], width), "down": (width, fc["ff"])}

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return S.linear(S.linear(x, self.gate_up, act=S.ACT_GLU_GELU), self.down)


MIXERS = {"lightning": Lightning, "channel_delta": ChannelDelta, "attention": BiasAttention, "latent_attention": LatentAttention,
          "latent_attention_2": GatedLatentAttention}
MLPS = {"relu2": DenseMlp, "gated_gelu": GatedMlp}
