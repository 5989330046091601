"""Functional wrappers over the hybrid-decoder entry points of include/plz.h (recurrent and attention mixers, fp32 residual stream,
sampling). Tensors are torch CUDA tensors in the model's type T (bf16, or fp32 in the 32-bit mode) unless noted; rows are b * n + t for
B sequences that advance in lockstep by n tokens."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

import plz_native as P

ACT_NONE, ACT_RELU2, ACT_GLU_GELU = 0, 1, 2
BIAS_FRONT, BIAS_BACK = 256, 256      # readable entries before distance 0 / after the last one of a bias row (tile-wide reads)


def code(dtype: torch.dtype) -> int:
    return {torch.bfloat16: 0, torch.float32: 1}[dtype]


def _ptr(t):
    return None if t is None else t.data_ptr()


def linear(x: torch.Tensor, w: torch.Tensor, bias=None, act: int = ACT_NONE, out_f32: bool = False, out=None) -> torch.Tensor:
    """act(x W^T + bias); x [M, K] rows of any pitch, w [N, K] (its rows may be pitched). ACT_GLU_GELU: rows 2 i, 2 i + 1 of w are a gate /
    up pair and the result is [M, N / 2]. out: a tensor (rows of any pitch) to write instead of a new one."""
    P._need_cuda(x, w)
    M, K = x.shape
    N = w.shape[0]
    assert w.shape[1] == K and x.stride(1) == 1 and w.stride(1) == 1 and x.dtype == w.dtype
    cols = N // 2 if act == ACT_GLU_GELU else N
    y = out
    if y is None:
        y = torch.empty(M, cols, dtype=torch.float32 if out_f32 else x.dtype, device=x.device)
    assert y.shape == (M, cols) and y.stride(1) == 1
    f32 = out_f32 and x.dtype != torch.float32
    P.check(P.lib().plz_seq_linear(code(x.dtype), x.data_ptr(), x.stride(0), M, K, w.data_ptr(), w.stride(0), N, _ptr(bias), act, y.data_ptr(),
                                   y.stride(0), int(f32), P.stream_ptr()), "plz_seq_linear")
    return y


def head_linear(x: torch.Tensor, x_head: int, w: torch.Tensor, out=None, gate=None) -> torch.Tensor:
    """out[m, h, :] = x[m, h, :] w[h]^T (times sigmoid(gate[m, h, :])); x [M, >= H heads, x_head columns apart], w [H, N, K], out [M, H, N]
    (any pitches, new and dense if None), gate a view [M, H * N]."""
    P._need_cuda(x, w)
    H, N, K = w.shape
    if out is None:
        out = torch.empty(x.shape[0], H, N, dtype=x.dtype, device=x.device)
    assert w.is_contiguous() and x.stride(1) == 1 and out.stride(2) == 1 and x.dtype == w.dtype and x.shape[1] >= (H - 1) * x_head + K
    d = P.HeadLinear(x.data_ptr(), x.stride(0), x_head, w.data_ptr(), out.data_ptr(), out.stride(0), out.stride(1), _ptr(gate),
                     0 if gate is None else gate.stride(0), x.shape[0], H, N, K)
    P.check(P.lib().plz_head_linear(code(x.dtype), C.byref(d), P.stream_ptr()), "plz_head_linear")
    return out


def embed(table: torch.Tensor, ids: torch.Tensor, scale: float, norm_w=None, norm_offset: float = 0.0, eps: float = 0.0, copy: bool = False):
    """(x fp32 [rows, W], the same in T, a second fp32 copy or None): table rows times scale, with norm_w then RMS-normed.
    The one in T is x itself in the 32-bit mode."""
    P._need_cuda(table, ids)
    rows, W = ids.numel(), table.shape[1]
    assert ids.dtype == torch.int64 and ids.is_contiguous()
    x = torch.empty(rows, W, dtype=torch.float32, device=table.device)
    x2 = torch.empty_like(x) if copy else None
    xb = x if table.dtype == torch.float32 else torch.empty(rows, W, dtype=table.dtype, device=table.device)
    P.check(P.lib().plz_seq_embed(code(table.dtype), table.data_ptr(), table.stride(0), ids.data_ptr(), rows, W, table.shape[0], float(scale),
                                  _ptr(norm_w), float(norm_offset), float(eps), x.data_ptr(), _ptr(x2), None if xb is x else xb.data_ptr(), None,
                                  P.stream_ptr()), "plz_seq_embed")
    return x, xb, x2


def stream_update(x: torch.Tensor, dtype: torch.dtype, eps: float, y=None, w=None, mult: float = 1.0, offset: float = 0.0, add_rows=None, add_vec=None,
                  w_next=None, out=None):
    """The residual stream x (fp32, in place) between two sublayers: x += mult * rms_norm(y) * (w + offset); x += add_rows + add_vec;
    out = x, or rms_norm(x) * (w_next + offset), in T. Absent parts are None."""
    d = P.Stream(_ptr(y), 0 if y is None else y.stride(0), _ptr(w), float(offset), float(mult), float(eps), x.shape[0], x.shape[1], x.data_ptr(),
                 _ptr(add_rows), _ptr(add_vec), _ptr(w_next), _ptr(out))
    P.check(P.lib().plz_seq_stream(code(dtype), C.byref(d), P.stream_ptr()), "plz_seq_stream")


def residual_norm(y: torch.Tensor, w: torch.Tensor, w_offset: float, mult: float, eps: float, x: torch.Tensor, xb: torch.Tensor):
    """x += mult * rms_norm(y) * (w + w_offset) in place; xb follows (nothing to do when it is x)."""
    stream_update(x, y.dtype, eps, y, w, mult, w_offset, out=None if xb is x else xb)


def rows_norm(x: torch.Tensor, idx, w: torch.Tensor, w_offset: float, eps: float, dtype: torch.dtype) -> torch.Tensor:
    rows = x.shape[0] if idx is None else idx.numel()
    out = torch.empty(rows, x.shape[1], dtype=dtype, device=x.device)
    P.check(P.lib().plz_seq_rows_norm(code(dtype), x.data_ptr(), _ptr(idx), w.data_ptr(), float(w_offset), float(eps), rows, x.shape[1],
                                      out.data_ptr(), P.stream_ptr()), "plz_seq_rows_norm")
    return out


def norm_gate(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float, groups: int) -> torch.Tensor:
    """o fp32 [rows, groups * L]; gate a T view [rows, groups * L]; w fp32 [L]."""
    rows, W = o.shape
    out = torch.empty(rows, W, dtype=gate.dtype, device=o.device)
    P.check(P.lib().plz_seq_norm_gate(code(gate.dtype), o.data_ptr(), gate.data_ptr(), gate.stride(0), w.data_ptr(), float(eps), rows, groups,
                                      W // groups, out.data_ptr(), P.stream_ptr()), "plz_seq_norm_gate")
    return out


def delta_prep(proj: torch.Tensor, offs, a: torch.Tensor, taps: torch.Tensor, A_log: torch.Tensor, dt_bias: torch.Tensor, conv, B: int, n: int,
               H: int, G: int, dk: int, dv: int, q_scale: float):
    """(q, k, v, log decay, beta), all fp32; offs = columns of (q, k, v, beta) in proj; conv (inputs kept for the convolution) is updated."""
    dev, rows = proj.device, B * n
    f = lambda w: torch.empty(rows, w, dtype=torch.float32, device=dev)
    q, k, v, lg, beta = f(G * dk), f(G * dk), f(H * dv), f(H * dk), f(H)
    d = P.DeltaPrep(proj.data_ptr(), proj.stride(0), *offs, a.data_ptr(), a.stride(0), taps.data_ptr(), A_log.data_ptr(), dt_bias.data_ptr(),
                    _ptr(conv), taps.shape[1], B, n, H, G, dk, dv, float(q_scale), q.data_ptr(), k.data_ptr(), v.data_ptr(), lg.data_ptr(), beta.data_ptr())
    P.check(P.lib().plz_delta_prep(code(proj.dtype), C.byref(d), P.stream_ptr()), "plz_delta_prep")
    return q, k, v, lg, beta


def _chunk_ws(chunked: bool, B, n, H, dk, dv, device):
    need = P.lib().plz_chunk_ws_bytes(B, n, H, dk, dv) if chunked else 0
    return (torch.empty(need, dtype=torch.uint8, device=device), need) if need else (None, 0)


def delta_rule(q, k, v, logg, beta, state: torch.Tensor, B: int, n: int, H: int, G: int, dk: int, dv: int, chunked: bool = False) -> torch.Tensor:
    """o fp32 [B * n, H * dv]; state fp32 [B, H, dk, dv] in place. chunked: 64 tokens at a time on the tensor cores (dk <= 128; larger
    key sizes run token by token)."""
    ws, need = _chunk_ws(chunked, B, n, H, dk, dv, state.device)
    o = torch.empty(B * n, H * dv, dtype=torch.float32, device=state.device)
    d = P.DeltaRule(q.data_ptr(), k.data_ptr(), v.data_ptr(), logg.data_ptr(), beta.data_ptr(), state.data_ptr(), o.data_ptr(), B, n, H, G, dk, dv)
    P.check(P.lib().plz_delta_rule(C.byref(d), _ptr(ws), need, P.stream_ptr()), "plz_delta_rule")
    return o


def decay_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: torch.Tensor, B: int, n: int, H: int, dk: int,
                    dv: int, chunked: bool = False) -> torch.Tensor:
    """q, k, v: slices (before silu) of one projection; o fp32 [B * n, H * dv]; state fp32 [B, H, dk, dv] in place. chunked: as in
    delta_rule (bf16 projections)."""
    ws, need = _chunk_ws(chunked, B, n, H, dk, dv, state.device)
    assert q.stride(0) == k.stride(0) == v.stride(0)
    o = torch.empty(B * n, H * dv, dtype=torch.float32, device=state.device)
    d = P.DecayAttn(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), decay.data_ptr(), state.data_ptr(), o.data_ptr(), B, n, H, dk, dv)
    P.check(P.lib().plz_decay_attn(code(q.dtype), C.byref(d), _ptr(ws), need, P.stream_ptr()), "plz_decay_attn")
    return o


def attn_prep(proj: torch.Tensor, offs, wq: torch.Tensor, wk: torch.Tensor, mix, v_first, v_first_write: bool, kc: torch.Tensor, vc: torch.Tensor,
              pos: torch.Tensor, B: int, n: int, eps: float) -> torch.Tensor:
    """Normalised queries [B * n, qw]; keys and (mixed) values go into the caches kc [B, cap, kw], vc [B, cap, vw] at pos."""
    qw, kw, vw = wq.numel(), kc.shape[2], vc.shape[2]
    q = torch.empty(B * n, qw, dtype=proj.dtype, device=proj.device)
    d = P.AttnPrep(proj.data_ptr(), proj.stride(0), *offs, wq.data_ptr(), wk.data_ptr(), _ptr(mix), _ptr(v_first), int(v_first_write), q.data_ptr(),
                   kc.data_ptr(), vc.data_ptr(), kc.stride(0), vc.stride(0), pos.data_ptr(), B, n, qw, kw, vw, kc.shape[1], float(eps))
    P.check(P.lib().plz_attn_prep(code(proj.dtype), C.byref(d), P.stream_ptr()), "plz_attn_prep")
    return q


@dataclass
class DistanceBias:
    """Bias by distance of every head, as the attention kernels read it."""
    rows: torch.Tensor      # fp32 [H, BIAS_FRONT + D + BIAS_BACK]: zeros, distances 0 .. D - 1, the last one repeated
    top: torch.Tensor       # fp32 [H], the largest of each head
    D: int

    @classmethod
    def from_distances(cls, by_distance: torch.Tensor) -> "DistanceBias":
        """by_distance [H, D]: the biases of distances 0 .. D - 1; the last one holds for all beyond."""
        H, D = by_distance.shape
        rows = torch.zeros(H, BIAS_FRONT + D + BIAS_BACK, dtype=torch.float32, device=by_distance.device)
        rows[:, BIAS_FRONT:BIAS_FRONT + D] = by_distance
        rows[:, BIAS_FRONT + D:] = by_distance[:, -1:]
        return cls(rows, by_distance.float().max(1).values.contiguous(), D)


def attention_bias(q: torch.Tensor, kc: torch.Tensor, vc: torch.Tensor, bias: DistanceBias | None, pos: torch.Tensor, host_pos: int, B: int, n: int,
                   H: int, G: int, dk: int, dv: int, scale: float, sink: bool, sinks=None, k2=None, gate=None, cap: int | None = None) -> torch.Tensor:
    """Causal attention of n new tokens per sequence (their keys and values already in kc, vc [B, tokens, ...]).
    host_pos: the value of pos, or -1 (one token only) when the launch is to be replayed at other positions.
    sinks fp32 [H]: scores of a learned sink (sink alone: score 0). k2 [B, tokens, dk2]: the last dk2 of the dk key columns, shared by all
    heads. gate: view [B * n, H * dv], the output is multiplied by its sigmoid."""
    o = torch.empty(B * n, H * dv, dtype=q.dtype, device=q.device)
    bp, ldb, nb, top = (None, 0, 0, None) if bias is None else (bias.rows.data_ptr() + 4 * BIAS_FRONT, bias.rows.stride(0), bias.D, bias.top.data_ptr())
    d = P.AttnBias(q.data_ptr(), q.stride(0), kc.data_ptr(), vc.data_ptr(), kc.stride(0), vc.stride(0), o.data_ptr(), o.stride(0), bp, ldb, nb, top,
                   pos.data_ptr(), host_pos, cap or kc.shape[1], B, n, H, G, dk, dv, int(sink), float(scale), _ptr(sinks), kc.stride(1), vc.stride(1),
                   _ptr(k2), 0 if k2 is None else k2.stride(0), 0 if k2 is None else k2.shape[2], _ptr(gate), 0 if gate is None else gate.stride(0))
    need = P.lib().plz_attn_bias_ws_bytes(B, H, G, dv, kc.shape[1]) if n == 1 else 0
    ws = torch.empty(need, dtype=torch.uint8, device=q.device) if need else None
    P.check(P.lib().plz_attn_bias(code(q.dtype), C.byref(d), _ptr(ws), need, P.stream_ptr()), "plz_attn_bias")
    return o


@dataclass
class Rotation:
    """Rotary positions of one head part: frequency of every pair, factor on cos and sin."""
    freq: torch.Tensor      # fp64 [pairs], device
    m: float

    def args(self):
        return self.freq.data_ptr(), self.freq.numel(), float(self.m)


def _turns(rot: Rotation | None):
    return (None, 0, 1.0) if rot is None else rot.args()


def latent_prep(proj: torch.Tensor, offs, wq: torch.Tensor, wc: torch.Tensor, c: torch.Tensor, kr, rot: Rotation | None, pos: torch.Tensor, B: int,
                n: int, eps: float) -> torch.Tensor:
    """Normed query latent [B * n, q_rank]; the normed latent and the rotated key part go into the caches c [B, cap, R], kr [B, cap, dr] (or
    None) at pos. offs: columns of (query latent, latent, key part) in proj."""
    cq = torch.empty(B * n, wq.numel(), dtype=proj.dtype, device=proj.device)
    d = P.LatentPrep(proj.data_ptr(), proj.stride(0), *offs, wq.data_ptr(), wc.data_ptr(), cq.data_ptr(), c.data_ptr(), _ptr(kr), c.stride(0),
                     0 if kr is None else kr.stride(0), pos.data_ptr(), *_turns(rot), B, n, wq.numel(), wc.numel(), 0 if kr is None else kr.shape[2],
                     c.shape[1], float(eps))
    P.check(P.lib().plz_latent_prep(code(proj.dtype), C.byref(d), P.stream_ptr()), "plz_latent_prep")
    return cq


def rotate(x: torch.Tensor, out: torch.Tensor, rot: Rotation, pos: torch.Tensor, B: int, n: int):
    """out[:, h] = x[:, h] with its leading pairs turned by position * frequency; x, out views [B * n, H, dr] (out may be x)."""
    assert x.shape == out.shape and x.stride(2) == 1 and out.stride(2) == 1 and x.dtype == out.dtype
    d = P.Rotate(x.data_ptr(), x.stride(0), x.stride(1), out.data_ptr(), out.stride(0), out.stride(1), pos.data_ptr(), *rot.args(), B, n, x.shape[1],
                 x.shape[2])
    P.check(P.lib().plz_rotate(code(x.dtype), C.byref(d), P.stream_ptr()), "plz_rotate")


def latent_attention(q: torch.Tensor, c: torch.Tensor, kr, sinks, pos: torch.Tensor, host_pos: int, B: int, n: int, scale: float) -> torch.Tensor:
    """Causal attention of n new tokens per sequence whose keys are the cached rows [c | kr] and whose values are c, for all heads alike.
    q [B * n, H, R + dr], c [B, cap, R], kr [B, cap, dr] or None, sinks fp32 [H] or None; [B * n, H, R]. host_pos as in attention_bias."""
    H, R, dr = q.shape[1], c.shape[2], 0 if kr is None else kr.shape[2]
    assert q.is_contiguous() and q.shape[2] == R + dr
    o = torch.empty(B * n, H, R, dtype=q.dtype, device=q.device)
    need = P.lib().plz_latent_attn_ws_bytes(code(q.dtype), B, n, H, R, dr, c.shape[1])
    ws = torch.empty(need, dtype=torch.uint8, device=q.device)
    d = P.LatentAttn(q.data_ptr(), q.stride(0), c.data_ptr(), _ptr(kr), c.stride(0), 0 if kr is None else kr.stride(0), o.data_ptr(), o.stride(0),
                     _ptr(sinks), pos.data_ptr(), host_pos, c.shape[1], B, n, H, R, dr, float(scale))
    P.check(P.lib().plz_latent_attn(code(q.dtype), C.byref(d), _ptr(ws), need, P.stream_ptr()), "plz_latent_attn")
    return o


def advance(pos: torch.Tensor, n: int):
    P.check(P.lib().plz_advance(pos.data_ptr(), n, P.stream_ptr()), "plz_advance")


def sample(logits: torch.Tensor, pos: torch.Tensor, temperature: float = 0.0, top_k: int = 0, seed: int = 0) -> torch.Tensor:
    """Next token int64 [rows] of fp32 logits [rows, V]; temperature 0 is greedy."""
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    out = torch.empty(logits.shape[0], dtype=torch.int64, device=logits.device)
    P.check(P.lib().plz_sample(logits.data_ptr(), logits.stride(0), logits.shape[0], logits.shape[1], float(temperature), int(top_k),
                               seed & 0xFFFFFFFF, pos.data_ptr(), out.data_ptr(), P.stream_ptr()), "plz_sample")
    return out
