"""Kernels of attention over cached latents and of the steps around it, each mechanism alone, against plain float64."""
import pytest
import torch

import latent_cases as H
import latodra_oracle as O
from helpers import check_status

pytestmark = pytest.mark.gpu
DT = [torch.float32, torch.bfloat16]


def rel(a, b):
    a, b = a.detach().double().cpu(), b.detach().double().cpu()
    assert torch.isfinite(a).all()
    return ((a - b).abs().max() / b.abs().max().clamp(min=1e-30)).item()


def tol(dt, f32=5e-6, b16=1e-2):
    return f32 if dt == torch.float32 else b16


def rnd(*s, seed=0, dt=torch.float32):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed)).to(dt).cuda()


def d(t):
    return t.double().cpu()


def at(pos):
    return torch.tensor([pos], dtype=torch.int32, device="cuda")


def rotation(entry):
    import mixers
    import seq_ops as S
    f, m = mixers.rotary_frequencies(entry)
    return S.Rotation(torch.tensor(f, dtype=torch.float64, device="cuda"), m)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("M", [1, 2, 8, 9, 17, 130, 300])
@pytest.mark.parametrize("ff,K", [(96, 72), (17, 30), (264, 200), (20, 9)])
def test_gated_linear(dt, M, ff, K):
    import seq_ops as S
    x, g, u = rnd(M, K, seed=M, dt=dt), rnd(ff, K, seed=1, dt=dt) * 2 * K ** -0.5, rnd(ff, K, seed=2, dt=dt) * K ** -0.5
    x[0] *= 8                                             # both ends of the activation
    w = torch.stack((g, u), 1).view(2 * ff, K)
    want = O.gelu_tanh(d(x) @ d(g).T) * (d(x) @ d(u).T)
    assert rel(S.linear(x, w, act=S.ACT_GLU_GELU), want) < tol(dt)
    check_status()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("M", [1, 2, 7, 16, 40])
@pytest.mark.parametrize("Hh,N,K,gap", [(3, 72, 24, 16), (5, 9, 13, 0), (2, 64, 512, 8), (1, 33, 40, 0)])
def test_linear_per_head(dt, M, Hh, N, K, gap):
    import seq_ops as S
    x, w = rnd(M, Hh * (K + gap), seed=1, dt=dt), rnd(Hh, N, K, seed=2, dt=dt) * K ** -0.5
    gate = rnd(M, Hh * N + 8, seed=3, dt=dt)[:, 8:]
    want = torch.einsum("mhk,hnk->mhn", d(x).view(M, Hh, K + gap)[:, :, :K], d(w))
    out = torch.full((M, Hh, N + 8), 7.0, dtype=dt, device="cuda")
    S.head_linear(x, K + gap, w, out[:, :, :N])
    assert rel(out[:, :, :N], want) < tol(dt) and (out[:, :, N:] == 7).all()
    assert rel(S.head_linear(x, K + gap, w, gate=gate), want * O.sigmoid(d(gate).reshape(M, Hh, N))) < tol(dt)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("W", [30, 64, 2100, 5000, 9000])
def test_stream_between_sublayers(dt, W):
    import seq_ops as S
    rows, eps = 5, 1e-3
    f = lambda seed: rnd(W, seed=seed)
    for parts in range(16):
        x, y, e = rnd(rows, W), rnd(rows, W, seed=1, dt=dt) * 0.02, rnd(rows, W, seed=2)
        want, kw = d(x), {}
        if parts & 1:
            want = want + 0.8 * O.rms(d(y), eps) * (d(f(3)) + 0.5)
            kw.update(y=y, w=f(3), mult=0.8)
        if parts & 2:
            want = want + d(e)
            kw["add_rows"] = e
        if parts & 4:
            want = want + d(f(4))
            kw["add_vec"] = f(4)
        out = torch.empty(rows, W, dtype=dt, device="cuda")
        wo = want
        if parts & 8:
            wo = O.rms(want, eps) * (d(f(5)) + 0.5)
            kw["w_next"] = f(5)
        S.stream_update(x, dt, eps, offset=0.5, out=out, **kw)
        assert rel(x, want) < 2e-6 and rel(out, wo) < tol(dt, 3e-6, 6e-3)
    table, ids = rnd(20, W, dt=dt), torch.tensor([3, 19, 3]).cuda()
    x, xb, x2 = S.embed(table, ids, 1.0, f(6), 0.0, eps, True)
    want = O.rms(d(table)[ids.cpu()], eps) * d(f(6))
    assert rel(x, want) < 2e-6 and torch.equal(x, x2) and rel(xb, want) < tol(dt, 2e-6, 5e-3)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("Hh,dr,dims", [(3, 16, 16), (5, 6, 6), (2, 24, 10), (32, 64, 64), (1, 7, 4), (4, 128, 128)])
@pytest.mark.parametrize("pos", [0, 5, 131071])
def test_rotation(dt, Hh, dr, dims, pos):
    import seq_ops as S
    entry = H.rot(dims, 1e4, (4.0, 64, 8.0, 1.0))
    B, n, gap = 2, 3, 8
    x = rnd(B * n, Hh, gap + dr, seed=3, dt=dt)
    want = torch.cat([O.rotate(d(x)[b * n:b * n + n, :, gap:], range(pos, pos + n), entry) for b in range(B)])
    out = torch.empty(B * n, Hh, dr, dtype=dt, device="cuda")
    S.rotate(x[:, :, gap:], out, rotation(entry), at(pos), B, n)
    assert rel(out, want) < tol(dt, 3e-6, 5e-3)
    keep = x[:, :, :gap].clone()
    S.rotate(x[:, :, gap:], x[:, :, gap:], rotation(entry), at(pos), B, n)
    assert torch.equal(x[:, :, gap:], out) and torch.equal(x[:, :, :gap], keep)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("rq,R,dr,dims", [(56, 72, 16, 16), (13, 21, 6, 6), (24, 48, 0, 0), (1536, 512, 64, 64), (3000, 1000, 24, 10), (4000, 2000, 8, 8)])
def test_latent_preparation(dt, rq, R, dr, dims):
    import seq_ops as S
    B, n, pos, cap = 2, 3, 4, 9
    offs = (8, (8 + rq + 7) // 8 * 8, ((8 + rq + 7) // 8 * 8 + R + 7) // 8 * 8)
    p = rnd(B * n, offs[2] + dr + 8, seed=1, dt=dt) * 0.3
    wq, wc = rnd(rq, seed=2), rnd(R, seed=3)
    c = torch.full((B, cap, R), 5.0, dtype=dt, device="cuda")
    kr = torch.full((B, cap, dr), 5.0, dtype=dt, device="cuda") if dr else None
    entry = H.rot(dims, 300.0) if dr else None
    cq = S.latent_prep(p, offs, wq, wc, c, kr, rotation(entry) if dr else None, at(pos), B, n, 1e-3)
    assert rel(cq, O.rms(d(p)[:, offs[0]:offs[0] + rq], 1e-3) * d(wq)) < tol(dt)
    assert rel(c[:, pos:pos + n].reshape(B * n, R), O.rms(d(p)[:, offs[1]:offs[1] + R], 1e-3) * d(wc)) < tol(dt)
    assert (c[:, :pos] == 5).all() and (c[:, pos + n:] == 5).all()
    if dr:
        want = torch.cat([O.rotate(d(p)[b * n:b * n + n, offs[2]:offs[2] + dr], range(pos, pos + n), entry) for b in range(B)])
        assert rel(kr[:, pos:pos + n].reshape(B * n, dr), want) < tol(dt)
        assert (kr[:, :pos] == 5).all() and (kr[:, pos + n:] == 5).all()


def reference(q, k, v, sinks, scale, pos, n):
    """One sequence: q [n, H, D], k [T, H, D], v [T, H, dv]."""
    out = torch.empty(n, q.shape[1], v.shape[2], dtype=torch.float64)
    for h in range(q.shape[1]):
        s = torch.zeros(pos + n, pos + n, dtype=torch.float64)
        s[pos:] = q[:, h] @ k[:pos + n, h].T * scale
        out[:, h] = (O.causal_softmax(s, None if sinks is None else sinks[h]) @ v[:pos + n, h])[pos:]
    return out


LATENT = [(3, 72, 16), (5, 48, 0), (16, 512, 64), (4, 128, 8), (20, 320, 40), (40, 64, 64), (64, 256, 0), (100, 136, 24), (3, 21, 6), (2, 640, 0), (1, 8, 8), (8, 512, 128)]


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("Hh,R,dr", LATENT)
@pytest.mark.parametrize("B,n,pos", [(1, 1, 0), (3, 1, 126), (1, 1, 127), (2, 1, 700), (1, 2, 0), (2, 3, 126), (1, 37, 250)])
def test_attention_over_latents(dt, Hh, R, dr, B, n, pos):
    """Whatever lies in the cache past the sequence must not matter; one key stands out, at the borders of a tile and at both ends."""
    import seq_ops as S
    cap, T, scale = pos + n + 70, pos + n, (R + dr) ** -0.5
    q = rnd(B * n, Hh, R + dr, seed=1, dt=dt)
    c, kr = rnd(B, cap, R, seed=2, dt=dt), rnd(B, cap, dr, seed=3, dt=dt) if dr else None
    far = [j for j in (0, 1, 126, 127, 128, 129, 255, 256, T - 2, T - 1) if 0 <= j < T]
    for b in range(B):
        j = far[(b * 3 + n + Hh) % len(far)]
        q[b * n:(b + 1) * n, 0, :R] = c[b, j] * 1.5            # the first head looks at key j
    c[:, T:] = float("nan")
    if dr:
        kr[:, T:] = float("nan")
    sinks = rnd(Hh, seed=4) * 2 if dr else None
    want = torch.cat([reference(d(q)[b * n:b * n + n], (d(c[b]) if kr is None else torch.cat((d(c[b]), d(kr[b])), 1))[:, None].expand(cap, Hh, R + dr),
                                d(c[b])[:, None].expand(cap, Hh, R), None if sinks is None else d(sinks), scale, pos, n) for b in range(B)])
    for host in ((pos, -1) if n == 1 else (pos,)):
        assert rel(S.latent_attention(q, c, kr, sinks, at(pos), host, B, n, scale), want) < tol(dt)
    check_status()


def test_latent_attention_long_and_split():
    """Thousands of keys over many splits, then the same workspace plan on a nearly empty cache."""
    import seq_ops as S
    for B, Hh, pos in ((1, 16, 5000), (1, 16, 3), (70, 32, 1500), (150, 8, 300)):
        R, dr, cap = 256, 64, 5100
        q, c, kr = rnd(B, Hh, R + dr, dt=torch.bfloat16), rnd(B, cap, R, seed=1, dt=torch.bfloat16), rnd(B, cap, dr, seed=2, dt=torch.bfloat16)
        c[:, pos // 2] *= 4
        got = S.latent_attention(q, c, kr, None, at(pos), -1, B, 1, 0.05)
        for b in (0, B - 1):
            k = torch.cat((d(c[b]), d(kr[b])), 1)[:, None].expand(cap, Hh, R + dr)
            assert rel(got[b], reference(d(q)[b:b + 1], k, d(c[b])[:, None].expand(cap, Hh, R), None, 0.05, pos, 1)[0]) < 1e-2
    check_status()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("Hh,dn,dr,dv", [(3, 24, 16, 40), (2, 128, 64, 128), (5, 56, 24, 72), (2, 40, 0, 16), (2, 64, 128, 72), (3, 10, 6, 7), (1, 200, 40, 144), (2, 8, 8, 8)])
@pytest.mark.parametrize("B,n,pos", [(1, 2, 0), (2, 130, 0), (1, 64, 100), (2, 33, 127), (1, 300, 129)])
def test_attention_with_a_shared_key_part(dt, Hh, dn, dr, dv, B, n, pos):
    """Own and shared key columns, learned sinks, gate, keys and values side by side in one buffer."""
    import seq_ops as S
    T, scale, gap = pos + n, (dn + dr) ** -0.5, 8
    q = rnd(B * n, Hh * (dn + dr), seed=1, dt=dt)
    off_v = (Hh * dn + 7) // 8 * 8
    kv = rnd(B, T, off_v + (Hh * dv + 7) // 8 * 8, seed=2, dt=dt)
    k2 = rnd(B, T + 9, dr, seed=3, dt=dt) if dr else None
    far = [j for j in (0, 127, 128, T - 1) if j < T]
    for b in range(B):
        j = far[(b + n + Hh) % len(far)]
        q.view(B, n, Hh, dn + dr)[b, :, 0, :dn] = kv[b, j, :dn] * 2
    if dr:
        k2[:, T:] = float("nan")
    sinks, gate = rnd(Hh, seed=4) * 2, rnd(B * n, Hh * dv + gap, seed=5, dt=dt)[:, gap:]
    for use_sink, use_gate in ((True, False), (False, True), (True, True)):
        want = []
        for b in range(B):
            k = d(kv[b])[:, :Hh * dn].reshape(T, Hh, dn)
            if dr:
                k = torch.cat((k, d(k2[b, :T])[:, None].expand(T, Hh, dr)), 2)
            o = reference(d(q)[b * n:b * n + n].view(n, Hh, dn + dr), k, d(kv[b])[:, off_v:off_v + Hh * dv].reshape(T, Hh, dv), d(sinks) if use_sink else None, scale, pos, n)
            want.append(o.reshape(n, Hh * dv))
        want = torch.cat(want)
        if use_gate:
            want = want * O.sigmoid(d(gate))
        got = S.attention_bias(q, kv, kv[:, :, off_v:], None, at(pos), pos, B, n, Hh, Hh, dn + dr, dv, scale, use_sink, sinks if use_sink else None, k2,
                               gate if use_gate else None)
        assert rel(got, want) < tol(dt)
    check_status()
