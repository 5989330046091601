"""Kernels of the hybrid decoders, each mechanism alone, against the plain implementation (oracle/gopunex_oracle.py) in float64."""
import pytest
import torch

import gopunex_oracle as O
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


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("M", [1, 2, 7, 8, 9, 16, 17, 130, 300])
@pytest.mark.parametrize("N,K", [(192, 72), (13, 30), (64, 24), (520, 200), (40, 9)])
def test_linear(dt, M, N, K):
    import seq_ops as S
    x, w, b = rnd(M, K + 8, seed=M, dt=dt)[:, :K], rnd(N, K, seed=1, dt=dt) * K ** -0.5, rnd(N, seed=2, dt=dt)
    lin = x.double().cpu() @ w.double().cpu().T
    assert rel(S.linear(x, w), lin) < tol(dt)
    assert rel(S.linear(x, w, b, S.ACT_RELU2), O.squared_relu(lin + b.double().cpu())) < tol(dt)
    if dt == torch.bfloat16 and M <= 16:
        assert rel(S.linear(x, w, b, out_f32=True), lin + b.double().cpu()) < 1e-4


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("W", [30, 64, 260, 5000])
def test_embedding_and_norms(dt, W):
    import seq_ops as S
    table, ids = rnd(50, W, dt=dt), torch.tensor([[3, 49, 0], [7, 7, 11]]).cuda()
    x, xb, _ = S.embed(table, ids, 0.37)
    assert rel(x, table.double().cpu()[ids.cpu().reshape(-1)] * 0.37) < 1e-6 and (xb is x) == (dt == torch.float32)
    y, w = rnd(6, W, seed=3, dt=dt) * 0.01, rnd(W, seed=4)
    want = x.double().cpu() + 0.7 * O.rms(y.double().cpu(), 1e-3) * (1 + w.double().cpu())
    S.residual_norm(y, w, 1.0, 0.7, 1e-3, x, xb)
    assert rel(x, want) < 2e-6 and rel(xb, want) < tol(dt, 2e-6, 5e-3)
    idx = torch.tensor([5, 0, 0]).cuda()
    assert rel(S.rows_norm(x, idx, w, 1.0, 1e-3, dt), O.rms(want[[5, 0, 0]], 1e-3) * (1 + w.double().cpu())) < tol(dt)
    check_status()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("groups,L", [(1, 40), (3, 17), (9, 64), (1, 700), (2, 320)])
def test_norm_gate(dt, groups, L):
    import seq_ops as S
    o, gate, w = rnd(5, groups * L) * 0.1, rnd(5, groups * L + 8, seed=1, dt=dt)[:, :groups * L], rnd(L, seed=2)
    od = o.double().cpu().view(5, groups, L)
    want = O.rms(od, 1e-4) * w.double().cpu() * O.sigmoid(gate.double().cpu().reshape(5, groups, L))
    assert rel(S.norm_gate(o, gate, w, 1e-4, groups), want.view(5, -1)) < tol(dt)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("H,G,dk,dv,taps", [(4, 2, 16, 24, 4), (3, 3, 20, 8, 3), (2, 1, 5, 9, 2), (2, 2, 144, 72, 4), (2, 1, 8, 12, 1), (1, 1, 16, 16, 6)])
@pytest.mark.parametrize("cuts", [(60,), (1,) * 9 + (51,), (2, 3, 1, 30, 1, 23), (17, 43)])
def test_delta_preparation(dt, H, G, dk, dv, taps, cuts):
    """Convolution across portions (two sequences in lockstep), activation, unit norms, decay and step size."""
    import seq_ops as S
    B, n = 2, sum(cuts)
    C = 2 * G * dk + H * dv
    offs = [0, (G * dk + 7) // 8 * 8]
    offs += [offs[1] + (G * dk + 7) // 8 * 8]
    offs += [offs[2] + (H * dv + 7) // 8 * 8]
    W = offs[3] + H
    proj, a = rnd(B, n, W, seed=1, dt=dt), rnd(B, n, H * dk, seed=2, dt=dt)
    tp, al, db = rnd(C, taps, seed=3), rnd(H, seed=4), rnd(H * dk, seed=5)
    conv = torch.zeros(B, taps - 1, C, dtype=dt, device="cuda") if taps > 1 else None
    got, at = [[] for _ in range(5)], 0
    for c in cuts:
        out = S.delta_prep(proj[:, at:at + c].reshape(B * c, W).contiguous(), offs, a[:, at:at + c].reshape(B * c, -1).contiguous(), tp, al, db, conv, B, c,
                           H, G, dk, dv, dk ** -0.5)
        for g, t in zip(got, out):
            g.append(t.view(B, c, -1))
        at += c
    got = [torch.cat(g, 1) for g in got]
    pd = proj.double().cpu()
    for b in range(B):
        sl = [pd[b, :, offs[i]:offs[i] + w] for i, w in enumerate((G * dk, G * dk, H * dv))]
        tw = tp.double().cpu().split([G * dk, G * dk, H * dv])
        q, k, v = (O.silu(O.causal_conv(x, t)) for x, t in zip(sl, tw))
        want = [O.unit(q.view(n, G, dk)) * dk ** -0.5, O.unit(k.view(n, G, dk)), v,
                -torch.exp(al.double().cpu())[None, :, None] * O.softplus(a[b].double().cpu() + db.double().cpu()).view(n, H, dk), O.sigmoid(pd[b, :, offs[3]:])]
        for name, g, w in zip(("q", "k", "v", "decay", "beta"), got, want):
            assert rel(g[b], w.reshape(n, -1)) < 3e-6, name


def _delta_case(n, H, G, dk, dv, B=2, seed=0, strong=True, alike=False):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    q, k = O.unit(r(B, n, G, dk)) * dk ** -0.5, O.unit(r(B, n, G, dk))
    if alike:                                   # nearly equal keys: the corrections of a chunk are large
        k = O.unit(r(1, 1, G, dk) + 0.3 * r(B, n, G, dk))
    v, beta = r(B, n, H, dv), torch.rand(B, n, H, generator=g)
    lg = -torch.rand(B, n, H, dk, generator=g) * 0.05
    if strong:                                  # some channels forget everything at once, in the middle of any block
        lg = torch.where(torch.rand(lg.shape, generator=g) < 0.04, -torch.rand(lg.shape, generator=g) * 150, lg)
    return q, k, v, lg, beta, r(B, H, dk, dv)


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("n,H,G,dk,dv,alike", [(1, 2, 1, 16, 8, False), (64, 2, 2, 32, 64, False), (65, 4, 2, 24, 20, True), (200, 2, 1, 128, 128, False), (150, 1, 1, 7, 5, False),
                                              (130, 3, 3, 72, 136, True), (63, 2, 2, 200, 16, False)])
def test_delta_rule(chunked, n, H, G, dk, dv, alike):
    import seq_ops as S
    B = 2
    q, k, v, lg, beta, S0 = _delta_case(n, H, G, dk, dv, B, seed=n, alike=alike)
    st = S0.cuda().clone()
    f = lambda t: t.reshape(B * n, -1).contiguous().cuda()
    o = S.delta_rule(f(q), f(k), f(v), f(lg), f(beta), st, B, n, H, G, dk, dv, chunked).view(B, n, H, dv)
    check_status()
    limit = 1e-4 if chunked else 5e-6
    for b in range(B):
        for h in range(H):
            # the plain rule starts from zero: write the initial state with unit keys and no decay first
            eye = torch.eye(dk, dtype=torch.float64)
            pre = lambda x, z: torch.cat([z, x.double()])
            qq, kk = pre(q[b, :, h // (H // G)], torch.zeros(dk, dk, dtype=torch.float64)), pre(k[b, :, h // (H // G)], eye)
            want = O.gated_delta(qq, kk, pre(v[b, :, h], S0[b, h].double()), pre(torch.exp(lg[b, :, h].double()), torch.ones(dk, dk, dtype=torch.float64)),
                                 torch.cat([torch.ones(dk, dtype=torch.float64), beta[b, :, h].double()]))[dk:]
            assert rel(o[b, :, h], want) < limit, (b, h)
    # the state that is left: read it out with unit queries, no write, no decay
    z = torch.zeros(B, dk, H, dk).cuda()
    probe = torch.eye(dk).view(1, dk, 1, dk).expand(B, dk, G, dk).reshape(B * dk, -1).contiguous().cuda()
    read = S.delta_rule(probe, probe, torch.zeros(B * dk, H * dv).cuda(), z.reshape(B * dk, -1), torch.zeros(B * dk, H).cuda(), st.clone(), B, dk, H, G, dk, dv)
    assert rel(read.view(B, dk, H, dv).permute(0, 2, 1, 3), st) < 1e-6


@pytest.mark.parametrize("dt,chunked", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("n,H,dk,dv", [(1, 2, 16, 8), (64, 2, 32, 64), (65, 3, 24, 20), (200, 2, 128, 128), (150, 1, 7, 5), (330, 1, 72, 136)])
def test_decayed_linear_attention(dt, chunked, n, H, dk, dv):
    import seq_ops as S
    B = 2
    W = H * (2 * dk + dv) + 8
    W = (W + 7) // 8 * 8
    proj = rnd(B * n, W, seed=n, dt=dt)
    decay = torch.tensor([0.999, 0.2, 0.7][:H], device="cuda")
    S0 = torch.zeros(B, H, dk, dv, device="cuda")
    cut = n // 3
    rows = lambda lo, hi: torch.cat([proj[b * n + lo:b * n + hi] for b in range(B)])
    parts, st = [], S0.clone()
    for lo, hi in ((0, cut), (cut, n)):
        if hi > lo:
            pp = rows(lo, hi)
            sl = (pp[:, :H * dk], pp[:, H * dk:2 * H * dk], pp[:, 2 * H * dk:2 * H * dk + H * dv])
            parts.append(S.decay_attention(*sl, decay, st, B, hi - lo, H, dk, dv, chunked).view(B, hi - lo, H, dv))
    o = torch.cat(parts, 1)
    for b in range(B):
        pd = proj[b * n:(b + 1) * n].double().cpu()
        for h in range(H):
            q, k, v = (O.silu(pd[:, at + h * w:at + (h + 1) * w]) for at, w in ((0, dk), (H * dk, dk), (2 * H * dk, dv)))
            assert rel(o[b, :, h], O.decayed_linear_attention(q, k, v, decay[h].double().item())) < (1e-4 if chunked else 1e-5)


def _attention_want(q, k, v, tab, scale, sink, pos):
    """q [n, H, dk] at positions pos ..; k, v [T, G, .]; tab [H, D]."""
    n, H, _ = q.shape
    T, G, _ = k.shape
    i, j = torch.arange(pos, pos + n)[:, None], torch.arange(T)[None]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale + tab[h][(i - j).clamp(0, tab.shape[1] - 1)]
        p = O.softmax_off_by_one(s, i >= j) if sink else torch.softmax(s.masked_fill(i < j, float("-inf")), -1)
        out.append(p @ v[:, h // (H // G)])
    return torch.stack(out, 1)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("n,pos,H,G,dk,dv,D,sink", [(128, 0, 2, 1, 128, 128, 40, True), (300, 0, 4, 2, 48, 64, 200, True), (77, 130, 4, 1, 64, 128, 300, True),
                                                   (2, 511, 4, 4, 128, 48, 100, False), (257, 255, 3, 1, 80, 72, 513, True), (129, 1, 2, 1, 16, 8, 5, True),
                                                   (1, 777, 12, 2, 72, 128, 50, True), (1, 0, 8, 1, 24, 64, 200, True), (1, 70, 4, 4, 200, 256, 90, False),
                                                   (40, 20, 3, 3, 9, 11, 30, True), (1, 33, 3, 3, 9, 11, 30, True), (150, 3, 2, 2, 136, 200, 64, True), (1, 5000, 2, 1, 64, 64, 33, True)])
def test_attention_with_bias_and_sink(dt, n, pos, H, G, dk, dv, D, sink):
    """Any portion at any position; the cache past its end holds NaN, which nothing may read."""
    import seq_ops as S
    B, T = 2, pos + n
    q, kc, vc = rnd(B * n, H * dk, dt=dt), rnd(B, T + 9, G * dk, seed=1, dt=dt), rnd(B, T + 9, G * dv, seed=2, dt=dt)
    kc[:, T:] = float("nan")
    vc[:, T:] = float("nan")
    tab = rnd(H, D, seed=3) * 3
    o = S.attention_bias(q, kc, vc, S.DistanceBias.from_distances(tab), torch.tensor([pos], dtype=torch.int32, device="cuda"), pos if n > 1 else -1, B, n, H, G,
                         dk, dv, dk ** -0.5, sink)
    check_status()
    c = lambda t: t.double().cpu()
    for b in range(B):
        want = _attention_want(c(q.view(B, n, H, dk)[b]), c(kc[b, :T]).view(T, G, dk), c(vc[b, :T]).view(T, G, dv), c(tab), dk ** -0.5, sink, pos)
        assert rel(o.view(B, n, H, dv)[b], want) < tol(dt, 2e-6, 1e-2)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_far_away(dt, decode):
    """One key per probe stands out by its score; its distance runs over the tile borders, the bias table's last entries and the very
    first tokens. The query must return that key's value, weighted as its bias says."""
    import seq_ops as S
    H, dk, dv, D, T = 1, 32, 16, 200, 700
    kc, vc = rnd(1, T, dk, dt=dt) * 0.02, rnd(1, T, dv, seed=1, dt=dt)
    tab = torch.linspace(2.0, -2.0, D)[None].cuda()
    tab[0, -1] = 1.5                       # a jump at the last entry: one entry off shows
    for dist in (0, 1, 31, 32, 127, 128, 129, D - 2, D - 1, D, D + 1, 255, 256, 512, T - 1):
        i = T - 1
        k2 = kc.clone()
        k2[0, i - dist] = 1.0
        n = 1 if decode else 130
        q = torch.zeros(n, dk, device="cuda", dtype=dt)
        q[-1] = 1.0
        o = S.attention_bias(q, k2, vc, S.DistanceBias.from_distances(tab), torch.tensor([T - n], dtype=torch.int32, device="cuda"), T - n if n > 1 else -1, 1, n, H, 1,
                             dk, dv, 0.15, True)
        c = lambda t: t.double().cpu()
        want = _attention_want(c(q).view(n, 1, dk), c(k2[0]).view(T, 1, dk), c(vc[0]).view(T, 1, dv), c(tab), 0.15, True, T - n)
        assert rel(o[-1], want[-1].view(-1)) < tol(dt, 3e-6, 1.2e-2), dist


def test_sink_takes_the_weight_of_low_scores():
    import seq_ops as S
    for n in (1, 40):
        q, kc, vc = torch.full((n, 16), 4.0, device="cuda"), torch.full((1, 60, 16), -1.0, device="cuda"), torch.ones(1, 60, 16, device="cuda")
        for dt in DT:
            o = S.attention_bias(q.to(dt), kc.to(dt), vc.to(dt), None, torch.tensor([60 - n], dtype=torch.int32, device="cuda"), 60 - n if n > 1 else -1, 1, n, 1, 1, 16, 16,
                                 0.1, True)
            e = 60 * 2.718281828 ** -6.4
            assert abs(o[-1, 0].item() - e / (1 + e)) < 2e-3


def test_sampling():
    import seq_ops as S
    lg = rnd(4, 1000)
    lg[1, 17] = lg[1, 900] = 50.0                                   # equal: the first wins
    pos = torch.tensor([5], dtype=torch.int32, device="cuda")
    assert S.sample(lg, pos).tolist() == [lg[0].argmax().item(), 17, lg[2].argmax().item(), lg[3].argmax().item()]
    same = S.sample(lg, pos, 1.3, 0, seed=9)
    assert torch.equal(same, S.sample(lg, pos, 1.3, 0, seed=9))     # a draw is a function of seed, position and row
    top = lg.topk(5).indices
    for t in range(50):
        d = S.sample(lg, torch.tensor([t], dtype=torch.int32, device="cuda"), 2.0, 5, seed=1)
        assert all(d[r].item() in top[r].tolist() for r in (0, 2, 3))
    # frequencies follow softmax(logits / temperature)
    small = torch.tensor([[0.0, 1.0, 2.0, -1.0]], device="cuda").expand(4096, 4).contiguous()
    f = torch.bincount(S.sample(small, pos, 0.8, 0, seed=3), minlength=4).double().cpu() / 4096
    assert (f - torch.softmax(torch.tensor([0.0, 1.0, 2.0, -1.0], dtype=torch.float64) / 0.8, 0)).abs().max() < 0.03
