"""bench.py --workload hybrid [--design gopunex|latodra]: a hybrid decoder beside PalettizedQwen at equal width, feed-forward width,
attention heads and depth; random weights, synthetic tokens. Gopunex: lightning, channel-delta and distance-bias attention layers in turn;
Latodra: rotated and gated latent attention in turn.

One JSON line per size with prefill and decode throughput of both models, then one per kernel: time, algorithmic bytes and FLOPs, and
the fraction of its roofline max(bytes / copy bandwidth, FLOPs / GEMM peak), for the kernels of the new design and the like kernels of the
closest model. Times are CUDA events around CUDA graphs or eager launches after warm-up; inputs rotate over more than L2 or are larger.
"""
import json
import os
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
PKG = os.path.join(ROOT, "qwen-palettize_b200")
if PKG not in sys.path:
    sys.path.insert(0, PKG)

SIZES = {   # width, ff, attention heads / kv heads (of 128), recurrent heads (of 128), layers
    "small": (1024, 3072, 16, 8, 8, 6),
    "medium": (2560, 9728, 32, 8, 20, 6),
    "large": (4096, 12288, 32, 8, 32, 6),
}
LATENT = {"small": (512, 256), "medium": (1024, 512), "large": (1536, 512)}   # query latent, key / value latent; heads of 128 + 64 rotated, values 128
VOCAB = 32768
L2_BYTES = 126 << 20


def gopunex_config(width, ff, H, G, R, n_layers):
    mix = {"lightning": {"decay": [0.9 + 0.099 * i / R for i in range(R)], "dim": 128, "heads": R, "vdim": 128},
           "channel_delta": {"conv": 4, "dim": 128, "heads": R, "kv_heads": R, "vdim": 128},
           "attention": {"bias_max": 512, "dim": 128, "heads": H, "kv_heads": G, "scale": 128 ** -0.5, "v_mix": True, "vdim": 128}}
    order = ["lightning", "channel_delta", "attention"]
    return {"architecture": "Gopunex", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "residual_mult": 0.7, "vocab": VOCAB, "width": width,
            "layers": [{"type": order[i % 3], "mixer": mix[order[i % 3]], "mlp": {"ff": ff, "kind": "dense"}} for i in range(n_layers)]}


def latodra_config(size):
    width, ff, H, _, _, n_layers = SIZES[size]
    rq, R = LATENT[size]
    plain = {"dim": 128, "heads": H, "kv_rank": R, "q_rank": rq, "vdim": 128}
    mix = [("latent_attention", {**plain, "rot_dim": 64, "scale": 192 ** -0.5, "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "fast": 32.0, "original": 4096, "slow": 1.0}}}),
           ("latent_attention_2", {**plain, "scale": 128 ** -0.5})]
    return {"architecture": "Latodra", "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": width,
            "layers": [{"type": mix[i % 2][0], "mixer": mix[i % 2][1], "mlp": {"ff": ff, "kind": "dense"}} for i in range(n_layers)]}


def timed(torch, fn, reps, warm=3):
    for i in range(warm):
        fn(i)
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for i in range(reps):
        fn(i)
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / reps


def graphed(torch, fn, count, reps=5):
    """ms per call of fn(0) .. fn(count - 1) captured in one graph."""
    fn(0)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(count):
            fn(i)
    return timed(torch, lambda _: g.replay(), reps) / count


def models(torch, design, size, dev, pk):
    import decode_model as DM
    import hybrid_model
    import plz_native as P
    width, ff, H, G, R, n_layers = SIZES[size]
    cfg = gopunex_config(*SIZES[size]) if design == "gopunex" else latodra_config(size)
    hyb = hybrid_model.ARCHITECTURES[cfg["architecture"]].random(cfg, dev, seed=1)
    qwen = DM.PalettizedQwen.random(DM.ModelConfig(hidden=width, n_heads=H, n_kv_heads=G, head_dim=128, intermediate=ff, n_layers=n_layers, vocab=VOCAB),
                                    dev, seed=1, max_positions=4096)
    sizes = {"recurrent_heads": R} if design == "gopunex" else {"latents": LATENT[size]}
    out = {"workload": "hybrid", "design": design, "size": size, "width": width, "ff": ff, "attention_heads": [H, G], **sizes, "layers": n_layers, "vocab": VOCAB,
           "weights": "random", "peaks": pk, "prefill": {}, "decode": {}}
    for B, S in ((1, 2048), (8, 2048)):
        ids = torch.randint(0, VOCAB, (B, S), device=dev)
        ch = hyb.new_cache(B, S + 64)
        cq = qwen.new_cache(B, S + 64)

        def ph(_):
            ch.reset()
            hyb.prefill(ids, ch)

        def pq(_):
            cq.reset()
            qwen.prefill(ids, cq)
        th, tq = timed(torch, ph, 5), timed(torch, pq, 5)
        out["prefill"][f"B{B}_S{S}"] = {f"{design}_ms": th, f"{design}_tok_s": B * S / th * 1e3, "palettized_qwen_ms": tq, "palettized_qwen_tok_s": B * S / tq * 1e3}
        del ch, cq
    for B in (1, 8, 64):
        T, steps = 2048, 20
        ch = hyb.new_cache(B, T + 64)
        ch.length = T
        ch.pos.fill_(T)
        tok = torch.randint(0, VOCAB, (B,), device=dev)
        th = timed(torch, lambda _: hyb.decode_step(tok, ch), steps, warm=4)
        cq = qwen.new_cache(B, T + 64)
        g = None
        try:
            g, _ = qwen.decode_graph(tok, cq, T)
            tq = timed(torch, lambda _: g.replay(), steps)
        except P.PlzError:          # its small-M launch has no form for this batch and width
            P.lib().plz_set_smallm_overlap(0)
            tq = None
        out["decode"][f"B{B}_T{T}"] = {f"{design}_ms": th, f"{design}_tok_s": B / th * 1e3, "palettized_qwen_ms": tq, "palettized_qwen_tok_s": B / tq * 1e3 if tq else None,
                                       f"{design}_weight_and_state_bytes": hyb.weight_bytes() + ch.nbytes() + sum(st["S"].numel() * 4 for st in ch.layers if "S" in st)}
        del ch, cq, g
    return out


class Rows:
    """Lines of the per-kernel table."""

    def __init__(self, size, pk):
        self.size, self.bw, self.fl, self.rows = size, pk["hbm_gbs"] * 1e9, pk["tflops_burst"] * 1e12, []

    def add(self, kernel, phase, ms, nbytes, flops=0.0, like=None):
        tb, tf = nbytes / self.bw, flops / self.fl
        self.rows.append({"kernel": kernel, "size": self.size, "phase": phase, "us": ms * 1e3, "MB": nbytes / 1e6, "GFLOP": flops / 1e9, "bound": "flops" if tf > tb else "bytes",
                          "frac_of_roofline": max(tb, tf) * 1e3 / ms, "like": like})


def latodra_kernels(torch, size, dev, pk):
    """Rows of the per-kernel table of Latodra at one size."""
    import mixers
    import plz_ops as ops
    import seq_ops as S
    from bench import make_weight, weight_bytes
    width, ff, H, G, _, _ = SIZES[size]
    rq, R = LATENT[size]
    dn, dr, dv = 128, 64, 128
    T_ = Rows(size, pk)
    add = T_.add
    bf = lambda *s: torch.randn(*s, device=dev, dtype=torch.bfloat16)
    f32 = lambda *s: torch.randn(*s, device=dev)
    gen = torch.Generator(device=dev).manual_seed(0)
    freq, m = mixers.rotary_frequencies(latodra_config(size)["layers"][0]["mixer"]["rot"])
    rot = S.Rotation(torch.tensor(freq, dtype=torch.float64, device=dev), m)
    n_in = rq + R + dr
    # ---- prefill, 8 x 2048 tokens
    B, n = 8, 2048
    M = B * n
    pos = torch.zeros(1, dtype=torch.int32, device=dev)
    x = bf(M, width)

    def gemm(name, K, N, act=S.ACT_NONE, like="lut_gemm_pair (hard)"):
        xi, w = x if K == width else bf(M, K), bf(N, K) * K ** -0.5
        t = timed(torch, lambda _: S.linear(xi, w, act=act), 5)
        add(name, "prefill", t, 2.0 * (M * K + N * K + M * (N // 2 if act == S.ACT_GLU_GELU else N)), 2.0 * M * N * K, like)
    gemm("lut_gemm<dense, gated epilogue>", width, 2 * ff, S.ACT_GLU_GELU)
    gemm("lut_gemm<dense> latents", width, n_in, like="lut_gemm_pair (hard), as wide as the latents")
    gemm("lut_gemm<dense> queries", rq, H * (dn + dr))
    gemm("lut_gemm<dense> keys and values", R, H * (dn + dv))
    gemm("lut_gemm<dense> output", H * dv, width)
    if width % 256 == 0:
        pw = make_weight(torch, ops, ff, width, dev, gen)
        t = timed(torch, lambda _: ops.hard_forward(pw, x), 5)
        add("closest: lut_gemm_pair (hard)", "prefill", t, 2.0 * (M * width + M * ff) + ff * width / 4, 2.0 * M * ff * width)
        pw = make_weight(torch, ops, n_in // 64 * 64, width, dev, gen)
        t = timed(torch, lambda _: ops.hard_forward(pw, x), 5)
        add("closest: lut_gemm_pair (hard), as wide as the latents", "prefill", t, 2.0 * M * (width + pw.N) + pw.N * width / 4, 2.0 * M * pw.N * width)
    pairs = B * H * n * (n + 1) / 2
    kv, kr, sinks, gate = bf(B, n, H * (dn + dv)), bf(B, n, dr), f32(H), bf(M, H * dv)
    q = bf(M, H * (dn + dr))
    t = timed(torch, lambda _: S.attention_bias(q, kv, kv[:, :, H * dn:], None, pos, 0, B, n, H, H, dn + dr, dv, 192 ** -0.5, True, sinks, kr), 5)
    add("attn_bias_tc<3, 2> (rotated part, sinks)", "prefill", t, 2.0 * M * (H * (dn + dr + dn + dv + dv) + dr), 2.0 * pairs * (dn + dr + dv), "attn_fwd")
    qp = bf(M, H * dn)
    t = timed(torch, lambda _: S.attention_bias(qp, kv, kv[:, :, H * dn:], None, pos, 0, B, n, H, H, dn, dv, 128 ** -0.5, False, gate=gate), 5)
    add("attn_bias_tc<2, 2> (gate)", "prefill", t, 2.0 * M * H * (2 * dn + 3 * dv), 2.0 * pairs * (dn + dv), "attn_fwd")
    k1, v1 = bf(M, G * 128), bf(M, G * 128)
    t = timed(torch, lambda _: ops.attention_forward(qp, k1, v1, B, n, H, G), 5)
    add("closest: attn_fwd", "prefill", t, 2.0 * (2 * M * H * 128 + 2 * M * G * 128), 4.0 * pairs * 128)
    proj, cc, krc, wq, wc = bf(M, n_in), bf(B, n, R), bf(B, n, dr), f32(rq), f32(R)
    t = timed(torch, lambda _: S.latent_prep(proj, (0, rq, rq + R), wq, wc, cc, krc, rot, pos, B, n, 1e-6), 5)
    add("latent_prep", "prefill", t, 4.0 * M * n_in, like="qknorm_rope")
    qr = q.view(M, H, dn + dr)[:, :, dn:]
    t = timed(torch, lambda _: S.rotate(qr, qr, rot, pos, B, n), 5)
    add("rotate", "prefill", t, 4.0 * M * H * dr, like="qknorm_rope")
    cos, sin = ops.rope_tables(n, 128, 1e6, dev)
    nq = bf(128)
    qk = bf(M, (H + G) * 128)
    t = timed(torch, lambda _: ops.qknorm_rope_forward2(qk[:, :H * 128], nq, H, qk[:, H * 128:], nq, G, cos, sin, n), 5)
    add("closest: qknorm_rope", "prefill", t, 2.0 * M * 128 * 2 * (H + G))
    y, xr, out, nw, nx = bf(M, width), f32(M, width), bf(M, width), f32(width), f32(width)
    t = timed(torch, lambda _: S.stream_update(xr, torch.bfloat16, 1e-6, y, nw, 1.0, 0.0, w_next=nx, out=out), 5)
    add("stream (norm, residual, next norm)", "prefill", t, M * width * 12.0, like="rms (add)")
    t = timed(torch, lambda _: ops.add_rmsnorm_forward(y, out, nq.new_ones(width)), 5)
    add("closest: rms (add)", "prefill", t, M * width * 8.0)
    del x, kv, kr, gate, q, qp, k1, v1, proj, cc, krc, qk, y, xr, out
    # ---- decode, 2048 tokens cached
    T = 2048
    pos = torch.tensor([T - 1], dtype=torch.int32, device=dev)
    copies_of = lambda nbytes, most: max(1, min(most, int(3 * L2_BYTES // nbytes) + 1))
    for B in (1, 8, 64):
        ph = f"decode B{B}"
        shapes = (("latents", n_in, width, S.ACT_NONE), ("queries", H * (dn + dr), rq, S.ACT_NONE), ("output", width, H * dv, S.ACT_NONE),
                  ("gate / up", 2 * ff, width, S.ACT_GLU_GELU), ("down", width, ff, S.ACT_NONE))
        for name, N, K, act in shapes:
            c = copies_of(N * K * 2, 64)
            ws = [bf(N, K) for _ in range(c)]
            xi = bf(B, K)
            t = graphed(torch, lambda i: S.linear(xi, ws[i % c], act=act), c)
            add("Linear " + name, ph, t, 2.0 * N * K, 2.0 * B * N * K, "small-M LUT Linear")
            del ws
        if width % 256 == 0:
            xm = bf(B, width)
            c = copies_of(weight_bytes(ff, width), 200)
            pws = [make_weight(torch, ops, ff, width, dev, gen) for _ in range(c)]
            t = graphed(torch, lambda i: ops.hard_forward_smallm(pws[i % c], xm), c)
            add("closest: small-M LUT Linear", ph, t, weight_bytes(ff, width), 2.0 * B * ff * width)
            del pws
        for name, N, K in (("head_linear into the latent", R, dn), ("head_linear out of it (gate)", dv, R)):
            c = copies_of(H * N * K * 2, 64)
            ws = [bf(H, N, K) for _ in range(c)]
            xi, g = bf(B, H * K), bf(B, H * N) if N == dv else None
            t = graphed(torch, lambda i: S.head_linear(xi, K, ws[i % c], gate=g), c)
            add(name, ph, t, 2.0 * H * N * K + 2.0 * B * H * (N + K), 2.0 * B * H * N * K, "small-M LUT Linear")
            del ws
        kvb = B * T * (R + dr) * 2
        c = copies_of(kvb, 200)
        cs, krs = [bf(B, T, R) for _ in range(c)], [bf(B, T, dr) for _ in range(c)]
        qa, sinks = bf(B, H, R + dr), f32(H)
        t = graphed(torch, lambda i: S.latent_attention(qa, cs[i % c], krs[i % c], sinks, pos, -1, B, 1, 192 ** -0.5), c)
        add("latent_tc + combine", ph, t, kvb, 2.0 * B * T * H * (2 * R + dr), "attn_decode")
        del cs, krs
        kvb = 2 * B * T * G * 128 * 2
        c = copies_of(kvb, 48)
        ks, vs = [bf(B, T, G * 128) for _ in range(c)], [bf(B, T, G * 128) for _ in range(c)]
        qd = bf(B, H * 128)
        t = graphed(torch, lambda i: ops.attention_decode(qd, ks[i % c], vs[i % c], T, H, G), c)
        add("closest: attn_decode", ph, t, kvb)
        del ks, vs
        proj, cc, krc = bf(B, n_in), bf(B, T, R), bf(B, T, dr)
        t = graphed(torch, lambda i: S.latent_prep(proj, (0, rq, rq + R), wq, wc, cc, krc, rot, pos, B, 1, 1e-6), 20)
        add("latent_prep", ph, t, 4.0 * B * n_in, like="qknorm_rope")
        qr = bf(B, H * (dn + dr)).view(B, H, dn + dr)[:, :, dn:]
        t = graphed(torch, lambda i: S.rotate(qr, qa[:, :, R:], rot, pos, B, 1), 20)
        add("rotate", ph, t, 4.0 * B * H * dr, like="qknorm_rope")
        qk = bf(B, (H + G) * 128)
        t = graphed(torch, lambda i: ops.qknorm_rope_forward2(qk[:, :H * 128], nq, H, qk[:, H * 128:], nq, G, cos[:1], sin[:1], 1), 20)
        add("closest: qknorm_rope", ph, t, 2.0 * B * 128 * 2 * (H + G))
        y, xr, out = bf(B, width), f32(B, width), bf(B, width)
        t = graphed(torch, lambda i: S.stream_update(xr, torch.bfloat16, 1e-6, y, nw, 1.0, 0.0, w_next=nx, out=out), 20)
        add("stream (norm, residual, next norm)", ph, t, B * width * 12.0, like="rms (add)")
        one = nq.new_ones(width)
        t = graphed(torch, lambda i: ops.add_rmsnorm_forward(y, out, one), 20)
        add("closest: rms (add)", ph, t, B * width * 8.0)
    return T_.rows


def kernels(torch, size, dev, pk):
    """Rows of the per-kernel table at one size."""
    import plz_ops as ops
    import seq_ops as S
    width, ff, H, G, R, _ = SIZES[size]
    T_ = Rows(size, pk)
    add = T_.add
    bf = lambda *s: torch.randn(*s, device=dev, dtype=torch.bfloat16)
    f32 = lambda *s: torch.randn(*s, device=dev)
    dk = dv = 128
    unit = lambda t: (t.view(t.shape[0], -1, dk) / t.view(t.shape[0], -1, dk).norm(dim=-1, keepdim=True)).reshape(t.shape[0], -1).contiguous()
    # ---- prefill, 8 x 2048 tokens (every tensor exceeds L2 or nearly so)
    B, n = 8, 2048
    M = B * n
    pos = torch.zeros(1, dtype=torch.int32, device=dev)
    x = bf(M, width)
    w_up = bf(ff, width) * width ** -0.5
    t = timed(torch, lambda _: S.linear(x, w_up, act=S.ACT_RELU2), 5)
    add("lut_gemm<dense, relu^2 epilogue>", "prefill", t, 2.0 * (M * width + ff * width + M * ff), 2.0 * M * ff * width, "lut_gemm_pair (hard)")
    from bench import make_weight
    gen = torch.Generator(device=dev).manual_seed(0)
    if width % 256 == 0:
        pw = make_weight(torch, ops, ff, width, dev, gen)
        t = timed(torch, lambda _: ops.hard_forward(pw, x), 5)
        add("closest: lut_gemm_pair (hard)", "prefill", t, 2.0 * (M * width + M * ff) + ff * width / 4, 2.0 * M * ff * width)
    q, kc, vc = bf(M, H * dk), bf(B, n, G * dk), bf(B, n, G * dv)
    bias = S.DistanceBias.from_distances(f32(H, 512))
    afl = 4.0 * B * H * 128 * n * (n + 1) / 2
    ab = 2.0 * (2 * M * H * 128 + 2 * M * G * 128)
    t = timed(torch, lambda _: S.attention_bias(q, kc, vc, bias, pos, 0, B, n, H, G, dk, dv, dk ** -0.5, True), 5)
    add("attn_bias_tc", "prefill", t, ab, afl, "attn_fwd")
    t = timed(torch, lambda _: ops.attention_forward(q, kc.view(M, -1), vc.view(M, -1), B, n, H, G), 5)
    add("closest: attn_fwd", "prefill", t, ab, afl)
    proj = bf(M, (H + 2 * G) * 128)
    wq, wk, mix, vf = f32(H * dk), f32(G * dk), torch.tensor([0.3], device=dev), bf(M, G * dv)
    offs = (0, H * dk, (H + G) * dk)
    t = timed(torch, lambda _: S.attn_prep(proj, offs, wq, wk, mix, vf, False, kc, vc, pos, B, n, 1e-6), 5)
    add("attn_prep", "prefill", t, 2.0 * M * 128 * (2 * (H + 2 * G) + G), like="qknorm_rope")
    cos, sin = ops.rope_tables(n, 128, 1e6, dev)
    nq = bf(128)
    t = timed(torch, lambda _: ops.qknorm_rope_forward2(proj[:, :H * dk], nq, H, proj[:, H * dk:(H + G) * dk], nq, G, cos, sin, n), 5)
    add("closest: qknorm_rope", "prefill", t, 2.0 * M * 128 * 2 * (H + G))
    y, xr, xb, nw = bf(M, width), f32(M, width), bf(M, width), f32(width)
    t = timed(torch, lambda _: S.residual_norm(y, nw, 1.0, 0.7, 1e-6, xr, xb), 5)
    add("residual_norm", "prefill", t, M * width * (2 + 4 + 4 + 2.0), like="rms (add)")
    t = timed(torch, lambda _: ops.add_rmsnorm_forward(y, xb, nq.new_ones(width)), 5)
    add("closest: rms (add)", "prefill", t, M * width * 8.0)
    # recurrences
    qf, kf, vv, lg, be = unit(f32(M, R * dk)), unit(f32(M, R * dk)), f32(M, R * dv), -0.1 * torch.rand(M, R * dk, device=dev), torch.rand(M, R, device=dev)
    st = f32(B, R, dk, dv)
    # FLOPs of the recurrence as defined: S k, k u^T, S q per token and head; bytes of its inputs and output
    t = timed(torch, lambda _: S.delta_rule(qf, kf, vv, lg, be, st, B, n, R, R, dk, dv, True), 5)
    add("delta_chunk + chunk_scan", "prefill", t, M * R * 4.0 * (3 * dk + 2 * dv), 6.0 * M * R * dk * dv, "attn_fwd")
    dproj = bf(M, R * (2 * dk + 2 * dv))
    decay = torch.rand(R, device=dev)
    o_st = (dproj[:, :R * dk], dproj[:, R * dk:2 * R * dk], dproj[:, 2 * R * dk:2 * R * dk + R * dv], decay)
    t = timed(torch, lambda _: S.decay_attention(*o_st, st, B, n, R, dk, dv, True), 5)
    add("decay_chunk + chunk_scan", "prefill", t, M * R * (2.0 * (2 * dk + dv) + 4.0 * dv), 4.0 * M * R * dk * dv, "attn_fwd")
    C = R * (2 * dk + dv)
    pj = bf(M, C + 512)
    a2 = bf(M, R * dk)
    taps, al, db = f32(C, 4), f32(R), f32(R * dk)
    conv = torch.zeros(B, 3, C, device=dev, dtype=torch.bfloat16)
    t = timed(torch, lambda _: S.delta_prep(pj, (0, R * dk, 2 * R * dk, C), a2, taps, al, db, conv, B, n, R, R, dk, dv, dk ** -0.5), 5)
    add("delta_prep", "prefill", t, M * R * (2.0 * (2 * dk + dv) + 2.0 * dk + 4.0 * (3 * dk + dv)), like="qknorm_rope")
    of = f32(M, R * dv)
    t = timed(torch, lambda _: S.norm_gate(of, dproj[:, 2 * R * dk:2 * R * dk + R * dv], f32(dv), 1e-6, R), 5)
    add("norm_gate (per head)", "prefill", t, M * R * dv * 8.0, like="rms (add)")
    wn = f32(R * dv)
    t = timed(torch, lambda _: S.norm_gate(of, dproj[:, 2 * R * dk:2 * R * dk + R * dv], wn, 1e-6, 1), 5)
    add("norm_gate (all heads)", "prefill", t, M * R * dv * 8.0, like="rms (add)")
    del x, q, kc, vc, proj, vf, y, xr, xb, qf, kf, vv, lg, be, st, dproj, pj, a2, of
    # ---- decode
    from bench import weight_bytes
    T = 2048
    for B in (1, 8, 64):
        copies = max(1, min(64, 3 * L2_BYTES // (ff * width * 2) + 1))
        ws = [bf(ff, width) for _ in range(copies)]
        xm = bf(B, width)
        t = graphed(torch, lambda i: S.linear(xm, ws[i % copies], act=S.ACT_RELU2), copies)
        add("linear_rows" if B <= 8 else "lut_gemm<dense>", f"decode B{B}", t, 2.0 * ff * width, 2.0 * B * ff * width, "small-M LUT Linear")
        del ws
        if width % 256 == 0:
            copies = 3 * L2_BYTES // weight_bytes(ff, width) + 1
            copies = min(copies, 200)
            pws = [make_weight(torch, ops, ff, width, dev, gen) for _ in range(copies)]
            t = graphed(torch, lambda i: ops.hard_forward_smallm(pws[i % copies], xm), copies)
            add("closest: small-M LUT Linear", f"decode B{B}", t, weight_bytes(ff, width), 2.0 * B * ff * width)
            del pws
        kvb = 2 * B * T * G * 128 * 2
        copies = max(1, min(48, 3 * L2_BYTES // kvb + 1))
        ks, vs = [bf(B, T, G * dk) for _ in range(copies)], [bf(B, T, G * dv) for _ in range(copies)]
        pos = torch.tensor([T - 1], dtype=torch.int32, device=dev)
        qd = bf(B, H * dk)
        t = graphed(torch, lambda i: S.attention_bias(qd, ks[i % copies], vs[i % copies], bias, pos, -1, B, 1, H, G, dk, dv, dk ** -0.5, True), copies)
        add("attn_decode (bias, sink)", f"decode B{B}", t, kvb, 0.0, "attn_decode")
        t = graphed(torch, lambda i: ops.attention_decode(qd, ks[i % copies], vs[i % copies], T, H, G), copies)
        add("closest: attn_decode", f"decode B{B}", t, kvb)
        del ks, vs
        sb = 2 * B * R * dk * dv * 4
        copies = max(1, min(64, 3 * L2_BYTES // sb + 1))
        sts = [f32(B, R, dk, dv) for _ in range(copies)]
        qf, kf, vv, lg, be = f32(B, R * dk), unit(f32(B, R * dk)), f32(B, R * dv), -0.1 * torch.rand(B, R * dk, device=dev), torch.rand(B, R, device=dev)
        t = graphed(torch, lambda i: S.delta_rule(qf, kf, vv, lg, be, sts[i % copies], B, 1, R, R, dk, dv), copies)
        add("recurrent<delta>", f"decode B{B}", t, sb, like="attn_decode")
        dproj = bf(B, R * (2 * dk + 2 * dv))
        t = graphed(torch, lambda i: S.decay_attention(dproj[:, :R * dk], dproj[:, R * dk:2 * R * dk], dproj[:, 2 * R * dk:2 * R * dk + R * dv], decay, sts[i % copies], B, 1, R, dk, dv), copies)
        add("recurrent<decay>", f"decode B{B}", t, sb, like="attn_decode")
        del sts
    return T_.rows


def case(torch, dev, design="gopunex"):
    """One launch of every kernel of the design on a small case (width 1024, 2048 tokens, then three single tokens): for ncu."""
    import hybrid_model
    cfg = gopunex_config(*SIZES["small"][:5], 3) if design == "gopunex" else dict(latodra_config("small"), layers=latodra_config("small")["layers"][:2])
    m = hybrid_model.ARCHITECTURES[cfg["architecture"]].random(cfg, dev, seed=1)
    c = m.new_cache(1, 2048 + 8)
    m.prefill(torch.randint(0, VOCAB, (1, 2048), device=dev), c)
    m.use_graph = False
    for _ in range(3):
        m.decode_step(torch.zeros(1, dtype=torch.int64, device=dev), c)
    torch.cuda.synchronize()


def run(args, pk, sampler_cls):
    import torch
    import plz_native as P
    torch.cuda.set_device(0)
    dev = torch.device("cuda", 0)
    sampler = sampler_cls(0)
    sampler.start()
    for size in args.sizes.split(","):
        t0 = time.time()
        out = models(torch, args.design, size, dev, pk)
        rows = (kernels if args.design == "gopunex" else latodra_kernels)(torch, size, dev, pk)
        st = P.device_status()
        assert st[0] == 0, f"device status {st}"
        out["seconds"] = time.time() - t0
        print(json.dumps(out), flush=True)
        for r in rows:
            print(json.dumps(r), flush=True)
        torch.cuda.empty_cache()
    t1 = time.time()
    print(json.dumps({"clocks": sampler.stop(t1 - 60, t1)}), flush=True)
