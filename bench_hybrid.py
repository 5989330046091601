"""bench.py --workload hybrid: the Gopunex decoder (lightning, channel-delta and distance-bias attention layers in turn) beside
PalettizedQwen at equal width, feed-forward width, attention heads and depth; random weights, synthetic tokens.

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
VOCAB = 32768
L2_BYTES = 126 << 20


def gopunex_config(width, ff, H, G, R, n_layers):
    mix = {"lightning": {"decay": [0.9 + 0.099 * i / R for i in range(R)], "dim": 128, "heads": R, "vdim": 128},
           "channel_delta": {"conv": 4, "dim": 128, "heads": R, "kv_heads": R, "vdim": 128},
           "attention": {"bias_max": 512, "dim": 128, "heads": H, "kv_heads": G, "scale": 128 ** -0.5, "v_mix": True, "vdim": 128}}
    order = ["lightning", "channel_delta", "attention"]
    return {"architecture": "Gopunex", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "residual_mult": 0.7, "vocab": VOCAB, "width": width,
            "layers": [{"type": order[i % 3], "mixer": mix[order[i % 3]], "mlp": {"ff": ff, "kind": "dense"}} for i in range(n_layers)]}


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


def models(torch, size, dev, pk):
    import decode_model as DM
    import plz_native as P
    from hybrid_model import Gopunex
    width, ff, H, G, R, n_layers = SIZES[size]
    gop = Gopunex.random(gopunex_config(*SIZES[size]), dev, seed=1)
    qwen = DM.PalettizedQwen.random(DM.ModelConfig(hidden=width, n_heads=H, n_kv_heads=G, head_dim=128, intermediate=ff, n_layers=n_layers, vocab=VOCAB),
                                    dev, seed=1, max_positions=4096)
    out = {"workload": "hybrid", "size": size, "width": width, "ff": ff, "attention_heads": [H, G], "recurrent_heads": R, "layers": n_layers, "vocab": VOCAB,
           "weights": "random", "peaks": pk, "prefill": {}, "decode": {}}
    for B, S in ((1, 2048), (8, 2048)):
        ids = torch.randint(0, VOCAB, (B, S), device=dev)
        cg = gop.new_cache(B, S + 64)
        cq = qwen.new_cache(B, S + 64)

        def pg(_):
            cg.reset()
            gop.prefill(ids, cg)

        def pq(_):
            cq.reset()
            qwen.prefill(ids, cq)
        tg, tq = timed(torch, pg, 5), timed(torch, pq, 5)
        out["prefill"][f"B{B}_S{S}"] = {"gopunex_ms": tg, "gopunex_tok_s": B * S / tg * 1e3, "palettized_qwen_ms": tq, "palettized_qwen_tok_s": B * S / tq * 1e3}
        del cg, cq
    for B in (1, 8, 64):
        T, steps = 2048, 20
        cg = gop.new_cache(B, T + 64)
        cg.length = T
        cg.pos.fill_(T)
        tok = torch.randint(0, VOCAB, (B,), device=dev)
        tg = timed(torch, lambda _: gop.decode_step(tok, cg), steps, warm=4)
        cq = qwen.new_cache(B, T + 64)
        g = None
        try:
            g, _ = qwen.decode_graph(tok, cq, T)
            tq = timed(torch, lambda _: g.replay(), steps)
        except P.PlzError:          # its small-M launch has no form for this batch and width
            P.lib().plz_set_smallm_overlap(0)
            tq = None
        out["decode"][f"B{B}_T{T}"] = {"gopunex_ms": tg, "gopunex_tok_s": B / tg * 1e3, "palettized_qwen_ms": tq, "palettized_qwen_tok_s": B / tq * 1e3 if tq else None,
                                       "gopunex_weight_and_state_bytes": gop.weight_bytes() + cg.nbytes() + sum(st["S"].numel() * 4 for st in cg.layers if "S" in st)}
        del cg, cq, g
    return out


def kernels(torch, size, dev, pk):
    """Rows of the per-kernel table at one size."""
    import plz_ops as ops
    import seq_ops as S
    width, ff, H, G, R, _ = SIZES[size]
    bw, fl_peak = pk["hbm_gbs"] * 1e9, pk["tflops_burst"] * 1e12
    rows = []

    def add(kernel, phase, ms, nbytes, flops=0.0, like=None):
        ideal = max(nbytes / bw, flops / fl_peak) * 1e3
        rows.append({"kernel": kernel, "size": size, "phase": phase, "us": ms * 1e3, "MB": nbytes / 1e6, "GFLOP": flops / 1e9, "bound": "flops" if flops / fl_peak > nbytes / bw else "bytes",
                     "frac_of_roofline": ideal / ms, "like": like})
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
    return rows


def case(torch, dev):
    """One launch of every kernel of the design on a small case (width 1024, 2048 tokens, then three single tokens): for ncu."""
    from hybrid_model import Gopunex
    m = Gopunex.random(gopunex_config(*SIZES["small"][:5], 3), dev, seed=1)
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
        out = models(torch, size, dev, pk)
        rows = kernels(torch, size, dev, pk)
        st = P.device_status()
        assert st[0] == 0, f"device status {st}"
        out["seconds"] = time.time() - t0
        print(json.dumps(out), flush=True)
        for r in rows:
            print(json.dumps(r), flush=True)
        torch.cuda.empty_cache()
    t1 = time.time()
    print(json.dumps({"clocks": sampler.stop(t1 - 60, t1)}), flush=True)
