// Causal attention with a per-head bias by distance and a sink on the tensor cores (tcgen05.mma, accumulators in TMEM), for a portion of
// n new tokens against the key / value cache that already holds them. bf16, key head sizes up to 192 in 64-column blocks, value head
// sizes up to 128 (multiples of 8), any n and any cache length.
//
// The structure is that of the plain causal kernel (attention.cu): one CTA takes two neighbouring 128-query tiles of a head and walks
// the key / value tiles they share once; warps 0-3 / 4-7 are the softmax groups of the two tiles (thread = query row = TMEM lane), warp 8
// issues TMA copies and MMAs, so that one group's exponentials run under the other group's products. What differs:
//   - tiles come through 4-D tensor maps (head column, head, token, sequence), so head sizes that are no multiple of 64, ragged token
//     counts and the end of the cache read as zeros and are clipped on the store;
//   - the first query sits at position pos of the sequence: a key tile may straddle the diagonal of two query rows' tiles, and every
//     element is masked by position where a tile touches the diagonal;
//   - the bias depends on i - j only: a tile row r, column c reads table[d0 + r - c], i.e. consecutive lanes read consecutive words.
//     A tile that lies wholly beyond the last table entry adds one constant per head, folded into the exponent;
//   - the running maximum uses the head's largest bias as a bound (any bound serves the softmax), so the bias is added once, in the
//     exponent of the second pass;
//   - with a sink the running maximum starts at its score (0 if it is not learned) and the denominator at 1;
//   - the last key columns may come from a second tensor that all heads share (a rotated part beside the heads' own), as blocks of their
//     own of the key tile;
//   - the weights P go back to TMEM over the scores they came from and are the A operand of P V from there; shared memory holds queries,
//     keys and values only, and the output leaves through the space of the queries;
//   - the output may be multiplied by the sigmoid of a gate on its way out.
#include "attention_tiles.cuh"

namespace plz {
namespace {

constexpr int kThreads = 288;   // warps 0..3 / 4..7: softmax of tile A / B, warp 8: TMA + MMA

struct TcParams {
    int n, H, G, pos;            // pos: position of the first query
    int k1_blocks;               // 64-column blocks of the heads' own keys; the others come from the shared tensor
    int k_steps[3];              // 16-wide reduction steps of Q K^T in each block
    int dv_blocks;               // 64-column boxes of the output
    float scale_log2e;
    const float* bias; long long ldb; int n_bias; const float* bias_top;
    int sink; const float* sinks;
    const __nv_bfloat16* gate; long long ldg; int dv;
    StatusWord* status;
};

template <int DKB, int DVB>
struct TcCfg {
    static constexpr uint32_t QK = DKB * kBlk, V = DVB * kBlk, QS = (DKB > DVB ? DKB : DVB) * kBlk;   // QS: a query tile, later the output
    static constexpr uint32_t OFF_K = 2 * QS, OFF_V = OFF_K + 2 * QK, OFF_BAR = OFF_V + V;
    static constexpr uint32_t SMEM = OFF_BAR + 1024 + 256;
};

template <int BLOCKS>
__device__ __forceinline__ void load_boxes(uint32_t dst, const CUtensorMap* map, uint32_t bar, int head, int tok, int b) {
#pragma unroll
    for (int i = 0; i < BLOCKS; ++i) tma_load_4d(dst + i * kBlk, map, bar, i * 64, head, tok, b);
}
// the first k1 blocks from one tensor, the others from a second one
template <int BLOCKS>
__device__ __forceinline__ void load_boxes2(uint32_t dst, const CUtensorMap* map, const CUtensorMap* map2, int k1, uint32_t bar, int head, int head2, int tok, int b) {
#pragma unroll
    for (int i = 0; i < BLOCKS; ++i) {
        if (i < k1) tma_load_4d(dst + i * kBlk, map, bar, i * 64, head, tok, b);
        else tma_load_4d(dst + i * kBlk, map2, bar, (i - k1) * 64, head2, tok, b);
    }
}

// S = Q K^T: both K-major
template <int DKB>
__device__ __forceinline__ void mma_qk(uint32_t d, uint32_t sQ, uint32_t sK, const int (&steps)[3]) {
    const uint32_t idesc = make_idesc(128, 128, 0, 0);
    const uint64_t ad = make_sdesc(sQ, 16u, 1024u), bd = make_sdesc(sK, 16u, 1024u);
#pragma unroll
    for (int i = 0; i < DKB; ++i) {
        for (int ks = 0; ks < steps[i]; ++ks) {
            const uint32_t off = (uint32_t)(i * (kBlk >> 4) + ks * 2);
            umma_bf16_words<1>(d, (uint32_t)ad + off, (uint32_t)(ad >> 32), (uint32_t)bd + off, (uint32_t)(bd >> 32), idesc, (i > 0 || ks > 0) ? 1u : 0u);
        }
    }
}
// O (+)= P V: P in TMEM, V MN-major (rows = keys)
template <int DVB>
__device__ __forceinline__ void mma_pv(uint32_t d, uint32_t tP, uint32_t sV, bool accumulate) {
    const uint32_t idesc = make_idesc(128, 64 * DVB, 0, 1);
    const uint64_t bd = make_sdesc(sV, kBlk, 1024u);
#pragma unroll
    for (int ks = 0; ks < 8; ++ks)
        umma_ts(d, tP + ks * 8u, (uint32_t)bd + (uint32_t)(ks * 128), (uint32_t)(bd >> 32), idesc, (ks > 0 || accumulate) ? 1u : 0u);
}

struct Group {
    uint32_t tS, tO, s_full, p_full, o_full, out_ready;
    uint8_t* pOut; uint32_t sOut;   // space of the query tile, free once the last scores are in
    int qt, n_kv;              // query tile; key tiles it walks
};

// MASK: some element of the tile may lie above the diagonal. NEAR: the bias varies over the tile.
template <bool MASK, bool NEAR>
__device__ __forceinline__ float exp_pass(const Group& G, uint32_t lane_off, int r, int lim, float c, float add, const float* brow) {
    float l_tile = 0.f;
#pragma unroll 1
    for (int cb = 0; cb < 4; ++cb) {
        float bb[32];
        if (NEAR) {
#pragma unroll
            for (int i = 0; i < 32; ++i) bb[i] = __ldg(brow - (cb * 32 + i));
        }
        uint32_t v[32], o[16];
        tmem_ld_32x32(G.tS + lane_off + cb * 32, v);
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            const int e = 2 * i, c0 = cb * 32 + e;
            const float a0 = NEAR ? fmaf(bb[e], kLog2e, add) : add, a1 = NEAR ? fmaf(bb[e + 1], kLog2e, add) : add;
            float p0 = exp2f(fmaf(__uint_as_float(v[e]), c, a0));
            float p1 = exp2f(fmaf(__uint_as_float(v[e + 1]), c, a1));
            if (MASK) { if (c0 > lim) p0 = 0.f; if (c0 + 1 > lim) p1 = 0.f; }
            l_tile += p0 + p1;
            o[i] = pack_bf16x2(p0, p1);
        }
        tmem_st_32x16(G.tS + lane_off + cb * 16, o);      // over columns of this row that have been read
    }
    tmem_wait_st();
    return l_tile;
}

template <int DVB>
__device__ __forceinline__ void softmax_group(const Group& G, const TcParams& p, const CUtensorMap* tmO, int h, int b, int warp_in_group, int lane,
                                              volatile uint32_t* abort_flag) {
    const int r = warp_in_group * 32 + lane;
    const uint32_t lane_off = (uint32_t)(warp_in_group * 32) << 16;
    const float c = p.scale_log2e;
    const int i0 = p.pos + G.qt * kT;                       // position of the tile's first query
    const float* bias = p.bias ? p.bias + (long long)h * p.ldb : nullptr;
    const float top = bias ? p.bias_top[h] * kLog2e : 0.f, far = bias ? bias[p.n_bias - 1] * kLog2e : 0.f;
    float m_run = p.sink ? (p.sinks ? p.sinks[h] * kLog2e : 0.f) : -INFINITY, l_run = p.sink ? 1.f : 0.f;
    bool ok = true;
    for (int j = 0; j < G.n_kv && ok; ++j) {
        ok = mbar_wait(G.s_full, j & 1, abort_flag, p.status, ST_TIMEOUT_ACCUM, 20);
        if (!ok) break;
        tc_fence_after_sync();
        const int d0 = i0 - j * kT;                         // distance of (row 0, column 0)
        const bool mask = d0 < kT - 1;
        const bool near = bias != nullptr && d0 - (kT - 1) < p.n_bias - 1;
        const int lim = d0 + r;                             // last visible column of this row
        float m_tile = -INFINITY;
#pragma unroll 1
        for (int cb = 0; cb < 4; ++cb) {
            uint32_t v[32];
            tmem_ld_32x32(G.tS + lane_off + cb * 32, v);
#pragma unroll
            for (int i = 0; i < 32; ++i)
                if (!mask || cb * 32 + i <= lim) m_tile = fmaxf(m_tile, __uint_as_float(v[i]));
        }
        const float m_new = fmaxf(m_run, fmaf(m_tile, c, near ? top : far));
        const float alpha = (m_run == -INFINITY) ? 0.f : exp2f(m_run - m_new);
        if (j > 0) {
            ok = mbar_wait(G.o_full, (j - 1) & 1, abort_flag, p.status, ST_TIMEOUT_ACCUM, 21);
            if (!ok) break;
            tc_fence_after_sync();
            if (__any_sync(0xFFFFFFFFu, m_new > m_run)) {
#pragma unroll 1
                for (int cb = 0; cb < 2 * DVB; ++cb) {
                    uint32_t v[32];
                    tmem_ld_32x32(G.tO + lane_off + cb * 32, v);
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
                    tmem_st_32x32(G.tO + lane_off + cb * 32, v);
                }
            }
        }
        // a row that has seen no key yet (all of the tile masked, no sink) keeps m = -inf: its exponents are all masked
        const float add = (m_new == -INFINITY ? 0.f : -m_new) + (near ? 0.f : far);
        const float* brow = near ? bias + d0 + r : nullptr;
        float l_tile;
        if (near) l_tile = mask ? exp_pass<true, true>(G, lane_off, r, lim, c, add, brow) : exp_pass<false, true>(G, lane_off, r, lim, c, add, brow);
        else l_tile = mask ? exp_pass<true, false>(G, lane_off, r, lim, c, add, brow) : exp_pass<false, false>(G, lane_off, r, lim, c, add, brow);
        l_run = l_run * alpha + l_tile;
        m_run = m_new;
        tc_fence_before_sync();
        __syncwarp();
        if (lane == 0) mbar_arrive(G.p_full);
    }
    if (ok) ok = mbar_wait(G.o_full, (G.n_kv - 1) & 1, abort_flag, p.status, ST_TIMEOUT_ACCUM, 22);
    if (ok) {
        tc_fence_after_sync();
        const float inv_l = l_run > 0.f ? 1.0f / l_run : 0.f;
        const __nv_bfloat16* gate = p.gate && G.qt * kT + r < p.n ? p.gate + ((long long)b * p.n + G.qt * kT + r) * p.ldg + (long long)h * p.dv : nullptr;
#pragma unroll 1
        for (int cb = 0; cb < 2 * DVB; ++cb) {
            uint32_t v[32];
            tmem_ld_32x32(G.tO + lane_off + cb * 32, v);
#pragma unroll
            for (int g = 0; g < 4; ++g) {
                uint32_t o[4];
                float f[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(v[g * 8 + i]) * inv_l;
                if (gate && cb * 32 + g * 8 < p.dv) {
                    const uint4 q = __ldg(reinterpret_cast<const uint4*>(gate + cb * 32 + g * 8));
                    const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        f[2 * i] *= __fdividef(1.0f, 1.0f + __expf(-__uint_as_float(w[i] << 16)));
                        f[2 * i + 1] *= __fdividef(1.0f, 1.0f + __expf(-__uint_as_float(w[i] & 0xFFFF0000u)));
                    }
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) o[i] = pack_bf16x2(f[2 * i], f[2 * i + 1]);
                *reinterpret_cast<uint4*>(tile_chunk(G.pOut, r, cb * 4 + g)) = make_uint4(o[0], o[1], o[2], o[3]);
            }
        }
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(G.out_ready);
        if (r == 0 && mbar_wait(G.out_ready, 0, abort_flag, p.status, ST_TIMEOUT_ACCUM, 23)) {
            for (int i = 0; i < p.dv_blocks; ++i) tma_store_4d(tmO, G.sOut + i * kBlk, i * 64, h, G.qt * kT, b);
            tma_store_commit();
            tma_store_wait_all();
        }
    }
}

template <int DKB, int DVB>
__global__ void __launch_bounds__(kThreads, 1)
attn_bias_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                    const __grid_constant__ CUtensorMap tmO, const __grid_constant__ CUtensorMap tmQ2, const __grid_constant__ CUtensorMap tmK2, const TcParams p) {
    using C = TcCfg<DKB, DVB>;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t* smem = smem_raw + (base - raw);
    const uint32_t sQ0 = base, sK0 = base + C::OFF_K, sV = base + C::OFF_V;
    const uint32_t bar = base + C::OFF_BAR;
    const uint32_t q_full = bar, k_full0 = bar + 8, k_empty0 = bar + 24, v_full = bar + 40, v_empty = bar + 48;
    auto s_full = [&](int g) { return bar + 56u + 8u * g; };
    auto p_full = [&](int g) { return bar + 72u + 8u * g; };
    auto o_full = [&](int g) { return bar + 88u + 8u * g; };
    auto out_ready = [&](int g) { return bar + 104u + 8u * g; };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + C::OFF_BAR + 128);
    volatile uint32_t* abort_flag = tmem_slot + 1;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n_qt = (p.n + kT - 1) / kT;
    const int n_pairs = (n_qt + 1) / 2;
    const int pi = n_pairs - 1 - (int)blockIdx.x;   // heavy pairs first
    const int qtA = 2 * pi, qtB = 2 * pi + 1;
    const bool hasB = qtB < n_qt;
    const int h = blockIdx.y, b = blockIdx.z;
    const int hk = h / (p.H / p.G);
    auto kv_tiles = [&](int qt) { return (p.pos + min(p.n, (qt + 1) * kT) + kT - 1) / kT; };
    const int n_kvA = kv_tiles(qtA);
    const int n_kv = hasB ? kv_tiles(qtB) : n_kvA;

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1); mbar_init(v_full, 1); mbar_init(v_empty, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(k_full0 + 8 * i, 1); mbar_init(k_empty0 + 8 * i, 1);
            mbar_init(s_full(i), 1); mbar_init(p_full(i), 4); mbar_init(o_full(i), 1); mbar_init(out_ready(i), 4);
        }
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 8) { tmem_alloc(smem_u32((const void*)tmem_slot), 512); tmem_relinquish(); }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *tmem_slot;
    auto tS = [&](int g) { return tmem + 128u * g; };
    auto tO = [&](int g) { return tmem + 256u + 128u * g; };

    if (warp == 8) {
        if (lane == 0) {
            tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
            mbar_arrive_expect_tx(q_full, hasB ? 2 * C::QK : C::QK);
            load_boxes2<DKB>(sQ0, &tmQ, &tmQ2, p.k1_blocks, q_full, h, h, qtA * kT, b);
            if (hasB) load_boxes2<DKB>(sQ0 + C::QS, &tmQ, &tmQ2, p.k1_blocks, q_full, h, h, qtB * kT, b);
            bool ok = true;
            for (int j = 0; j < 2 && j < n_kv; ++j) {
                mbar_arrive_expect_tx(k_full0 + 8 * j, C::QK);
                load_boxes2<DKB>(sK0 + j * C::QK, &tmK, &tmK2, p.k1_blocks, k_full0 + 8 * j, hk, 0, j * kT, b);
            }
            mbar_arrive_expect_tx(v_full, C::V);
            load_boxes<DVB>(sV, &tmV, v_full, hk, 0, b);
            ok = mbar_wait(q_full, 0, abort_flag, p.status, ST_TIMEOUT_FULL, 10);
            if (ok) ok = mbar_wait(k_full0, 0, abort_flag, p.status, ST_TIMEOUT_FULL, 11);
            if (ok) {
                tc_fence_after_sync();
                mma_qk<DKB>(tS(0), sQ0, sK0, p.k_steps);
                umma_commit(s_full(0));
                if (hasB) { mma_qk<DKB>(tS(1), sQ0 + C::QS, sK0, p.k_steps); umma_commit(s_full(1)); }
            }
            for (int j = 0; j < n_kv && ok; ++j) {
                const int s = j & 1, s1 = (j + 1) & 1;
                ok = mbar_wait(v_full, j & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 15);
                if (!ok) break;
#pragma unroll
                for (int g = 0; g < 2; ++g) {
                    const int n_g = g == 0 ? n_kvA : n_kv;
                    if ((g == 1 && !hasB) || j >= n_g) continue;
                    ok = mbar_wait(p_full(g), j & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 12);
                    if (!ok) break;
                    tc_fence_after_sync();
                    mma_pv<DVB>(tO(g), tS(g), sV, j > 0);
                    umma_commit(o_full(g));
                    if (j + 1 < n_g) {
                        ok = mbar_wait(k_full0 + 8 * s1, ((j + 1) >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 13);
                        if (!ok) break;
                        tc_fence_after_sync();
                        mma_qk<DKB>(tS(g), sQ0 + g * C::QS, sK0 + s1 * C::QK, p.k_steps);
                        umma_commit(s_full(g));
                    }
                }
                if (!ok) break;
                umma_commit(v_empty);
                umma_commit(k_empty0 + 8 * s);
                if (j + 1 < n_kv) {
                    ok = mbar_wait(v_empty, j & 1, abort_flag, p.status, ST_TIMEOUT_EMPTY, 16);
                    if (!ok) break;
                    mbar_arrive_expect_tx(v_full, C::V);
                    load_boxes<DVB>(sV, &tmV, v_full, hk, (j + 1) * kT, b);
                }
                if (j + 2 < n_kv) {
                    ok = mbar_wait(k_empty0 + 8 * s, (j >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_EMPTY, 14);
                    if (!ok) break;
                    mbar_arrive_expect_tx(k_full0 + 8 * s, C::QK);
                    load_boxes2<DKB>(sK0 + s * C::QK, &tmK, &tmK2, p.k1_blocks, k_full0 + 8 * s, hk, 0, (j + 2) * kT, b);
                }
            }
        }
    } else {
        const int g = warp >> 2;
        if (g == 0 || hasB) {
            Group G;
            G.tS = tS(g); G.tO = tO(g); G.s_full = s_full(g); G.p_full = p_full(g); G.o_full = o_full(g); G.out_ready = out_ready(g);
            G.pOut = smem + g * C::QS; G.sOut = sQ0 + g * C::QS; G.qt = g == 0 ? qtA : qtB; G.n_kv = g == 0 ? n_kvA : n_kv;
            softmax_group<DVB>(G, p, &tmO, h, b, warp & 3, lane, abort_flag);
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 8) { tc_fence_after_sync(); tmem_dealloc(tmem, 512); }
}

template <int DKB, int DVB>
int launch_t(const AttnBiasArgs& a, cudaStream_t stream) {
    using C = TcCfg<DKB, DVB>;
    CUtensorMap tmQ, tmK, tmV, tmO;
    int rc;
    const uint64_t keys = (uint64_t)a.host_pos + a.n;
    const int dk1 = a.dk - a.dk2;
    const uint64_t qb = (uint64_t)a.n * a.ldq;
    if ((rc = make_tmap_bf16_heads(&tmQ, a.q, dk1, a.H, a.n, a.B, a.ldq, qb, kT, a.dk))) return rc;
    if ((rc = make_tmap_bf16_heads(&tmK, a.k, dk1, a.G, keys, a.B, a.k_tok, a.k_batch, kT))) return rc;
    if ((rc = make_tmap_bf16_heads(&tmV, a.v, a.dv, a.G, keys, a.B, a.v_tok, a.v_batch, kT))) return rc;
    if ((rc = make_tmap_bf16_heads(&tmO, a.o, a.dv, a.H, a.n, a.B, a.ldo, (uint64_t)a.n * a.ldo, kT))) return rc;
    CUtensorMap tmQ2 = tmQ, tmK2 = tmK;
    if (a.k2) {
        if ((rc = make_tmap_bf16_heads(&tmQ2, (const __nv_bfloat16*)a.q + dk1, a.dk2, a.H, a.n, a.B, a.ldq, qb, kT, a.dk))) return rc;
        if ((rc = make_tmap_bf16_heads(&tmK2, a.k2, a.dk2, 1, keys, a.B, a.dk2, a.k2_batch, kT))) return rc;
    }
    TcParams p = {};
    p.n = a.n; p.H = a.H; p.G = a.G; p.pos = a.host_pos; p.dv_blocks = (a.dv + 63) / 64;
    p.k1_blocks = (dk1 + 63) / 64;
    for (int i = 0; i < DKB; ++i) {
        const int left = i < p.k1_blocks ? dk1 - 64 * i : a.dk2 - 64 * (i - p.k1_blocks);
        p.k_steps[i] = ((left < 64 ? left : 64) + 15) / 16;
    }
    p.scale_log2e = a.scale * kLog2e; p.bias = a.bias; p.ldb = a.ldb; p.n_bias = a.n_bias; p.bias_top = a.bias_top; p.sink = a.sink || a.sinks; p.sinks = a.sinks;
    p.gate = (const __nv_bfloat16*)a.gate; p.ldg = a.ldg; p.dv = a.dv;
    p.status = device_status_ptr();
    auto kern = attn_bias_tc_kernel<DKB, DVB>;
    static bool once[64] = {};
    int dev = 0;
    PLZ_CUDA_CHECK(cudaGetDevice(&dev));
    if (!once[dev & 63]) { PLZ_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM)); once[dev & 63] = true; }
    const int n_qt = (a.n + kT - 1) / kT;
    kern<<<dim3((n_qt + 1) / 2, a.H, a.B), kThreads, C::SMEM, stream>>>(tmQ, tmK, tmV, tmO, tmQ2, tmK2, p);
    PLZ_LAUNCH_CHECK();
    return PLZ_OK;
}

}  // namespace

// n >= 2 tokens, bf16, key parts and dv multiples of 8, at most three 64-column blocks of keys and dv <= 128, 16-byte aligned rows,
// positive scale, host_pos known
int launch_attn_bias_tc(const AttnBiasArgs& a, cudaStream_t stream) {
    const int blocks = (a.dk - a.dk2 + 63) / 64 + (a.dk2 + 63) / 64;
    if (blocks == 1) return a.dv <= 64 ? launch_t<1, 1>(a, stream) : launch_t<1, 2>(a, stream);
    if (blocks == 2) return a.dv <= 64 ? launch_t<2, 1>(a, stream) : launch_t<2, 2>(a, stream);
    return a.dv <= 64 ? launch_t<3, 1>(a, stream) : launch_t<3, 2>(a, stream);
}

}  // namespace plz
