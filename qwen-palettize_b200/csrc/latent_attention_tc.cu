// Attention over cached latents on the tensor cores (tcgen05.mma, accumulators in TMEM): a few query rows (token, head) against many cached
// tokens, bf16, latents up to 512 columns. It serves single tokens and short portions, where the cache is read once and every row of it
// meets all heads.
//
// Everything is transposed, so that the long dimensions are the 128-row side of the products and the query rows (16 .. 64) the narrow one:
//   S^T [key = TMEM lane][query row]      = [C | KR] Q^T      the cached tile as it lies (K-major), queries K-major
//   O^T [latent column = lane][query row] += C^T P^T          the SAME shared-memory tile read MN-major, P^T written by the softmax threads
// A cached byte enters shared memory once and serves as key and as value.
//
// One CTA takes N query rows of a sequence and one split of its keys, 128 keys at a time. Warps 0-3 are the softmax threads (thread = key),
// warp 4 issues the MMAs, warp 5 the copies. A tile arrives as units of 128 latent columns (32 KB) in a ring plus the shared key part; a unit
// is handed back as soon as the value product of its columns has run, so that the next tile streams in under the rest of the current one.
// The maximum of a query row runs over the lanes: 31 shuffles per 32 rows inside a warp, the four warps meet in shared memory. The reference
// of the exponentials moves only when the maximum has grown by more than 8 (in log2 units), so O^T is rarely rescaled. Rows of the last
// tile beyond the sequence are cleared in shared memory (a weight of zero times whatever lies there would not be safe).
// Partial sums of the key splits go to the workspace that latent_combine_kernel merges.
#include "attention_tiles.cuh"
#include "latent_attention.cuh"

namespace plz {
namespace {

constexpr int kLatThreads = 192;
constexpr uint32_t kUnit = 2 * kBlk;            // 128 keys x 128 latent columns
constexpr uint32_t kPBytes = 128 * 128;         // P^T: 128 keys x 64 query rows
constexpr int kMaxUnits = 8;
constexpr uint32_t kSmemBudget = 227 * 1024 - 1024 - 5120;   // alignment; barriers and softmax exchange (kExtra)
constexpr uint32_t kExtra = 5120;
constexpr float kLazy = 8.0f;

struct LatTcParams {
    LatentParams l;
    const int* pos;
    int units, c_blocks, r_blocks;              // per tile: units of c, 64-column blocks of c and of kr
    int ring, r_ring;                           // resident units, resident copies of the shared key part
    uint32_t off_r, off_p, off_q, off_x;
    uint32_t tmem_cols;
    StatusWord* status;
};

template <int W, bool MAX>
__device__ __forceinline__ float over_lanes(float (&v)[W], int lane) {     // lane (mod W) gets the result of column lane (mod W)
#pragma unroll
    for (int half = W / 2; half >= 1; half >>= 1) {
        const bool up = (lane & half) != 0;
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float send = up ? v[i] : v[i + half], keep = up ? v[i + half] : v[i];
            const float got = __shfl_xor_sync(0xFFFFFFFFu, send, half);
            v[i] = MAX ? fmaxf(keep, got) : keep + got;
        }
    }
    float r = v[0];
    if (W == 16) {
        const float got = __shfl_xor_sync(0xFFFFFFFFu, r, 16);
        r = MAX ? fmaxf(r, got) : r + got;
    }
    return r;
}

// N / 16 groups of 16 columns from TMEM
template <int N>
__device__ __forceinline__ void load_cols(uint32_t t, float (&s)[N]) {
#pragma unroll
    for (int g = 0; g < N / 32; ++g) {
        uint32_t v[32];
        tmem_ld_32x32(t + g * 32, v);
#pragma unroll
        for (int i = 0; i < 32; ++i) s[g * 32 + i] = __uint_as_float(v[i]);
    }
    if (N % 32) {
        uint32_t v[16];
        tmem_ld_32x16(t + N / 32 * 32, v);
#pragma unroll
        for (int i = 0; i < 16; ++i) s[N / 32 * 32 + i] = __uint_as_float(v[i]);
    }
}
template <int N>
__device__ __forceinline__ void store_cols(uint32_t t, const float (&s)[N]) {
#pragma unroll
    for (int g = 0; g < N / 32; ++g) {
        uint32_t v[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(s[g * 32 + i]);
        tmem_st_32x32(t + g * 32, v);
    }
    if (N % 32) {
        uint32_t v[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(s[N / 32 * 32 + i]);
        tmem_st_32x16(t + N / 32 * 32, v);
        tmem_wait_st();
    }
}
// result of every column over the 32 lanes: lane i gets columns i (r[0]) and, for N > 32, 32 + i (mod 16 for a group of 16; r[1])
template <int N, bool MAX>
__device__ __forceinline__ void columns_over_lanes(const float (&s)[N], int lane, float (&r)[2]) {
    if (N >= 32) {
        float t[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) t[i] = s[i];
        r[0] = over_lanes<32, MAX>(t, lane);
    }
    if (N == 64) {
        float t[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) t[i] = s[N - 32 + i];
        r[1] = over_lanes<32, MAX>(t, lane);
    }
    if (N % 32) {
        float t[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) t[i] = s[N - 16 + i];
        r[N / 32] = over_lanes<16, MAX>(t, lane);
    }
}

template <int N>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmR, const __grid_constant__ CUtensorMap tmQ,
                 const __grid_constant__ CUtensorMap tmQr, const LatTcParams p) {
    constexpr int G = (N + 31) / 32;            // column groups of a lane
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t* smem = smem_raw + (base - raw);
    const uint32_t bar = base + p.off_x;
    auto u_full = [&](int s) { return bar + 8u * s; };
    auto u_empty = [&](int s) { return bar + 64u + 8u * s; };
    auto r_full = [&](int s) { return bar + 128u + 8u * s; };
    auto r_empty = [&](int s) { return bar + 144u + 8u * s; };
    auto s_full = [&](int s) { return bar + 160u + 8u * s; };
    const uint32_t q_full = bar + 176, p_full = bar + 184, o_done = bar + 192, mx_full = bar + 200;
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + p.off_x + 208);
    volatile uint32_t* abort_flag = tmem_slot + 1;
    float* wmax = reinterpret_cast<float*>(smem + p.off_x + 256);         // [2][4][64]
    float* own = wmax + 2 * 4 * 64;                                       // per warp: [64] reference, [64] correction

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = blockIdx.x, r0 = (int)blockIdx.y * N, b = blockIdx.z;
    const int rows = p.l.n * p.l.H, H = p.l.H, R = p.l.R;
    if (threadIdx.x == 0) {
        for (int s = 0; s < kMaxUnits; ++s) { mbar_init(u_full(s), 1); mbar_init(u_empty(s), 1); }
        for (int s = 0; s < 2; ++s) { mbar_init(r_full(s), 1); mbar_init(r_empty(s), 1); mbar_init(s_full(s), 1); }
        mbar_init(q_full, 1); mbar_init(p_full, 4); mbar_init(o_done, 1); mbar_init(mx_full, 4);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 4) { tmem_alloc(smem_u32((const void*)tmem_slot), p.tmem_cols); tmem_relinquish(); }
    if (warp == 5 && lane == 0) { tma_prefetch_desc(&tmC); tma_prefetch_desc(&tmQ); if (p.r_blocks) { tma_prefetch_desc(&tmR); tma_prefetch_desc(&tmQr); } }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *tmem_slot;
    auto tS = [&](int s) { return tmem + (uint32_t)(s * N); };
    auto tO = [&](int m) { return tmem + (uint32_t)((2 + m) * N); };

    pdl_launch_dependents();
    pdl_wait();
    const int pos = *p.pos;
    const int total = pos + (min(rows, r0 + N) - 1) / H + 1;              // keys that some row of this CTA sees
    int chunk = (total + p.l.splits - 1) / p.l.splits;
    chunk = (chunk + kT - 1) / kT * kT;
    const int k0 = split * chunk, k1 = min(total, k0 + chunk);
    const int tiles = k1 > k0 ? (k1 - k0 + kT - 1) / kT : 0;

    if (warp == 5) {
        if (lane == 0 && tiles > 0) {
            bool ok = true;
            mbar_arrive_expect_tx(q_full, (uint32_t)(p.c_blocks + p.r_blocks) * N * 128u);
            for (int i = 0; i < p.c_blocks; ++i) tma_load_4d(base + p.off_q + i * N * 128, &tmQ, q_full, i * 64, 0, r0, b);
            for (int i = 0; i < p.r_blocks; ++i) tma_load_4d(base + p.off_q + (p.c_blocks + i) * N * 128, &tmQr, q_full, i * 64, 0, r0, b);
            int idx = 0, nr = 0;                // units and key parts issued
            for (int j = 0; j < tiles && ok; ++j) {
                const int tok = k0 + j * kT;
                if (p.r_blocks) {
                    const int s = j % p.r_ring;
                    if (j >= p.r_ring) ok = mbar_wait(r_empty(s), (j / p.r_ring - 1) & 1, abort_flag, p.status, ST_TIMEOUT_EMPTY, 80);
                    if (!ok) break;
                    mbar_arrive_expect_tx(r_full(s), (uint32_t)p.r_blocks * kBlk);
                    for (int i = 0; i < p.r_blocks; ++i) tma_load_4d(base + p.off_r + (s * p.r_blocks + i) * kBlk, &tmR, r_full(s), i * 64, 0, tok, b);
                    ++nr;
                }
                for (int m = 0; m < p.units; ++m) {
                    const int s = idx % p.ring;
                    if (idx >= p.ring) ok = mbar_wait(u_empty(s), (idx / p.ring - 1) & 1, abort_flag, p.status, ST_TIMEOUT_EMPTY, 81);
                    if (!ok) break;
                    const int nb = min(2, p.c_blocks - 2 * m);
                    mbar_arrive_expect_tx(u_full(s), (uint32_t)nb * kBlk);
                    for (int i = 0; i < nb; ++i) tma_load_4d(base + s * kUnit + i * kBlk, &tmC, u_full(s), (2 * m + i) * 64, 0, tok, b);
                    ++idx;
                }
            }
            // every copy has landed before the CTA exits (bounded: another role may have given up)
            const uint64_t t0 = globaltimer_ns();
            while (!mbar_try_wait(q_full, 0) && globaltimer_ns() - t0 < 100000000ull) {}
            for (int i = idx > p.ring ? idx - p.ring : 0; i < idx; ++i)
                while (!mbar_try_wait(u_full(i % p.ring), (i / p.ring) & 1) && globaltimer_ns() - t0 < 100000000ull) {}
            for (int i = nr > p.r_ring ? nr - p.r_ring : 0; i < nr; ++i)
                while (!mbar_try_wait(r_full(i % p.r_ring), (i / p.r_ring) & 1) && globaltimer_ns() - t0 < 100000000ull) {}
        }
    } else if (warp == 4) {
        if (lane == 0 && tiles > 0) {
            const uint32_t id_s = make_idesc(128, N, 0, 0), id_o = make_idesc(128, N, 1, 1);
            const uint64_t dq = make_sdesc(base + p.off_q, 16u, 1024u), dp = make_sdesc(base + p.off_p, kBlk, 1024u);
            const bool ahead = p.ring >= 2 * p.units && (p.r_blocks == 0 || p.r_ring == 2);
            bool ok = mbar_wait(q_full, 0, abort_flag, p.status, ST_TIMEOUT_FULL, 82);
            // one 64-column block of S^T
            auto block = [&](int buf, uint32_t sA, int q_block, int cols, uint32_t& acc) {
                const uint64_t da = make_sdesc(sA, 16u, 1024u);
                const uint32_t bq = (uint32_t)dq + (uint32_t)(q_block * N * 8);
                const int steps = (min(64, cols) + 15) >> 4;
                for (int ks = 0; ks < steps; ++ks) {
                    umma_bf16_words<1>(tS(buf), (uint32_t)da + ks * 2u, (uint32_t)(da >> 32), bq + ks * 2u, (uint32_t)(dq >> 32), id_s, acc);
                    acc = 1u;
                }
            };
            auto scores = [&](int j) {
                uint32_t acc = 0u;
                if (p.r_blocks) {
                    const int s = j % p.r_ring;
                    if (!mbar_wait(r_full(s), (j / p.r_ring) & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 83)) return false;
                    tc_fence_after_sync();
                    for (int i = 0; i < p.r_blocks; ++i) block(j & 1, base + p.off_r + (s * p.r_blocks + i) * kBlk, p.c_blocks + i, p.l.dr - 64 * i, acc);
                    umma_commit(r_empty(s));
                }
                for (int m = 0; m < p.units; ++m) {
                    const int idx = j * p.units + m, s = idx % p.ring;
                    if (!mbar_wait(u_full(s), (idx / p.ring) & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 84)) return false;
                    tc_fence_after_sync();
                    for (int i = 0; i < min(2, p.c_blocks - 2 * m); ++i) block(j & 1, base + s * kUnit + i * kBlk, 2 * m + i, R - 64 * (2 * m + i), acc);
                }
                umma_commit(s_full(j & 1));
                return true;
            };
            if (ok) ok = scores(0);
            for (int j = 0; j < tiles && ok; ++j) {
                if (ahead && j + 1 < tiles) { ok = scores(j + 1); if (!ok) break; }
                ok = mbar_wait(p_full, j & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 85);
                if (!ok) break;
                tc_fence_after_sync();
                for (int m = 0; m < p.units; ++m) {
                    const int s = (j * p.units + m) % p.ring;
                    const uint64_t da = make_sdesc(base + s * kUnit, kBlk, 1024u);
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks)
                        umma_bf16_words<1>(tO(m), (uint32_t)da + ks * 128u, (uint32_t)(da >> 32), (uint32_t)dp + ks * 128u, (uint32_t)(dp >> 32), id_o, (j > 0 || ks > 0) ? 1u : 0u);
                    umma_commit(u_empty(s));
                }
                umma_commit(o_done);
                if (!ahead && j + 1 < tiles) ok = scores(j + 1);
            }
        }
    } else {
        const int t = threadIdx.x;                                        // key of the tile = TMEM lane
        const uint32_t lane_off = (uint32_t)(warp * 32) << 16;
        const float c = p.l.scale * kLatLog2e;
        const int lim0 = pos + r0 / H;                                    // last key that every row of this CTA sees
        float* my_m = own + warp * 128;
        float* my_a = my_m + 64;
        float l[N], m_run[2] = {kLatNegBig, kLatNegBig};
#pragma unroll
        for (int i = 0; i < N; ++i) l[i] = 0.f;
        // a warp goes on or gives up as one
        auto wait = [&](uint32_t mbar, uint32_t parity, uint32_t role) {
            return __all_sync(0xFFFFFFFFu, mbar_wait(mbar, parity, abort_flag, p.status, ST_TIMEOUT_ACCUM, role)) != 0;
        };
        bool ok = true;
        for (int j = 0; j < tiles && ok; ++j) {
            const int tok = k0 + j * kT + t;
            ok = wait(s_full(j & 1), (j >> 1) & 1, 86);
            if (!ok) break;
            tc_fence_after_sync();
            float s[N];
            load_cols<N>(tS(j & 1) + lane_off, s);
            if (k0 + j * kT + kT - 1 > min(lim0, k1 - 1)) {               // some key of the tile is hidden from some row
#pragma unroll
                for (int i = 0; i < N; ++i)
                    if (tok >= k1 || tok > pos + (r0 + i) / H) s[i] = -INFINITY;
            }
#pragma unroll
            for (int i = 0; i < N; ++i) s[i] *= c;
            float mx[2];
            columns_over_lanes<N, true>(s, lane, mx);
            float* w = wmax + (j & 1) * 256 + warp * 64;
            w[lane] = mx[0];
            if (G == 2) w[32 + lane] = mx[1];
            __syncwarp();
            if (lane == 0) mbar_arrive(mx_full);
            ok = wait(mx_full, j & 1, 87);
            if (!ok) break;
            bool moved = false;
#pragma unroll
            for (int g = 0; g < G; ++g) {
                const float* a = wmax + (j & 1) * 256 + g * 32 + lane;
                const float m = fmaxf(fmaxf(a[0], a[64]), fmaxf(a[128], a[192]));
                const bool up = m > m_run[g] + kLazy;
                my_a[g * 32 + lane] = up ? exp2f(m_run[g] - m) : 1.0f;
                if (up) m_run[g] = m;
                my_m[g * 32 + lane] = m_run[g];
                moved |= up;
            }
            moved = __any_sync(0xFFFFFFFFu, moved);                       // the same in all four warps; orders the writes above
            __syncwarp();
#pragma unroll
            for (int i = 0; i < N; i += 4) {
                const float4 m = *reinterpret_cast<const float4*>(my_m + i);
                s[i] = exp2f(s[i] - m.x); s[i + 1] = exp2f(s[i + 1] - m.y); s[i + 2] = exp2f(s[i + 2] - m.z); s[i + 3] = exp2f(s[i + 3] - m.w);
            }
            if (moved) {
#pragma unroll
                for (int i = 0; i < N; ++i) l[i] = fmaf(l[i], my_a[i], s[i]);
            } else {
#pragma unroll
                for (int i = 0; i < N; ++i) l[i] += s[i];
            }
            if (j > 0) {                                                  // P^T and O^T are free once the products of the tile before have run
                ok = wait(o_done, (j - 1) & 1, 88);
                if (!ok) break;
                tc_fence_after_sync();
                if (moved) {
#pragma unroll 1
                    for (int m = 0; m < p.units; ++m) {
                        float o[N];
                        load_cols<N>(tO(m) + lane_off, o);
#pragma unroll
                        for (int i = 0; i < N; ++i) o[i] *= my_a[i];
                        store_cols<N>(tO(m) + lane_off, o);
                    }
                }
            }
#pragma unroll
            for (int q = 0; q < N / 8; ++q)
                *reinterpret_cast<uint4*>(smem + p.off_p + swz128(t, q)) =
                    make_uint4(pack_bf16x2(s[q * 8], s[q * 8 + 1]), pack_bf16x2(s[q * 8 + 2], s[q * 8 + 3]), pack_bf16x2(s[q * 8 + 4], s[q * 8 + 5]),
                               pack_bf16x2(s[q * 8 + 6], s[q * 8 + 7]));
            if (tok >= total) {                                           // past the sequence: whatever the cache holds there must not count
                for (int m = 0; m < p.units; ++m) {
                    uint8_t* u = smem + ((j * p.units + m) % p.ring) * kUnit + t * 128;
#pragma unroll
                    for (int i = 0; i < 16; ++i) *reinterpret_cast<uint4*>(u + (i >> 3) * kBlk + (i & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
                }
            }
            tc_fence_before_sync();
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
        }
        if (ok && tiles > 0) ok = wait(o_done, (tiles - 1) & 1, 89);
        if (ok) {
            const long long row0 = (long long)b * rows + r0;
            const int S = p.l.splits;
            if (tiles > 0) {
                tc_fence_after_sync();
#pragma unroll 1
                for (int m = 0; m < p.units; ++m) {
                    float o[N];
                    load_cols<N>(tO(m) + lane_off, o);
                    const int d = m * 128 + t;
                    if (d < R) {
                        float* dst = p.l.ws_o + (row0 * S + split) * R + d;
#pragma unroll
                        for (int i = 0; i < N; ++i)
                            if (r0 + i < rows) dst[(long long)i * S * R] = o[i];
                    }
                }
            }
            float ls[2];
            columns_over_lanes<N, false>(l, lane, ls);
            // the exchange buffer of the other parity than the last tile's
            float* w = wmax + (tiles & 1) * 256 + warp * 64;
            w[lane] = ls[0];
            if (G == 2) w[32 + lane] = ls[1];
            __syncwarp();
            if (lane == 0) mbar_arrive(mx_full);
            ok = wait(mx_full, tiles & 1, 90);
            if (ok && warp == 0) {
#pragma unroll
                for (int g = 0; g < G; ++g) {
                    const int i = g * 32 + lane;
                    const float* a = wmax + (tiles & 1) * 256 + i;
                    if (i < N && r0 + i < rows) {
                        float* ml = p.l.ws_ml + ((row0 + i) * S + split) * 2;
                        ml[0] = m_run[g];
                        ml[1] = a[0] + a[64] + a[128] + a[192];
                    }
                }
            }
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 4) { tc_fence_after_sync(); tmem_dealloc(tmem, p.tmem_cols); }
}

// shared-memory plan of a CTA with N query rows; false if it does not fit
bool plan(int R, int dr, int N, LatTcParams* p) {
    p->c_blocks = (R + 63) / 64; p->r_blocks = (dr + 63) / 64; p->units = (R + 127) / 128;
    const uint32_t fixed = kPBytes + (uint32_t)(p->c_blocks + p->r_blocks) * N * 128;
    const uint32_t part = (uint32_t)p->r_blocks * kBlk;
    if (fixed + part + p->units * kUnit > kSmemBudget) return false;
    p->r_ring = fixed + 2 * part + p->units * kUnit <= kSmemBudget ? 2 : 1;
    uint32_t ring = (kSmemBudget - fixed - p->r_ring * part) / kUnit;
    if (ring > 2u * p->units) ring = 2u * p->units;
    if (ring > (uint32_t)kMaxUnits) ring = kMaxUnits;
    p->ring = (int)ring;
    p->off_r = ring * kUnit;
    p->off_p = p->off_r + p->r_ring * part;
    p->off_q = p->off_p + kPBytes;
    p->off_x = p->off_q + (uint32_t)(p->c_blocks + p->r_blocks) * N * 128;
    p->tmem_cols = 32;
    while (p->tmem_cols < (uint32_t)(N * (2 + p->units))) p->tmem_cols *= 2;
    return p->tmem_cols <= 512;
}

template <int N>
int launch_n(const LatentAttnArgs& a, const LatTcParams& p, cudaStream_t stream) {
    CUtensorMap tmC, tmQ;
    int rc;
    const int D = a.R + a.dr, rows = a.n * a.H;
    // a single token may be replayed at other positions: the whole cache; else what the portion sees
    const uint64_t keys = a.host_pos >= 0 ? (uint64_t)a.host_pos + a.n : (uint64_t)a.cap;
    if ((rc = make_tmap_bf16_heads(&tmC, a.c, a.R, 1, keys, a.B, a.R, a.c_batch, kT))) return rc;
    if ((rc = make_tmap_bf16_heads(&tmQ, a.q, a.R, 1, rows, a.B, D, (uint64_t)rows * D, N))) return rc;
    CUtensorMap tmR = tmC, tmQr = tmQ;
    if (a.dr) {
        if ((rc = make_tmap_bf16_heads(&tmR, a.kr, a.dr, 1, keys, a.B, a.dr, a.r_batch, kT))) return rc;
        if ((rc = make_tmap_bf16_heads(&tmQr, (const __nv_bfloat16*)a.q + a.R, a.dr, 1, rows, a.B, D, (uint64_t)rows * D, N))) return rc;
    }
    auto kern = latent_tc_kernel<N>;
    static bool once[64] = {};
    int dev = 0;
    PLZ_CUDA_CHECK(cudaGetDevice(&dev));
    if (!once[dev & 63]) { PLZ_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024)); once[dev & 63] = true; }
    const int gy = (rows + N - 1) / N;
    if (gy > 65535) { set_last_error("latent attention: %d query rows", rows); return PLZ_ERR_TOO_LARGE; }
    PLZ_LAUNCH_CHAIN(kern, dim3(p.l.splits, gy, a.B), dim3(kLatThreads), (size_t)(p.off_x + kExtra + 1024), stream, tmC, tmR, tmQ, tmQr, p);
    return PLZ_OK;
}

}  // namespace

bool latent_tc_fits(int R, int dr) {
    LatTcParams p = {};
    return R % 8 == 0 && dr % 8 == 0 && R <= 512 && plan(R, dr, 16, &p);
}

// the fewest CTAs that hold all rows, then the narrowest that is enough for that many
int latent_tc_rows(int rows, int R, int dr) {
    LatTcParams p = {};
    int widest = 16;
    for (int n = 32; n <= 64; n += 16)
        if (plan(R, dr, n, &p)) widest = n;
    const int ctas = (rows + widest - 1) / widest, each = (rows + ctas - 1) / ctas;
    return (each + 15) / 16 * 16;
}

int launch_latent_tc(const LatentAttnArgs& a, const LatentParams& l, cudaStream_t stream) {
    LatTcParams p = {};
    const int N = latent_tc_rows(a.n * a.H, a.R, a.dr);
    if (!plan(a.R, a.dr, N, &p)) { set_last_error("latent attention: no plan for R=%d dr=%d", a.R, a.dr); return PLZ_ERR_UNSUPPORTED; }
    p.l = l; p.pos = a.pos; p.status = device_status_ptr();
    if (N == 16) return launch_n<16>(a, p, stream);
    if (N == 32) return launch_n<32>(a, p, stream);
    if (N == 48) return launch_n<48>(a, p, stream);
    return launch_n<64>(a, p, stream);
}

}  // namespace plz
