// Attention over cached latents on the tensor cores (tcgen05.mma, accumulators in TMEM): a few query rows (token, head) against many cached
// tokens, bf16, latents up to 512 columns. It serves single tokens and short portions, where the cache is read once and every row of it
// meets all heads.
//
// Everything is transposed, so that the long dimensions are the 128-row side of the products and the query rows (16 .. 64) the narrow one:
//   S^T [key = TMEM lane][query row]      = [C | KR] Q^T      the cached tile as it lies (K-major), queries K-major
//   O^T [latent column = lane][query row] += C^T P^T          the SAME shared-memory tile read MN-major, P^T written by the softmax threads
// A cached byte enters shared memory once and serves as key and as value.
//
// One CTA takes N query rows of a sequence and one split of its keys, 128 keys at a time. Warps 0-7 are the softmax threads (thread = key and
// half of the query rows), warp 8 issues the MMAs, warp 9 the copies. A tile arrives as units of 128 latent columns (32 KB) in a ring plus the shared key part; a unit
// is handed back as soon as the value product of its columns has run, so that the next tile streams in under the rest of the current one.
// The maximum of a query row runs over the lanes: recursive halving inside a warp, its four warps meet in shared memory. The reference
// of the exponentials moves only when the maximum has grown by more than 8 (in log2 units), so O^T is rarely rescaled. Rows of the last
// tile beyond the sequence are cleared in shared memory (a weight of zero times whatever lies there would not be safe).
// Partial sums of the key splits go to the workspace that latent_combine_kernel merges.
#include "attention_tiles.cuh"
#include "latent_attention.cuh"

namespace plz {
namespace {

constexpr int kLatThreads = 320;
constexpr uint32_t kUnit = 2 * kBlk;            // 128 keys x 128 latent columns
// P^T: 128 keys, rows of 64 bytes (64-byte swizzle) for up to 32 query rows, else of 128
__host__ __device__ constexpr uint32_t p_row(int N) { return N <= 32 ? 64u : 128u; }
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

__device__ __forceinline__ float join(float a, float b, bool max) { return max ? fmaxf(a, b) : a + b; }
template <int W, bool MAX>
__device__ __forceinline__ float over_lanes(float (&v)[W], int lane) {     // lane (mod W) gets the result of column lane (mod W)
#pragma unroll
    for (int half = W / 2; half >= 1; half >>= 1) {
        const bool up = (lane & half) != 0;
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float send = up ? v[i] : v[i + half], keep = up ? v[i + half] : v[i];
            v[i] = join(keep, __shfl_xor_sync(0xFFFFFFFFu, send, half), MAX);
        }
    }
    float r = v[0];
#pragma unroll
    for (int o = W; o < 32; o <<= 1) r = join(r, __shfl_xor_sync(0xFFFFFFFFu, r, o), MAX);
    return r;
}
// result of every one of NC columns (8, 16, 24, 32) over the 32 lanes: lane i gets column i, for 24 columns lanes 16 .. 31 get 16 + i % 8
template <int NC, bool MAX>
__device__ __forceinline__ float columns_over_lanes(const float (&s)[NC], int lane) {
    constexpr int W = NC == 24 ? 16 : NC;
    float t[W];
#pragma unroll
    for (int i = 0; i < W; ++i) t[i] = s[i];
    float r = over_lanes<W, MAX>(t, lane);
    if (NC == 24) {
        float u[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) u[i] = s[NC - 8 + i];
        const float q = over_lanes<8, MAX>(u, lane);
        if (lane >= 16) r = q;
    }
    return r;
}
// the column of a half that a lane holds after that
template <int NC>
__device__ __forceinline__ int column_of(int lane) { return NC == 24 ? (lane < 16 ? lane : 16 + (lane & 7)) : (lane & (NC - 1)); }

__device__ __forceinline__ void tmem_st_32x8(uint32_t taddr, const uint32_t (&r)[8]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]) : "memory");
}
template <int NC>
__device__ __forceinline__ void load_cols(uint32_t t, float (&s)[NC]) {
    if (NC == 32) {
        uint32_t v[32];
        tmem_ld_32x32(t, v);
#pragma unroll
        for (int i = 0; i < 32; ++i) s[i % NC] = __uint_as_float(v[i]);
    }
    if (NC & 16) {
        uint32_t v[16];
        tmem_ld_32x16(t, v);
#pragma unroll
        for (int i = 0; i < 16; ++i) s[i % NC] = __uint_as_float(v[i]);
    }
    if (NC & 8) {
        uint32_t v[8];
        tmem_ld_32x8(t + (NC - 8), v);
#pragma unroll
        for (int i = 0; i < 8; ++i) s[NC - 8 + i] = __uint_as_float(v[i]);
    }
}
template <int NC>
__device__ __forceinline__ void store_cols(uint32_t t, const float (&s)[NC]) {
    if (NC == 32) {
        uint32_t v[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(s[i % NC]);
        tmem_st_32x32(t, v);
    }
    if (NC & 16) {
        uint32_t v[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(s[i % NC]);
        tmem_st_32x16(t, v);
    }
    if (NC & 8) {
        uint32_t v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = __float_as_uint(s[NC - 8 + i]);
        tmem_st_32x8(t + (NC - 8), v);
    }
    tmem_wait_st();
}

template <int N>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmR, const __grid_constant__ CUtensorMap tmQ,
                 const __grid_constant__ CUtensorMap tmQr, const LatTcParams p) {
    constexpr int NC = N / 2;                   // query rows of a softmax thread
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
    const uint32_t q_full = bar + 176, p_full = bar + 184, o_done = bar + 192;
    auto mx_full = [&](int half) { return bar + 200u + 8u * half; };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + p.off_x + 216);
    volatile uint32_t* abort_flag = tmem_slot + 1;
    float* wmax = reinterpret_cast<float*>(smem + p.off_x + 256);         // [2][8 warps][32]
    float* own = wmax + 2 * 8 * 32;                                       // per warp: [32] reference, [32] correction

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = blockIdx.x, r0 = (int)blockIdx.y * N, b = blockIdx.z;
    const int rows = p.l.n * p.l.H, H = p.l.H, R = p.l.R;
    if (threadIdx.x == 0) {
        for (int s = 0; s < kMaxUnits; ++s) { mbar_init(u_full(s), 1); mbar_init(u_empty(s), 1); }
        for (int s = 0; s < 2; ++s) { mbar_init(r_full(s), 1); mbar_init(r_empty(s), 1); mbar_init(s_full(s), 1); }
        mbar_init(q_full, 1); mbar_init(p_full, 8); mbar_init(o_done, 1); mbar_init(mx_full(0), 4); mbar_init(mx_full(1), 4);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 8) { tmem_alloc(smem_u32((const void*)tmem_slot), p.tmem_cols); tmem_relinquish(); }
    if (warp == 9 && lane == 0) { tma_prefetch_desc(&tmC); tma_prefetch_desc(&tmQ); if (p.r_blocks) { tma_prefetch_desc(&tmR); tma_prefetch_desc(&tmQr); } }
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

    if (warp == 9) {
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
    } else if (warp == 8) {
        if (lane == 0 && tiles > 0) {
            const uint32_t id_s = make_idesc(128, N, 0, 0), id_o = make_idesc(128, N, 1, 1);
            // descriptors as words: only the low one (start address) moves
            const uint64_t dq = make_sdesc(base + p.off_q, 16u, 1024u), dk = make_sdesc(base, 16u, 1024u), dv = make_sdesc(base, kBlk, 1024u);
            const uint64_t dp = make_sdesc(base + p.off_p, kBlk, 8u * p_row(N)) ^ (N <= 32 ? (uint64_t)6 << 61 : 0ull);   // layout 2 -> 4: 64-byte swizzle
            const uint32_t q_lo = (uint32_t)dq, q_hi = (uint32_t)(dq >> 32), k_lo = (uint32_t)dk, k_hi = (uint32_t)(dk >> 32);
            const uint32_t v_lo = (uint32_t)dv, v_hi = (uint32_t)(dv >> 32), p_lo = (uint32_t)dp, p_hi = (uint32_t)(dp >> 32);
            const bool ahead = p.ring >= 2 * p.units && (p.r_blocks == 0 || p.r_ring == 2);
            bool ok = mbar_wait(q_full, 0, abort_flag, p.status, ST_TIMEOUT_FULL, 82);
            // one 64-column block of S^T
            auto block = [&](uint32_t ts, uint32_t a, uint32_t bq, int cols, uint32_t acc) {
                if (cols > 48) {
#pragma unroll
                    for (int ks = 0; ks < 4; ++ks) umma_bf16_words<1>(ts, a + ks * 2u, k_hi, bq + ks * 2u, q_hi, id_s, ks > 0 ? 1u : acc);
                } else {
                    for (int ks = 0; ks * 16 < cols; ++ks) umma_bf16_words<1>(ts, a + ks * 2u, k_hi, bq + ks * 2u, q_hi, id_s, ks > 0 ? 1u : acc);
                }
            };
            int s_unit = 0, s_ph = 0, v_unit = 0;          // ring positions of the scores (with its phase) and of the value products
            auto scores = [&](int j) {
                const uint32_t ts = tS(j & 1);
                if (p.r_blocks) {
                    const int s = p.r_ring == 2 ? (j & 1) : 0;
                    if (!mbar_wait_lean(r_full(s), (p.r_ring == 2 ? j >> 1 : j) & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 83)) return false;
                    tc_fence_after_sync();
                    for (int i = 0; i < p.r_blocks; ++i)
                        block(ts, k_lo + (p.off_r >> 4) + (uint32_t)(s * p.r_blocks + i) * (kBlk >> 4), q_lo + (uint32_t)((p.c_blocks + i) * N * 8), p.l.dr - 64 * i, i > 0 ? 1u : 0u);
                    umma_commit(r_empty(s));
                }
                uint32_t bq = q_lo;
                int left = R;
                for (int m = 0; m < p.units; ++m) {
                    if (!mbar_wait_lean(u_full(s_unit), s_ph, abort_flag, p.status, ST_TIMEOUT_FULL, 84)) return false;
                    tc_fence_after_sync();
                    const uint32_t a = k_lo + (uint32_t)s_unit * (kUnit >> 4);
                    block(ts, a, bq, left, (m > 0 || p.r_blocks) ? 1u : 0u);
                    if (left > 64) block(ts, a + (kBlk >> 4), bq + (uint32_t)(N * 8), left - 64, 1u);
                    bq += 2u * N * 8;
                    left -= 128;
                    if (++s_unit == p.ring) { s_unit = 0; s_ph ^= 1; }
                }
                umma_commit(s_full(j & 1));
                return true;
            };
            if (ok) ok = scores(0);
            for (int j = 0; j < tiles && ok; ++j) {
                if (ahead && j + 1 < tiles) { ok = scores(j + 1); if (!ok) break; }
                ok = mbar_wait_lean(p_full, j & 1, abort_flag, p.status, ST_TIMEOUT_FULL, 85);
                if (!ok) break;
                tc_fence_after_sync();
                const uint32_t acc = j > 0 ? 1u : 0u;
                for (int m = 0; m < p.units; ++m) {
                    const uint32_t a = v_lo + (uint32_t)v_unit * (kUnit >> 4), to = tO(m);
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks) umma_bf16_words<1>(to, a + ks * 128u, v_hi, p_lo + ks * p_row(N), p_hi, id_o, ks > 0 ? 1u : acc);
                    umma_commit(u_empty(v_unit));
                    if (++v_unit == p.ring) v_unit = 0;
                }
                umma_commit(o_done);
                if (!ahead && j + 1 < tiles) ok = scores(j + 1);
            }
        }
    } else {
        const int quarter = warp & 3, half = warp >> 2, t = quarter * 32 + lane;     // t: key of the tile = TMEM lane
        const int c0 = half * NC, mine = column_of<NC>(lane);                        // first query row of this thread; the one it owns after a reduction
        const uint32_t lane_off = ((uint32_t)(quarter * 32) << 16) + (uint32_t)c0;
        const float c = p.l.scale * kLatLog2e;
        const int lim0 = pos + r0 / H;                                    // last key that every row of this CTA sees
        float* my_m = own + warp * 64;
        float* my_a = my_m + 32;
        float l[NC], m_run = kLatNegBig;
#pragma unroll
        for (int i = 0; i < NC; ++i) l[i] = 0.f;
        // a warp goes on or gives up as one
        auto wait = [&](uint32_t mbar, uint32_t parity, uint32_t role) {
            return __all_sync(0xFFFFFFFFu, mbar_wait(mbar, parity, abort_flag, p.status, ST_TIMEOUT_ACCUM, role)) != 0;
        };
        // the four warps of a half exchange a value per query row; a buffer is written again two exchanges later
        auto publish = [&](int j, float v) {
            wmax[(j & 1) * 256 + warp * 32 + lane] = v;
            __syncwarp();
            if (lane == 0) mbar_arrive(mx_full(half));
        };
        auto shared_by = [&](int j, int w) { return wmax[(j & 1) * 256 + (half * 4 + w) * 32 + lane]; };
        bool ok = true;
        for (int j = 0; j < tiles && ok; ++j) {
            const int tok = k0 + j * kT + t;
            ok = wait(s_full(j & 1), (j >> 1) & 1, 86);
            if (!ok) break;
            tc_fence_after_sync();
            float s[NC];
            load_cols<NC>(tS(j & 1) + lane_off, s);
            if (k0 + j * kT + kT - 1 > min(lim0, k1 - 1)) {               // some key of the tile is hidden from some row
#pragma unroll
                for (int i = 0; i < NC; ++i)
                    if (tok >= k1 || tok > pos + (r0 + c0 + i) / H) s[i] = -INFINITY;
            }
            publish(j, columns_over_lanes<NC, true>(s, lane) * c);
            ok = wait(mx_full(half), j & 1, 87);
            if (!ok) break;
            const float m = fmaxf(fmaxf(shared_by(j, 0), shared_by(j, 1)), fmaxf(shared_by(j, 2), shared_by(j, 3)));
            const bool up = m > m_run + kLazy;
            my_a[mine] = up ? exp2f(m_run - m) : 1.0f;
            if (up) m_run = m;
            my_m[mine] = m_run;
            const bool moved = __any_sync(0xFFFFFFFFu, up);               // the same in all four warps
            __syncwarp();
#pragma unroll
            for (int i = 0; i < NC; i += 4) {
                const float4 r = *reinterpret_cast<const float4*>(my_m + i);
                s[i] = exp2f(fmaf(s[i], c, -r.x)); s[i + 1] = exp2f(fmaf(s[i + 1], c, -r.y));
                s[i + 2] = exp2f(fmaf(s[i + 2], c, -r.z)); s[i + 3] = exp2f(fmaf(s[i + 3], c, -r.w));
            }
            if (j > 0) {                                                  // P^T and O^T are free once the products of the tile before have run
                ok = wait(o_done, (j - 1) & 1, 88);
                if (!ok) break;
                tc_fence_after_sync();
                if (moved) {
#pragma unroll 1
                    for (int u = 0; u < p.units; ++u) {
                        float o[NC];
                        load_cols<NC>(tO(u) + lane_off, o);
#pragma unroll
                        for (int i = 0; i < NC; ++i) o[i] *= my_a[i];
                        store_cols<NC>(tO(u) + lane_off, o);
                    }
                }
            }
#pragma unroll
            for (int q = 0; q < NC / 8; ++q)
                *reinterpret_cast<uint4*>(smem + p.off_p + (N <= 32 ? t * 64u + ((((c0 >> 3) + q) ^ ((t >> 1) & 3)) << 4) : swz128(t, (c0 >> 3) + q))) =
                    make_uint4(pack_bf16x2(s[q * 8], s[q * 8 + 1]), pack_bf16x2(s[q * 8 + 2], s[q * 8 + 3]), pack_bf16x2(s[q * 8 + 4], s[q * 8 + 5]),
                               pack_bf16x2(s[q * 8 + 6], s[q * 8 + 7]));
            if (tok >= total && half == 0) {                              // past the sequence: whatever the cache holds there must not count
                for (int u = 0; u < p.units; ++u) {
                    uint8_t* z = smem + ((j * p.units + u) % p.ring) * kUnit + t * 128;
#pragma unroll
                    for (int i = 0; i < 16; ++i) *reinterpret_cast<uint4*>(z + (i >> 3) * kBlk + (i & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
                }
            }
            tc_fence_before_sync();
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
            if (moved) {
#pragma unroll
                for (int i = 0; i < NC; ++i) l[i] *= my_a[i];
            }
#pragma unroll
            for (int i = 0; i < NC; ++i) l[i] += s[i];
            __syncwarp();                                                 // my_m, my_a are written again in the next tile
        }
        if (ok) {
            publish(tiles, columns_over_lanes<NC, false>(l, lane));
            const long long row0 = (long long)b * rows + r0 + c0;
            const int S = p.l.splits;
            ok = wait(mx_full(half), tiles & 1, 90);
            if (ok && quarter == 0 && lane < NC && r0 + c0 + mine < rows) {
                float* ml = p.l.ws_ml + ((row0 + mine) * S + split) * 2;
                ml[0] = m_run;
                ml[1] = shared_by(tiles, 0) + shared_by(tiles, 1) + shared_by(tiles, 2) + shared_by(tiles, 3);
            }
            if (ok && tiles > 0) ok = wait(o_done, (tiles - 1) & 1, 89);
            if (ok && tiles > 0) {
                tc_fence_after_sync();
                const int valid = min(NC, rows - r0 - c0);
                const long long step = (long long)S * R;
#pragma unroll 1
                for (int u = 0; u < p.units; ++u) {
                    float o[NC];
                    load_cols<NC>(tO(u) + lane_off, o);
                    const int d = u * 128 + t;
                    if (d < R) {
                        float* dst = p.l.ws_o + (row0 * S + split) * R + d;
#pragma unroll
                        for (int i = 0; i < NC; ++i) {
                            if (i < valid) *dst = o[i];
                            dst += step;
                        }
                    }
                }
            }
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 8) { tc_fence_after_sync(); tmem_dealloc(tmem, p.tmem_cols); }
}

// shared-memory plan of a CTA with N query rows; false if it does not fit
bool plan(int R, int dr, int N, LatTcParams* p) {
    p->c_blocks = (R + 63) / 64; p->r_blocks = (dr + 63) / 64; p->units = (R + 127) / 128;
    const uint32_t p_bytes = 128 * p_row(N), fixed = p_bytes + (uint32_t)(p->c_blocks + p->r_blocks) * N * 128;
    const uint32_t part = (uint32_t)p->r_blocks * kBlk;
    if (fixed + part + p->units * kUnit > kSmemBudget) return false;
    // two whole tiles if they fit (then the scores run a tile ahead), else as many units as fit beside one key part
    p->r_ring = fixed + 2 * part + 2 * p->units * kUnit <= kSmemBudget && 2 * p->units <= kMaxUnits ? 2 : 1;
    uint32_t ring = (kSmemBudget - fixed - p->r_ring * part) / kUnit;
    if (ring > 2u * p->units) ring = 2u * p->units;
    if (ring > (uint32_t)kMaxUnits) ring = kMaxUnits;
    p->ring = (int)ring;
    p->off_r = ring * kUnit;
    p->off_p = p->off_r + p->r_ring * part;
    p->off_q = p->off_p + p_bytes;
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
