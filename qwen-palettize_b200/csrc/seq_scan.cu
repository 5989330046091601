// The sequential half of the chunked recurrences on the 5th-generation tensor cores: one CTA per (128 value columns, head, sequence)
// walks the chunks in order with the state resident in TMEM.
//
// Everything is transposed: the state is S^T [value column = TMEM lane][key column], so the state and U are A operands of M = 128
// products straight from tensor memory and only chunk constants come through shared memory. Per chunk
//
//   1. the eight epilogue warps (thread = value column and half of the columns) read S^T, write it back times e^{b_C}, and write its bf16 halves hi + lo as an
//      A operand into TMEM
//   2. MMA:  [U' | O] = S^T (-W | Q~)^T                        three products hi hi + hi lo + lo hi
//   3. epilogue warps: U = U' + U0 (global memory), halves hi + lo over U' in place
//   4. MMA:  O += U M^T ;  S^T += U K~
//   5. O is stored while step 2 of the next chunk runs (two O / U regions alternate)
//
// One warp issues the MMAs, one the bulk copies (two stages of each operand set). Waits are bounded as everywhere in this library.
// TMEM: S^T 64 KB columns' worth (KB * 64), two U | O regions of 128, S hi and lo KB * 32 each: 512 columns for 128 key columns.
#include "attention_tiles.cuh"
#include "seq_chunk.cuh"

namespace plz {
namespace {

constexpr int kScanThreads = 320;   // warps 0-7 epilogue (two per 32 value columns, half of the TMEM columns each), 8 MMA, 9 copies

__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

template <int KB, bool HASW>
struct ScanCfg {
    using W = ChunkWs<KB, HASW ? 128 : 64>;
    static constexpr uint32_t OFF_B = 2 * W::A_BYTES, OFF_DEC = OFF_B + 2 * W::B_BYTES, OFF_BAR = OFF_DEC + 2 * 512, SMEM = OFF_BAR + 1024 + 256;
    // TMEM columns
    static constexpr uint32_t T_UO = 0, T_S = 256, T_SH = T_S + 64 * KB, T_SL = T_SH + 32 * KB;
};

template <int KB, bool HASW>
__global__ void __launch_bounds__(kScanThreads, 1)
scan_kernel(const ScanArgs p, StatusWord* status) {
    using C = ScanCfg<KB, HASW>;
    using W = typename C::W;
    constexpr int DK = 64 * KB;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t* smem = smem_raw + (base - raw);
    const uint32_t bar = base + C::OFF_BAR;
    auto a_full = [&](int s) { return bar + 8u * s; };            // operand set A of stage s has landed
    auto b_full = [&](int s) { return bar + 16u + 8u * s; };
    auto a_free = [&](int s) { return bar + 32u + 8u * s; };      // the products that read it have completed
    auto b_free = [&](int s) { return bar + 48u + 8u * s; };
    const uint32_t s_ready = bar + 64, uo_full = bar + 72, u_ready = bar + 80, fin_full = bar + 88;
    auto u_read = [&](int q) { return bar + 96u + 8u * q; };      // both warps of a lane quarter have read U'
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + C::OFF_BAR + 128);
    volatile uint32_t* abort_flag = tmem_slot + 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y, b = blockIdx.z;
    const uint8_t* ws0 = p.ws + ((long long)b * p.H + h) * p.chunks * p.ws_stride;

    if (threadIdx.x == 0) {
        for (int s = 0; s < 2; ++s) { mbar_init(a_full(s), 1); mbar_init(b_full(s), 1); mbar_init(a_free(s), 1); mbar_init(b_free(s), 1); }
        for (int q = 0; q < 4; ++q) mbar_init(u_read(q), 2);
        mbar_init(s_ready, 8); mbar_init(uo_full, 1); mbar_init(u_ready, 8); mbar_init(fin_full, 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 8) { tmem_alloc(smem_u32((const void*)tmem_slot), 512); tmem_relinquish(); }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = *tmem_slot;

    if (warp == 9) {
        if (lane == 0) {
            bool ok = true;
            int in_a = 0, in_b = 0;                       // chunks whose copies have been issued
            for (int ch = 0; ch < p.chunks; ++ch) {
                const int s = ch & 1;
                const uint8_t* src = ws0 + (long long)ch * p.ws_stride;
                if (ch >= 2) ok = mbar_wait(a_free(s), ((ch >> 1) - 1) & 1, abort_flag, status, ST_TIMEOUT_EMPTY, 70);
                if (!ok) break;
                mbar_arrive_expect_tx(a_full(s), W::A_BYTES + W::DEC_BYTES);
                bulk_load(base + s * W::A_BYTES, src, W::A_BYTES, a_full(s));
                bulk_load(base + C::OFF_DEC + s * 512, src + W::OFF_DEC, W::DEC_BYTES, a_full(s));
                in_a = ch + 1;
                if (ch >= 2) ok = mbar_wait(b_free(s), ((ch >> 1) - 1) & 1, abort_flag, status, ST_TIMEOUT_EMPTY, 71);
                if (!ok) break;
                mbar_arrive_expect_tx(b_full(s), W::B_BYTES);
                bulk_load(base + C::OFF_B + s * W::B_BYTES, src + W::OFF_B, W::B_BYTES, b_full(s));
                in_b = ch + 1;
            }
            // every copy has landed before the CTA exits (bounded: another role may have given up)
            const uint64_t t0 = globaltimer_ns();
            for (int ch = in_a > 2 ? in_a - 2 : 0; ch < in_a; ++ch)
                while (!mbar_try_wait(a_full(ch & 1), (ch >> 1) & 1) && globaltimer_ns() - t0 < 100000000ull) {}
            for (int ch = in_b > 2 ? in_b - 2 : 0; ch < in_b; ++ch)
                while (!mbar_try_wait(b_full(ch & 1), (ch >> 1) & 1) && globaltimer_ns() - t0 < 100000000ull) {}
        }
    } else if (warp == 8) {
        if (lane == 0) {
            bool ok = true;
            constexpr uint32_t n1 = HASW ? 128 : 64;
            const uint32_t id1 = make_idesc(128, n1, 0, 0), idM = make_idesc(128, 64, 0, 0), idK = make_idesc(128, DK, 0, 1);
            for (int ch = 0; ch < p.chunks && ok; ++ch) {
                const int s = ch & 1;
                const uint32_t ph = (ch >> 1) & 1, uo = tmem + C::T_UO + 128u * s;
                ok = mbar_wait(a_full(s), ph, abort_flag, status, ST_TIMEOUT_FULL, 72) && mbar_wait(s_ready, ch & 1, abort_flag, status, ST_TIMEOUT_FULL, 73);
                if (!ok) break;
                tc_fence_after_sync();
                const uint64_t dA = make_sdesc(base + s * W::A_BYTES, 16u, 1024u);
                const uint32_t hi = (uint32_t)(dA >> 32);
#pragma unroll
                for (int pr = 0; pr < 3; ++pr) {       // hi hi, hi lo, lo hi
                    const uint32_t at = tmem + (pr == 2 ? C::T_SL : C::T_SH), bt = (uint32_t)dA + (pr == 1 ? (W::A_PLANE >> 4) : 0u);
#pragma unroll
                    for (int ks = 0; ks < DK / 16; ++ks)
                        umma_ts(uo + (HASW ? 0u : 64u), at + ks * 8u, bt + (uint32_t)((ks >> 2) * (W::A_BLOCK >> 4) + (ks & 3) * 2), hi, id1, (pr || ks) ? 1u : 0u);
                }
                umma_commit(uo_full);
                umma_commit(a_free(s));
                ok = mbar_wait(b_full(s), ph, abort_flag, status, ST_TIMEOUT_FULL, 74) && mbar_wait(u_ready, ch & 1, abort_flag, status, ST_TIMEOUT_FULL, 75);
                if (!ok) break;
                tc_fence_after_sync();
                const uint32_t sB = base + C::OFF_B + s * W::B_BYTES;
                const uint64_t dM = make_sdesc(sB, 16u, 1024u), dK = make_sdesc(sB + 2 * W::M_PLANE, kC * 128u, 1024u);
#pragma unroll
                for (int pr = 0; pr < 3; ++pr) {
                    const uint32_t at = uo + (pr == 2 ? 32u : 0u);
#pragma unroll
                    for (int ks = 0; ks < kC / 16; ++ks) {
                        umma_ts(tmem + C::T_S, at + ks * 8u, (uint32_t)dK + (pr == 1 ? (W::K_PLANE >> 4) : 0u) + (uint32_t)(ks * 128), (uint32_t)(dK >> 32), idK, 1u);
                        umma_ts(uo + 64u, at + ks * 8u, (uint32_t)dM + (pr == 1 ? (W::M_PLANE >> 4) : 0u) + (uint32_t)(ks * 2), (uint32_t)(dM >> 32), idM, 1u);
                    }
                }
                umma_commit(fin_full);
                umma_commit(b_free(s));
            }
        }
    } else {
        const int quarter = warp & 3, half = warp >> 2;
        const int d = (int)blockIdx.x * 128 + quarter * 32 + lane;   // value column
        const uint32_t lo = (uint32_t)(quarter * 32) << 16;
        const bool live = d < p.dv, in_u = d < p.dvp;
        float* Sg = p.state + ((long long)b * p.H + h) * p.dk * (long long)p.dv + d;
        bool ok = true;
        auto store_o = [&](int ch) {
            const int t0 = p.t_begin + ch * kC, L = min(kC, p.n - t0);
            float* og = p.o + (((long long)b * p.n + t0) * p.H + h) * p.dv + d;
            const long long pitch = (long long)p.H * p.dv;
            uint32_t v[32];
            tmem_ld_32x32(tmem + lo + C::T_UO + 128u * (ch & 1) + 64u + half * 32u, v);
            if (!live) return;
            float* at = og + (long long)half * 32 * pitch;
            if (L == kC) {
#pragma unroll
                for (int i = 0; i < 32; ++i, at += pitch) __stcs(at, __uint_as_float(v[i]));
            } else {
#pragma unroll
                for (int i = 0; i < 32; ++i, at += pitch)
                    if (half * 32 + i < L) *at = __uint_as_float(v[i]);
            }
        };
        for (int ch = 0; ch < p.chunks && ok; ++ch) {
            const int s = ch & 1;
            ok = mbar_wait(a_full(s), (ch >> 1) & 1, abort_flag, status, ST_TIMEOUT_ACCUM, 76);      // e^{b_C}
            if (ok && ch > 0) ok = mbar_wait(fin_full, (ch - 1) & 1, abort_flag, status, ST_TIMEOUT_ACCUM, 77);
            if (!ok) break;
            tc_fence_after_sync();
            const float* dec = reinterpret_cast<const float*>(smem + C::OFF_DEC + s * 512);
#pragma unroll 1
            for (int cb = half * KB; cb < (half + 1) * KB; ++cb) {
                uint32_t v[32];
                if (ch == 0) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        const int c = cb * 32 + i;
                        v[i] = (live && c < p.dk) ? __float_as_uint(Sg[(long long)c * p.dv]) : 0u;
                    }
                } else {
                    tmem_ld_32x32(tmem + lo + C::T_S + cb * 32u, v);
                }
                uint32_t hh[16], ll[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) split2(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]), hh[i], ll[i]);
                tmem_st_32x16(tmem + lo + C::T_SH + cb * 16u, hh);
                tmem_st_32x16(tmem + lo + C::T_SL + cb * 16u, ll);
#pragma unroll
                for (int i = 0; i < 32; i += 4) {
                    const float4 e = *reinterpret_cast<const float4*>(dec + cb * 32 + i);
                    v[i] = __float_as_uint(__uint_as_float(v[i]) * e.x); v[i + 1] = __float_as_uint(__uint_as_float(v[i + 1]) * e.y);
                    v[i + 2] = __float_as_uint(__uint_as_float(v[i + 2]) * e.z); v[i + 3] = __float_as_uint(__uint_as_float(v[i + 3]) * e.w);
                }
                tmem_st_32x32(tmem + lo + C::T_S + cb * 32u, v);      // waits for the stores
            }
            tc_fence_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(s_ready);
            // while the first products run: U0 of this chunk, the finished output of the previous one
            float u[32];
            {
                const float* U0 = reinterpret_cast<const float*>(ws0 + (long long)ch * p.ws_stride + W::OFF_U) + (long long)half * 32 * p.dvp + (in_u ? d : 0);
#pragma unroll
                for (int t = 0; t < 32; ++t) u[t] = __ldcs(U0 + (long long)t * p.dvp);
            }
            if (ch > 0) store_o(ch - 1);
            if (HASW) {
                ok = mbar_wait(uo_full, ch & 1, abort_flag, status, ST_TIMEOUT_ACCUM, 78);
                if (!ok) break;
                tc_fence_after_sync();
                uint32_t v[32];
                tmem_ld_32x32(tmem + lo + C::T_UO + 128u * s + half * 32u, v);
#pragma unroll
                for (int i = 0; i < 32; ++i) u[i] += __uint_as_float(v[i]);
                // the other half's warp of these lanes has read its columns too before they are overwritten
                tc_fence_before_sync();
                __syncwarp();
                if (lane == 0) mbar_arrive(u_read(quarter));
                ok = mbar_wait(u_read(quarter), ch & 1, abort_flag, status, ST_TIMEOUT_ACCUM, 80);
                if (!ok) break;
                tc_fence_after_sync();
            }
            // hi into columns 0..31, lo into 32..63 of the same region
            uint32_t hh[16], ll[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) split2(u[2 * i], u[2 * i + 1], hh[i], ll[i]);
            tmem_st_32x16(tmem + lo + C::T_UO + 128u * s + half * 16u, hh);
            tmem_st_32x16(tmem + lo + C::T_UO + 128u * s + 32u + half * 16u, ll);
            tmem_wait_st();
            tc_fence_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(u_ready);
        }
        if (ok) ok = mbar_wait(fin_full, (p.chunks - 1) & 1, abort_flag, status, ST_TIMEOUT_ACCUM, 79);
        if (ok) {
            tc_fence_after_sync();
            store_o(p.chunks - 1);
#pragma unroll 1
            for (int cb = half * KB; cb < (half + 1) * KB; ++cb) {
                uint32_t v[32];
                tmem_ld_32x32(tmem + lo + C::T_S + cb * 32u, v);
#pragma unroll
                for (int i = 0; i < 32; ++i)
                    if (live && cb * 32 + i < p.dk) Sg[(long long)(cb * 32 + i) * p.dv] = __uint_as_float(v[i]);
            }
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 8) { tc_fence_after_sync(); tmem_dealloc(tmem, 512); }
}

template <int KB, bool HASW>
int launch_t(const ScanArgs& a, cudaStream_t stream) {
    using C = ScanCfg<KB, HASW>;
    static bool once[64] = {};
    int dev = 0;
    PLZ_CUDA_CHECK(cudaGetDevice(&dev));
    if (!once[dev & 63]) { PLZ_CUDA_CHECK(cudaFuncSetAttribute((scan_kernel<KB, HASW>), cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM)); once[dev & 63] = true; }
    scan_kernel<KB, HASW><<<dim3((a.dv + 127) / 128, a.H, a.B), kScanThreads, C::SMEM, stream>>>(a, device_status_ptr());
    PLZ_LAUNCH_CHECK();
    return PLZ_OK;
}

}  // namespace

int launch_chunk_scan(const ScanArgs& a, bool has_w, int kb, cudaStream_t stream) {
    if (has_w) return kb == 1 ? launch_t<1, true>(a, stream) : launch_t<2, true>(a, stream);
    return kb == 1 ? launch_t<1, false>(a, stream) : launch_t<2, false>(a, stream);
}

}  // namespace plz
