// Chunked form of the two linear recurrences (prompts of bf16 models), 64 tokens per chunk. With b_i the cumulative log decay inside a
// chunk (per key channel; inclusive), S0 the state at its start, and all of it exact algebra on the token-by-token rule:
//
//   u_i = beta_i (v_i - S0^T (k_i e^{b_i}) - sum_{j<i} A'_ij u_j),      A'_ij = sum_c k_i k_j e^{b_i - b_j}
//   =>  U = T beta V - (T beta Kbar) S0 = U0 - W S0,                    T = (I + tril(beta A', -1))^{-1},  Kbar_i = k_i e^{b_i}
//   o_i = S0^T (q_i e^{b_i}) + sum_{j<=i} M_ij u_j,                     M_ij = sum_c q_i k_j e^{b_i - b_j}
//   S1  = diag(e^{b_C}) S0 + sum_j (k_j e^{b_C - b_j}) u_j^T
//
// (decayed linear attention: u = v, no W, scalar decay). Two launches per segment of chunks:
//   delta_chunk_kernel / decay_chunk_kernel   one CTA per (chunk, head, sequence), all in parallel: -W, U0, Q~, K~, M, e^{b_C}
//   scan_kernel (seq_scan.cu)                 one CTA per (128 value columns, head, sequence) walks the chunks in order.
//
// Exponents of decays are never positive: products e^{b_i - b_j} = e^{b_i - r} e^{r - b_j} use a reference r between the two tokens (the
// token before the 16- or 8-row block of i), and pairs inside one 8-row block are evaluated directly. So a decay of any strength
// underflows to zero and nothing overflows.
//
// The recurrence is fp32: every operand of a product is split into two bf16 terms (hi + lo) and the product takes the three terms
// hi hi + hi lo + lo hi, i.e. about 16 bits of mantissa, with fp32 accumulation and an fp32 state. The scan's products (128 x 64 .. 128
// x 64 .. 128) run on tcgen05 (seq_scan.cu); the 8- and 16-row blocks in here are 16 x 8 x 16 mma.sync on register fragments, whose
// operands are formed in registers (decays times keys) and never stored.
#include "seq_chunk.cuh"

namespace plz {
namespace {

constexpr float kL2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2a(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// z / (1 + e^-z) of a bf16 input, about 2^-21 relative
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + ex2a(-z * kL2e)); }
// two fp32 per instruction
struct F2x2 { uint64_t a, b; };
__device__ __forceinline__ F2x2 ld_f2x2(const float* p) {
    const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
    return {v.x, v.y};
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) { uint64_t d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) { uint64_t d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ uint64_t sub2(uint64_t a, uint64_t b) { uint64_t d; asm("sub.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ uint64_t ex2_2(uint64_t a) {
    return (uint64_t)__float_as_uint(ex2a(__uint_as_float((uint32_t)a))) | ((uint64_t)__float_as_uint(ex2a(__uint_as_float((uint32_t)(a >> 32)))) << 32);
}
// 16 bytes global -> shared, zeros when !in (the address must be valid all the same)
__device__ __forceinline__ void cp16z(uint32_t dst, const void* src, bool in) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct AFrag { uint32_t h[4], l[4]; };
__device__ __forceinline__ void mma_split(float (&d)[4], const AFrag& a, uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
    mma16816(d, a.h, bh0, bh1);
    mma16816(d, a.h, bl0, bl1);
    mma16816(d, a.l, bh0, bh1);
}
// the 16 x 16 blocks of M above the diagonal (the scan multiplies the whole tile), 256 threads
__device__ __forceinline__ void zero_upper(uint8_t* wM, uint32_t plane, int tid) {
    for (int e = tid; e < kC * kC / 8; e += 256) {
        const uint32_t r = e / (kC / 8), c = (e % (kC / 8)) * 8;
        if ((c >> 4) > (r >> 4)) {
            const uint32_t at = ChunkWs<1, 64>::at(kC, r, c);
            *reinterpret_cast<uint4*>(wM + at) = make_uint4(0u, 0u, 0u, 0u);
            *reinterpret_cast<uint4*>(wM + plane + at) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
}

struct ChunkParams {
    // delta: fp32 q, k [rows, G * dk], v [rows, H * dv], logg [rows, H * dk], beta [rows, H]; decay: bf16 slices, pitch ld
    const void* q; const void* k; const void* v; long long ld;
    const float* logg; const float* beta; const float* decay;
    float* state; float* o;
    uint8_t* ws; long long ws_stride;
    int n, t_begin, chunks;      // tokens per sequence; first token and number of chunks of this segment
    int H, G, dk, dv, dvp;
    int vec, vec_v;              // rows (of v) allow 16-byte loads
};

// ---------------------------------------------------------------------------------------------------------------------
// gated delta rule, per chunk
// ---------------------------------------------------------------------------------------------------------------------
template <int DK>
struct DeltaSmem {
    static constexpr int PK = DK + 4, PB = 17, PT = kC + 4;
    float q[kC][PK], k[kC][PK];      // k turns into Kbar = k e^b once A' and M are done
    union {
        float b[kC][PK];             // cumulative log2 decay
        struct { float t[kC][PT], tmp[4][16][20]; } inv;   // afterwards: T, and a block product per warp
    };
    float a[10][16][PB];             // beta A', strictly lower, as 16 x 16 blocks (I, J <= I) at I (I + 1) / 2 + J
    float beta[kC];
};

// 256 threads: warps 0-3 the products between blocks, warps 4-7 the 8 x 8 diagonal blocks, then all of them.
template <int DK>
__global__ void __launch_bounds__(256, 2)
delta_chunk_kernel(const ChunkParams p) {
    extern __shared__ __align__(16) uint8_t sm_raw[];
    DeltaSmem<DK>& s = *reinterpret_cast<DeltaSmem<DK>*>(sm_raw);
    constexpr int KS = DK / 16;
    const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31, r4 = lane >> 2, c2 = (lane & 3) * 2;
    const int ch = blockIdx.x, h = blockIdx.y, b = blockIdx.z, hk = h / (p.H / p.G);
    const int t0 = p.t_begin + ch * kC, L = min(kC, p.n - t0);
    const long long row0 = (long long)b * p.n + t0;
    uint8_t* ws = p.ws + (((long long)b * p.H + h) * p.chunks + ch) * p.ws_stride;
    using W = ChunkWs<DK / 64, 128>;
    uint8_t* wM = ws + W::OFF_B;
    float* U0 = reinterpret_cast<float*>(ws + W::OFF_U);
    const long long ldq = (long long)p.G * p.dk, ldg = (long long)p.H * p.dk;
    const float* qg = (const float*)p.q + (row0 * p.G + hk) * p.dk;
    const float* kg = (const float*)p.k + (row0 * p.G + hk) * p.dk;
    const float* gg = p.logg + (row0 * p.H + h) * p.dk;

    if (p.vec) {
#pragma unroll
        for (int i = 0; i < kC * DK / 4 / 256; ++i) {
            const int e = tid + i * 256, t = e / (DK / 4), c = (e % (DK / 4)) * 4;
            const bool in = t < L && c < p.dk;
            const int tc = min(t, L - 1), cc = min(c, p.dk - 4);
            cp16z(smem_u32(&s.q[t][c]), qg + tc * ldq + cc, in);
            cp16z(smem_u32(&s.k[t][c]), kg + tc * ldq + cc, in);
            cp16z(smem_u32(&s.b[t][c]), gg + tc * ldg + cc, in);
        }
        cp_commit();
    } else {
        for (int e = tid; e < kC * DK; e += 256) {
            const int t = e / DK, c = e % DK;
            const bool in = t < L && c < p.dk;
            s.q[t][c] = in ? qg[t * ldq + c] : 0.f;
            s.k[t][c] = in ? kg[t * ldq + c] : 0.f;
            s.b[t][c] = in ? gg[t * ldg + c] : 0.f;
        }
    }
    if (tid < kC) s.beta[tid] = tid < L ? p.beta[(row0 + tid) * p.H + h] : 0.f;
    cp_wait_all();
    __syncthreads();
    // inclusive sum over the 64 tokens, two threads per channel (the second half adds the first half's total)
    if (tid < 2 * DK) {
        const int c = tid % DK, h0 = tid / DK * 32;
        float run = 0.f;
#pragma unroll 16
        for (int t = 0; t < 32; ++t) { run = fmaf(s.b[h0 + t][c], kL2e, run); s.b[h0 + t][c] = run; }
    }
    __syncthreads();
    for (int e = tid; e < 32 * DK; e += 256) s.b[32 + e / DK][e % DK] += s.b[31][e % DK];
    __syncthreads();

    if (w < 4) {
        // ---- products between blocks. job = 16-row block rb against 8-column tiles nt0 .. nt0 + ntn - 1:
        //   part 0  tiles left of the diagonal 16-block, reference token 16 rb - 1
        //   part 1  rows 8..15 against columns 0..7 of the diagonal 16-block, reference token 16 rb + 7
        const int n_jobs = (w & 1) ? 3 : 1;
        for (int job = 0; job < n_jobs; ++job) {
            int rb, part = 0, nt0 = 0, ntn = 4;
            if (w == 0) rb = 3;
            else if (w == 2) rb = 2;
            else if (w == 1) { rb = job < 2 ? 3 : 0; part = job > 0; nt0 = 4; ntn = 2; }
            else { rb = job < 2 ? 1 : 2; part = job > 0; ntn = 2; }
            if (part) { nt0 = 2 * rb; ntn = 1; }
            const int ref = part == 0 ? 16 * rb - 1 : 16 * rb + 7;
            const int i0 = 16 * rb + r4, i1 = i0 + 8;
            float kk[4][4], qk[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) { kk[i][e] = 0.f; qk[i][e] = 0.f; }
#pragma unroll 1
            for (int ks = 0; ks < KS; ++ks) {
                AFrag ak, aq;
                float2 rr[2];
#pragma unroll
                for (int half = 0; half < 2; ++half) {          // k columns c2, c2 + 1 and + 8
                    const int c = ks * 16 + c2 + half * 8;
                    const float2 rf = *reinterpret_cast<const float2*>(&s.b[ref][c]);
                    rr[half] = rf;
                    float2 ka = make_float2(0.f, 0.f), qa = ka;
                    if (part == 0) {
                        const float2 bb = *reinterpret_cast<const float2*>(&s.b[i0][c]);
                        const float2 kv = *reinterpret_cast<const float2*>(&s.k[i0][c]), qv = *reinterpret_cast<const float2*>(&s.q[i0][c]);
                        const float e0 = ex2a(bb.x - rf.x), e1 = ex2a(bb.y - rf.y);
                        ka = make_float2(kv.x * e0, kv.y * e1); qa = make_float2(qv.x * e0, qv.y * e1);
                    }
                    split2(ka.x, ka.y, ak.h[half * 2], ak.l[half * 2]);
                    split2(qa.x, qa.y, aq.h[half * 2], aq.l[half * 2]);
                    const float2 bb = *reinterpret_cast<const float2*>(&s.b[i1][c]);
                    const float2 kv = *reinterpret_cast<const float2*>(&s.k[i1][c]), qv = *reinterpret_cast<const float2*>(&s.q[i1][c]);
                    const float e0 = ex2a(bb.x - rf.x), e1 = ex2a(bb.y - rf.y);
                    split2(kv.x * e0, kv.y * e1, ak.h[half * 2 + 1], ak.l[half * 2 + 1]);
                    split2(qv.x * e0, qv.y * e1, aq.h[half * 2 + 1], aq.l[half * 2 + 1]);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (i < ntn) {
                        const int j = (nt0 + i) * 8 + r4, c = ks * 16 + c2;
                        const float2 k0 = *reinterpret_cast<const float2*>(&s.k[j][c]), k1 = *reinterpret_cast<const float2*>(&s.k[j][c + 8]);
                        const float2 b0 = *reinterpret_cast<const float2*>(&s.b[j][c]), b1 = *reinterpret_cast<const float2*>(&s.b[j][c + 8]);
                        uint32_t bh0, bl0, bh1, bl1;
                        split2(k0.x * ex2a(rr[0].x - b0.x), k0.y * ex2a(rr[0].y - b0.y), bh0, bl0);
                        split2(k1.x * ex2a(rr[1].x - b1.x), k1.y * ex2a(rr[1].y - b1.y), bh1, bl1);
                        mma_split(kk[i], ak, bh0, bh1, bl0, bl1);
                        mma_split(qk[i], aq, bh0, bh1, bl0, bl1);
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (i < ntn) {
                    const int j = (nt0 + i) * 8 + c2, blk = rb * (rb + 1) / 2 + (nt0 + i) / 2, jj = ((nt0 + i) & 1) * 8 + c2;
                    if (part == 0) {
                        s.a[blk][r4][jj] = kk[i][0] * s.beta[i0]; s.a[blk][r4][jj + 1] = kk[i][1] * s.beta[i0];
                        put_split(wM + W::at(kC, i0, j), W::M_PLANE, qk[i][0], qk[i][1]);
                    }
                    s.a[blk][r4 + 8][jj] = kk[i][2] * s.beta[i1]; s.a[blk][r4 + 8][jj + 1] = kk[i][3] * s.beta[i1];
                    put_split(wM + W::at(kC, i1, j), W::M_PLANE, qk[i][2], qk[i][3]);
                }
            }
        }
    } else {
        // ---- pairs inside the 8-row diagonal blocks: lane = (row, one of four channel slices), all exponents explicit
        const int rb = w - 4;
        for (int blk = 0; blk < 2; ++blk) {
            const int base = 16 * rb + 8 * blk, ri = lane & 7, row = base + ri, quarter = lane >> 3;
            uint64_t ak[8], aq[8];          // pairs of partial sums
#pragma unroll
            for (int j = 0; j < 8; ++j) { ak[j] = 0ull; aq[j] = 0ull; }
#pragma unroll 1
            for (int c4 = quarter; c4 < DK / 4; c4 += 4) {
                const int c = c4 * 4;
                const F2x2 bi = ld_f2x2(&s.b[row][c]), ki = ld_f2x2(&s.k[row][c]), qi = ld_f2x2(&s.q[row][c]);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const F2x2 bj = ld_f2x2(&s.b[base + j][c]), kj = ld_f2x2(&s.k[base + j][c]);
                    // j > row: an exponent above zero, discarded below
                    const uint64_t e0 = mul2(ex2_2(sub2(bi.a, bj.a)), kj.a), e1 = mul2(ex2_2(sub2(bi.b, bj.b)), kj.b);
                    ak[j] = fma2(ki.a, e0, ak[j]); ak[j] = fma2(ki.b, e1, ak[j]);
                    aq[j] = fma2(qi.a, e0, aq[j]); aq[j] = fma2(qi.b, e1, aq[j]);
                }
            }
            float sk[8], sq[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                sk[j] = __uint_as_float((uint32_t)ak[j]) + __uint_as_float((uint32_t)(ak[j] >> 32));
                sq[j] = __uint_as_float((uint32_t)aq[j]) + __uint_as_float((uint32_t)(aq[j] >> 32));
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                sk[j] += __shfl_xor_sync(0xFFFFFFFFu, sk[j], 8); sk[j] += __shfl_xor_sync(0xFFFFFFFFu, sk[j], 16);
                sq[j] += __shfl_xor_sync(0xFFFFFFFFu, sq[j], 8); sq[j] += __shfl_xor_sync(0xFFFFFFFFu, sq[j], 16);
            }
            if (quarter == 0) {
#pragma unroll
                for (int j = 0; j < 8; ++j) s.a[rb * (rb + 1) / 2 + rb][8 * blk + ri][8 * blk + j] = j < ri ? sk[j] * s.beta[row] : 0.f;
            } else if (quarter == 1) {
#pragma unroll
                for (int j = 0; j < 8; j += 2)
                    put_split(wM + W::at(kC, row, base + j), W::M_PLANE, j <= ri ? sq[j] : 0.f, j + 1 <= ri ? sq[j + 1] : 0.f);
            } else if (quarter == 2 && blk == 0) {
                // rows 0..7 against columns 8..15 of the 16-row block lie above the diagonal
#pragma unroll
                for (int j = 0; j < 8; j += 2) put_split(wM + W::at(kC, row, base + 8 + j), W::M_PLANE, 0.f, 0.f);
            }
        }
    }
    __syncthreads();
    // ---- Q~, K~, e^{b_C}; k -> Kbar ---------------------------------------------------------------------------------------
#pragma unroll 2
    for (int e = tid; e < kC * DK / 4; e += 256) {
        const int t = e / (DK / 4), c = (e % (DK / 4)) * 4;
        const float4 qv = *reinterpret_cast<const float4*>(&s.q[t][c]), kv = *reinterpret_cast<const float4*>(&s.k[t][c]);
        const float4 bt = *reinterpret_cast<const float4*>(&s.b[t][c]), be = *reinterpret_cast<const float4*>(&s.b[kC - 1][c]);
        const float4 x = make_float4(ex2a(bt.x), ex2a(bt.y), ex2a(bt.z), ex2a(bt.w));
        put_split4(ws + W::at(128, 64 + t, c), W::A_PLANE, qv.x * x.x, qv.y * x.y, qv.z * x.z, qv.w * x.w);
        put_split4(ws + W::OFF_K + W::at(kC, t, c), W::K_PLANE, kv.x * ex2a(be.x - bt.x), kv.y * ex2a(be.y - bt.y), kv.z * ex2a(be.z - bt.z),
                   kv.w * ex2a(be.w - bt.w));
        *reinterpret_cast<float4*>(&s.k[t][c]) = make_float4(kv.x * x.x, kv.y * x.y, kv.z * x.z, kv.w * x.w);
    }
    if (tid < DK) reinterpret_cast<float*>(ws + W::OFF_DEC)[tid] = ex2a(s.b[kC - 1][tid]);
    zero_upper(wM, W::M_PLANE, tid);
    __syncthreads();
    // the values take the place of q while T is computed
    const float* vg = (const float*)p.v + (row0 * p.H + h) * (long long)p.dv;
    const long long ldv = (long long)p.H * p.dv;
    const bool v_in_smem = p.vec_v && p.dv <= DK;
    if (v_in_smem) {
#pragma unroll
        for (int i = 0; i < kC * DK / 4 / 256; ++i) {
            const int e = tid + i * 256, t = e / (DK / 4), c = (e % (DK / 4)) * 4;
            cp16z(smem_u32(&s.q[t][c]), vg + (long long)min(t, L - 1) * ldv + min(c, p.dv - 4), t < L && c < p.dv);
        }
        cp_commit();
    }

    // ---- T = (I + a)^{-1}: 16-row diagonal blocks by substitution, then block diagonals outwards -------------------------
    if (w < 4 && lane < 16) {
        const int blk = w * (w + 1) / 2 + w;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float v = i == lane ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < i; ++j) v = fmaf(-s.a[blk][i][j], x[j], v);
            x[i] = v;
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) s.inv.t[16 * w + i][16 * w + lane] = x[i];
    }
    __syncthreads();
    // a block takes two warps: 16 columns x 8 rows each
    for (int d = 1; d < 4; ++d) {
        const int J = w >> 1, I = J + d, col = lane & 15, rh = (w & 1) * 8 + (lane >> 4) * 4;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        if (I < 4) {
            for (int K = J; K < I; ++K) {
                const float(*ab)[DeltaSmem<DK>::PB] = s.a[I * (I + 1) / 2 + K];
#pragma unroll
                for (int kk = 0; kk < 16; ++kk) {
                    const float tv = s.inv.t[16 * K + kk][16 * J + col];
#pragma unroll
                    for (int i = 0; i < 4; ++i) acc[i] = fmaf(ab[rh + i][kk], tv, acc[i]);
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) s.inv.tmp[J][rh + i][col] = acc[i];
        }
        __syncthreads();
        if (I < 4) {
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i] = 0.f;
#pragma unroll
            for (int kk = 0; kk < 16; ++kk) {
                const float pv = s.inv.tmp[J][kk][col];
#pragma unroll
                for (int i = 0; i < 4; ++i) acc[i] = fmaf(s.inv.t[16 * I + rh + i][16 * I + kk], pv, acc[i]);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) s.inv.t[16 * I + rh + i][16 * J + col] = -acc[i];
        }
        __syncthreads();
    }

    // ---- -W = -(T beta) Kbar and U0 = (T beta) V. Warps w and w + 4 share an 8-column tile: row blocks {0, 3} and {1, 2} ------
    const int half_m = w >> 2;
    const int m0 = half_m ? 1 : 0, m1 = half_m ? 2 : 3;
    AFrag at[5];      // blocks (m0, 0 .. m0), then (m1, 0 .. m1)
#pragma unroll
    for (int f = 0; f < 5; ++f) {
        const int m = f <= m0 ? m0 : m1, ks = f <= m0 ? f : f - m0 - 1;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 16 * m + r4 + (x & 1) * 8, j = 16 * ks + c2 + (x >> 1) * 8;
            split2(s.inv.t[i][j] * s.beta[j], s.inv.t[i][j + 1] * s.beta[j + 1], at[f].h[x], at[f].l[x]);
        }
    }
    const int nt_w = DK / 8, nt_all = nt_w + p.dvp / 8;
    cp_wait_all();
    __syncthreads();
#pragma unroll 1
    for (int nt = w & 3; nt < nt_all; nt += 4) {
        const bool is_w = nt < nt_w;
        const int c = (is_w ? nt : nt - nt_w) * 8 + r4;
        float f[4][4];
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int j = 16 * ks + c2 + (x & 1) + (x >> 1) * 8;
                if (is_w) f[ks][x] = -s.k[j][c];
                else if (v_in_smem) f[ks][x] = s.q[j][c];
                // past the last token T's column has beta = 0, past the last value column nobody reads: any finite value will do
                else f[ks][x] = __ldg(vg + (long long)min(j, L - 1) * ldv + min(c, p.dv - 1));
            }
        float acc0[4] = {0.f, 0.f, 0.f, 0.f}, acc1[4] = {0.f, 0.f, 0.f, 0.f};
        uint32_t bh[4][2], bl[4][2];
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) { split2(f[ks][0], f[ks][1], bh[ks][0], bl[ks][0]); split2(f[ks][2], f[ks][3], bh[ks][1], bl[ks][1]); }
        if (half_m == 0) {
            mma_split(acc0, at[0], bh[0][0], bh[0][1], bl[0][0], bl[0][1]);
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) mma_split(acc1, at[1 + ks], bh[ks][0], bh[ks][1], bl[ks][0], bl[ks][1]);
        } else {
#pragma unroll
            for (int ks = 0; ks < 2; ++ks) mma_split(acc0, at[ks], bh[ks][0], bh[ks][1], bl[ks][0], bl[ks][1]);
#pragma unroll
            for (int ks = 0; ks < 3; ++ks) mma_split(acc1, at[2 + ks], bh[ks][0], bh[ks][1], bl[ks][0], bl[ks][1]);
        }
        const int cc = (is_w ? nt : nt - nt_w) * 8 + c2;
#pragma unroll
        for (int mm = 0; mm < 2; ++mm)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = 16 * (mm ? m1 : m0) + r4 + hf * 8;
                const float x = mm ? acc1[hf * 2] : acc0[hf * 2], y = mm ? acc1[hf * 2 + 1] : acc0[hf * 2 + 1];
                if (is_w) put_split(ws + W::at(128, i, cc), W::A_PLANE, x, y);
                else *reinterpret_cast<float2*>(U0 + (long long)i * p.dvp + cc) = make_float2(x, y);
            }
    }
}

// ---------------------------------------------------------------------------------------------------------------------
// decayed linear attention, per chunk
// ---------------------------------------------------------------------------------------------------------------------
template <int DK>
struct DecaySmem {
    static constexpr int PK = DK + 4;
    float q[kC][PK], k[kC][PK];
    float pw[kC + 1];               // powers of the decay
};
template <int DK>
__global__ void __launch_bounds__(256)
decay_chunk_kernel(const ChunkParams p) {
    extern __shared__ uint8_t sm_raw[];
    DecaySmem<DK>& s = *reinterpret_cast<DecaySmem<DK>*>(sm_raw);
    constexpr int KS = DK / 16;
    const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31, r4 = lane >> 2, c2 = (lane & 3) * 2;
    const int ch = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
    const int t0 = p.t_begin + ch * kC, L = min(kC, p.n - t0);
    const long long row0 = (long long)b * p.n + t0;
    uint8_t* ws = p.ws + (((long long)b * p.H + h) * p.chunks + ch) * p.ws_stride;
    using W = ChunkWs<DK / 64, 64>;
    uint8_t* wM = ws + W::OFF_B;
    float* U0 = reinterpret_cast<float*>(ws + W::OFF_U);
    const __nv_bfloat16* qg = (const __nv_bfloat16*)p.q + row0 * p.ld + (long long)h * p.dk;
    const __nv_bfloat16* kg = (const __nv_bfloat16*)p.k + row0 * p.ld + (long long)h * p.dk;
    const __nv_bfloat16* vg = (const __nv_bfloat16*)p.v + row0 * p.ld + (long long)h * p.dv;
    if (tid <= kC) s.pw[tid] = powf(p.decay[h], (float)tid);
    if (p.vec) {
#pragma unroll 4
        for (int e = tid; e < kC * DK / 8; e += 256) {
            const int t = e / (DK / 8), c = (e % (DK / 8)) * 8;
            float fq[8], fk[8];
            const bool in = t < L && c < p.dk;
            const long long at = min(t, L - 1) * p.ld + min(c, p.dk - 8);      // unconditional loads
            load8(qg + at, fq); load8(kg + at, fk);
#pragma unroll
            for (int i = 0; i < 8; ++i) { s.q[t][c + i] = in ? silu_fast(fq[i]) : 0.f; s.k[t][c + i] = in ? silu_fast(fk[i]) : 0.f; }
        }
        const int v8 = p.dvp / 8;
#pragma unroll 4
        for (int e = tid; e < kC * v8; e += 256) {
            const int t = e / v8, c = (e - t * v8) * 8;
            float f[8];
            const bool in = t < L && c < p.dv;
            load8(vg + min(t, L - 1) * p.ld + min(c, p.dv - 8), f);
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] = in ? silu_fast(f[i]) : 0.f;
            *reinterpret_cast<float4*>(U0 + (long long)t * p.dvp + c) = make_float4(f[0], f[1], f[2], f[3]);
            *reinterpret_cast<float4*>(U0 + (long long)t * p.dvp + c + 4) = make_float4(f[4], f[5], f[6], f[7]);
        }
    } else {
        for (int e = tid; e < kC * DK; e += 256) {
            const int t = e / DK, c = e % DK;
            const bool in = t < L && c < p.dk;
            s.q[t][c] = in ? silu_fast(to_f(qg[t * p.ld + c])) : 0.f;
            s.k[t][c] = in ? silu_fast(to_f(kg[t * p.ld + c])) : 0.f;
        }
        for (int e = tid; e < kC * p.dvp; e += 256) {
            const int t = e / p.dvp, c = e % p.dvp;
            U0[e] = (t < L && c < p.dv) ? silu_fast(to_f(vg[t * p.ld + c])) : 0.f;
        }
    }
    __syncthreads();
    // M: warps w and w + 4 share 16 rows, taking the 8-column tiles of either half
    const int rb = w & 3, nh = w >> 2, ntn = rb + 1;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll 2
    for (int ks = 0; ks < KS; ++ks) {
        AFrag a;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 16 * rb + r4 + (x & 1) * 8, c = ks * 16 + c2 + (x >> 1) * 8;
            const float2 f = *reinterpret_cast<const float2*>(&s.q[i][c]);
            split2(f.x, f.y, a.h[x], a.l[x]);
        }
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            if (nt < ntn) {
                const int j = (nh * ntn + nt) * 8 + r4, c = ks * 16 + c2;
                const float2 f0 = *reinterpret_cast<const float2*>(&s.k[j][c]), f1 = *reinterpret_cast<const float2*>(&s.k[j][c + 8]);
                uint32_t bh0, bl0, bh1, bl1;
                split2(f0.x, f0.y, bh0, bl0);
                split2(f1.x, f1.y, bh1, bl1);
                mma_split(acc[nt], a, bh0, bh1, bl0, bl1);
            }
        }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
        if (nt < ntn) {
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = 16 * rb + r4 + hf * 8, j = (nh * ntn + nt) * 8 + c2;
                const float m0 = i >= j ? acc[nt][hf * 2] * s.pw[i - j] : 0.f, m1 = i >= j + 1 ? acc[nt][hf * 2 + 1] * s.pw[i - j - 1] : 0.f;
                put_split(wM + W::at(kC, i, j), W::M_PLANE, m0, m1);
            }
        }
    }
    zero_upper(wM, W::M_PLANE, tid);
#pragma unroll 4
    for (int e = tid; e < kC * DK / 4; e += 256) {
        const int t = e / (DK / 4), c = (e % (DK / 4)) * 4;
        const float fq = s.pw[t + 1], fk = t < L ? s.pw[L - 1 - t] : 0.f;
        const float4 qv = *reinterpret_cast<const float4*>(&s.q[t][c]), kv = *reinterpret_cast<const float4*>(&s.k[t][c]);
        put_split4(ws + W::at(64, t, c), W::A_PLANE, qv.x * fq, qv.y * fq, qv.z * fq, qv.w * fq);
        put_split4(ws + W::OFF_K + W::at(kC, t, c), W::K_PLANE, kv.x * fk, kv.y * fk, kv.z * fk, kv.w * fk);
    }
    if (tid < DK) reinterpret_cast<float*>(ws + W::OFF_DEC)[tid] = s.pw[L];
}

template <int DK, bool DELTA>
int launch_chunked(ChunkParams p, int B, void* ws, long long ws_bytes, cudaStream_t stream) {
    p.dvp = (p.dv + 15) / 16 * 16;
    p.ws = (uint8_t*)ws;
    p.ws_stride = ChunkWs<DK / 64, DELTA ? 128 : 64>::bytes(p.dvp);
    const long long per_chunk = p.ws_stride * B * p.H;
    const int all = (p.n + kC - 1) / kC;
    long long seg = ws_bytes / per_chunk;
    if (seg < 1) { set_last_error("chunked recurrence: workspace of %lld bytes holds no chunk (%lld needed)", ws_bytes, per_chunk); return PLZ_ERR_WORKSPACE; }
    if ((uintptr_t)ws & 15) { set_last_error("chunked recurrence: workspace must be 16-byte aligned"); return PLZ_ERR_BAD_ALIGN; }
    if (seg > all) seg = all;
    const long long rounds = (all + seg - 1) / seg;
    seg = (all + rounds - 1) / rounds;
    const int smem = DELTA ? (int)sizeof(DeltaSmem<DK>) : (int)sizeof(DecaySmem<DK>);
    static bool once[64] = {};
    int dev = 0;
    PLZ_CUDA_CHECK(cudaGetDevice(&dev));
    if (!once[dev & 63]) {
        if (DELTA) PLZ_CUDA_CHECK(cudaFuncSetAttribute(delta_chunk_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        else PLZ_CUDA_CHECK(cudaFuncSetAttribute(decay_chunk_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        once[dev & 63] = true;
    }
    for (int c0 = 0; c0 < all; c0 += (int)seg) {
        p.t_begin = c0 * kC;
        p.chunks = all - c0 < (int)seg ? all - c0 : (int)seg;
        if (DELTA) delta_chunk_kernel<DK><<<dim3(p.chunks, p.H, B), 256, smem, stream>>>(p);
        else decay_chunk_kernel<DK><<<dim3(p.chunks, p.H, B), 256, smem, stream>>>(p);
        PLZ_LAUNCH_CHECK();
        const ScanArgs a = {p.ws, p.ws_stride, p.state, p.o, B, p.n, p.t_begin, p.chunks, p.H, p.dk, p.dv, p.dvp};
        const int rc = launch_chunk_scan(a, DELTA, DK / 64, stream);
        if (rc) return rc;
    }
    return PLZ_OK;
}
template <bool DELTA>
int launch_dk(const ChunkParams& p, int B, void* ws, long long ws_bytes, cudaStream_t stream) {
    if (p.dk <= 64) return launch_chunked<64, DELTA>(p, B, ws, ws_bytes, stream);
    if (p.dk <= 128) return launch_chunked<128, DELTA>(p, B, ws, ws_bytes, stream);
    set_last_error("chunked recurrence: key size %d (at most 128)", p.dk);
    return PLZ_ERR_UNSUPPORTED;
}

}  // namespace

// bytes that hold every chunk of n tokens; any amount down to one chunk of all heads works (the scan then runs in segments)
long long chunk_ws_bytes(int B, int n, int H, int dk, int dv) {
    if (dk > 128) return 0;
    const int dvp = (dv + 15) / 16 * 16;
    const long long per = dk <= 64 ? ChunkWs<1, 128>::bytes(dvp) : ChunkWs<2, 128>::bytes(dvp);
    const long long one = per * B * H, all = one * ((n + kC - 1) / kC), cap = 512ll << 20;
    return all <= cap ? all : (one > cap ? one : cap / one * one);
}

int launch_chunk_decay(const DecayAttnArgs& a, void* ws, long long ws_bytes, cudaStream_t stream) {
    ChunkParams p = {};
    p.q = a.q; p.k = a.k; p.v = a.v; p.ld = a.ld; p.decay = a.decay; p.state = a.state; p.o = a.o;
    p.n = a.n; p.H = a.H; p.G = a.H; p.dk = a.dk; p.dv = a.dv;
    p.vec = a.dk % 8 == 0 && a.dv % 8 == 0 && a.ld % 8 == 0 && !(((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v) & 15);
    return launch_dk<false>(p, a.B, ws, ws_bytes, stream);
}
int launch_chunk_delta(const DeltaRuleArgs& a, void* ws, long long ws_bytes, cudaStream_t stream) {
    ChunkParams p = {};
    p.q = a.q; p.k = a.k; p.v = a.v; p.logg = a.logg; p.beta = a.beta; p.state = a.state; p.o = a.o;
    p.n = a.n; p.H = a.H; p.G = a.G; p.dk = a.dk; p.dv = a.dv;
    p.vec_v = a.dv % 4 == 0 && !((uintptr_t)a.v & 15);
    p.vec = a.dk % 4 == 0 && !(((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.logg) & 15);
    return launch_dk<true>(p, a.B, ws, ws_bytes, stream);
}

}  // namespace plz
