// Dense Linear y = act(x W^T + b) for the hybrid decoders, weights bf16 or fp32 [N, K] row-major.
//
//   linear_rows_kernel   a handful of rows (token decode): bound by streaming W once. KS warps of a block share the reduction of
//                        two output rows, chosen so that the launch has enough loads in flight whatever N is; the first
//                        weights are requested before the wait on the previous kernel of the stream.
//   linear_skinny_kernel 2 .. 16 rows, bf16: the same streaming with mma.sync fragments loaded straight from memory.
//                        Both also serve one small product per head (grid y = head, z = group of 16 rows).
//   linear_tile_kernel   any shape and both types on the CUDA cores, fp32 products and sums: the 32-bit mode, and bf16 shapes
//                        that the tensor-core path's 16-byte rows exclude.
//   launch_seq_linear    picks one of them or the tcgen05 GEMM (lut_gemm.cu, dense B, bias and activation in its epilogue).
#include "seq_math.cuh"

namespace plz {
namespace {

struct LinParams {
    const void* x; long long ldx;
    const void* w; long long ldw;
    const void* bias;
    void* y; long long ldy;
    int M, N, K, act;
    // one product per head (plz_head_linear): elements between heads; outputs may be multiplied by sigmoid(gate)
    long long xh, wh, yh;
    const void* gate; long long ldg, gh;
};

// value of output (m, n) of a head, already summed, into y
template <typename T, typename TO>
__device__ __forceinline__ void put(const LinParams& p, int head, int m, int n, float v) {
    if (p.gate) v *= sigmoid_f(to_f(((const T*)p.gate)[(long long)m * p.ldg + head * p.gh + n]));
    ((TO*)p.y)[(long long)m * p.ldy + head * p.yh + n] = from_f<TO>(v);
}

template <typename T> struct Raw8;
template <> struct Raw8<__nv_bfloat16> {
    uint4 r;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { r = __ldg(reinterpret_cast<const uint4*>(p)); }
    __device__ __forceinline__ void zero() { r = make_uint4(0u, 0u, 0u, 0u); }
    __device__ __forceinline__ void unpack(float (&f)[8]) const {
        const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u); }
    }
};
template <> struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = __ldg(reinterpret_cast<const float4*>(p)); b = __ldg(reinterpret_cast<const float4*>(p + 4)); }
    __device__ __forceinline__ void zero() { a = make_float4(0.f, 0.f, 0.f, 0.f); b = a; }
    __device__ __forceinline__ void unpack(float (&f)[8]) const {
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    }
};

constexpr int kRowsBatch = 4;   // 8-element chunks of a weight row in flight per lane and row

// K % 8 == 0 and 16-byte aligned rows. Block = 8 warps = 8 / KS pairs of output rows.
template <typename T, typename TO, int MR>
__global__ void __launch_bounds__(256)
linear_rows_kernel(const LinParams p, int ks) {
    __shared__ float part[8][2][MR];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pairs = 8 / ks, pair = warp / ks, kw = warp % ks;
    const int n0 = ((int)blockIdx.x * pairs + pair) * 2;
    const int chunks = p.K >> 3, step = 32 * ks;
    const bool has0 = n0 < p.N, has1 = n0 + 1 < p.N;
    const int head = blockIdx.y;
    const T* w0 = (const T*)p.w + head * p.wh + (long long)n0 * p.ldw;
    const T* w1 = w0 + p.ldw;
    const T* x = (const T*)p.x + head * p.xh;
    Raw8<T> a[kRowsBatch], b[kRowsBatch];
    auto fetch = [&](int c) {
#pragma unroll
        for (int i = 0; i < kRowsBatch; ++i) {
            const int cc = c + i * step;
            if (has0 && cc < chunks) a[i].load(w0 + cc * 8); else a[i].zero();
            if (has1 && cc < chunks) b[i].load(w1 + cc * 8); else b[i].zero();
        }
    };
    int c = kw * 32 + lane;
    fetch(c);                          // weights do not depend on the previous kernel
    pdl_launch_dependents();
    pdl_wait();
    float s0[MR], s1[MR];
#pragma unroll
    for (int m = 0; m < MR; ++m) { s0[m] = 0.f; s1[m] = 0.f; }
    while (c < chunks) {
#pragma unroll
        for (int i = 0; i < kRowsBatch; ++i) {
            const int cc = c + i * step;
            if (cc < chunks) {
                float f0[8], f1[8];
                a[i].unpack(f0); b[i].unpack(f1);
#pragma unroll
                for (int m = 0; m < MR; ++m) {
                    if (m < p.M) {
                        float xv[8];
                        load8(x + (long long)m * p.ldx + cc * 8, xv);
#pragma unroll
                        for (int e = 0; e < 8; ++e) { s0[m] = fmaf(f0[e], xv[e], s0[m]); s1[m] = fmaf(f1[e], xv[e], s1[m]); }
                    }
                }
            }
        }
        c += kRowsBatch * step;
        if (c < chunks) fetch(c);
    }
#pragma unroll
    for (int m = 0; m < MR; ++m) {
        const float t0 = warp_sum(s0[m]), t1 = warp_sum(s1[m]);
        if (lane == 0) { part[warp][0][m] = t0; part[warp][1][m] = t1; }
    }
    __syncthreads();
    if (kw == 0 && lane < 2 * MR) {
        const int r = lane / MR, m = lane % MR;
        if (m < p.M && n0 + r < p.N) {
            float v = 0.f;
            for (int i = 0; i < ks; ++i) v += part[warp + i][r][m];
            if (p.act == ACT_GLU_GELU) {
                if (r == 0) {
                    float u = 0.f;
                    for (int i = 0; i < ks; ++i) u += part[warp + i][1][m];
                    put<T, TO>(p, head, m, n0 >> 1, gelu_tanh_f(v) * u);
                }
            } else {
                if (p.bias) v += to_f(((const T*)p.bias)[n0 + r]);
                put<T, TO>(p, head, m, n0 + r, activate(v, p.act));
            }
        }
    }
}

// 2 .. 16 rows of x, bf16: a warp takes 16 output rows (weight rows) as the A operand of m16n8k16 mma.sync, x as B. The order of the
// reduction index inside a product is free, so lane (r, q) loads 16 contiguous bytes of weight rows r and r + 8 and of x row r at
// k0 + 8 q and uses them as the fragments of two products: no shuffle, no shared memory, no unpacking. KS warps share the reduction.
template <typename TO, int NT>     // NT: groups of eight x rows
__global__ void __launch_bounds__(256)
linear_skinny_kernel(const LinParams p, int ks) {
    __shared__ float part[8][16][8 * NT + 1];
    constexpr int U = 4;           // 32-wide steps in flight
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r4 = lane >> 2, q8 = (lane & 3) * 8;
    const int groups = 8 / ks, grp = warp / ks, kw = warp % ks;
    const int n0 = ((int)blockIdx.x * groups + grp) * 16;
    const int head = blockIdx.y, m0 = (int)blockIdx.z * 8 * NT;
    const __nv_bfloat16* w0 = (const __nv_bfloat16*)p.w + head * p.wh + (long long)(n0 + r4) * p.ldw;
    const __nv_bfloat16* w1 = w0 + 8 * p.ldw;
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.x + head * p.xh;
    const bool has0 = n0 + r4 < p.N, has1 = n0 + r4 + 8 < p.N;
    const uint4 z = make_uint4(0u, 0u, 0u, 0u);
    uint4 a[U], b[U];
    auto fetch = [&](int k) {
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int kk = k + i * 32 * ks + q8;
            a[i] = has0 && kk < p.K ? __ldg(reinterpret_cast<const uint4*>(w0 + kk)) : z;
            b[i] = has1 && kk < p.K ? __ldg(reinterpret_cast<const uint4*>(w1 + kk)) : z;
        }
    };
    int k = kw * 32;
    fetch(k);                          // weights do not depend on the previous kernel
    pdl_launch_dependents();
    pdl_wait();
    float acc[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
    auto mma = [&](float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
        asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                     : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
    };
    while (k < p.K) {
        uint4 xv[U][NT];
#pragma unroll
        for (int i = 0; i < U; ++i)
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                const int kk = k + i * 32 * ks + q8, m = m0 + t * 8 + r4;
                xv[i][t] = m < p.M && kk < p.K ? *reinterpret_cast<const uint4*>(x + (long long)m * p.ldx + kk) : z;
            }
#pragma unroll
        for (int i = 0; i < U; ++i)
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                mma(acc[t], a[i].x, b[i].x, a[i].y, b[i].y, xv[i][t].x, xv[i][t].y);
                mma(acc[t], a[i].z, b[i].z, a[i].w, b[i].w, xv[i][t].z, xv[i][t].w);
            }
        k += U * 32 * ks;
        if (k < p.K) fetch(k);
    }
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) part[warp][r4 + (e >> 1) * 8][t * 8 + (lane & 3) * 2 + (e & 1)] = acc[t][e];
    __syncthreads();
    for (int e = threadIdx.x; e < groups * 16 * 8 * NT; e += 256) {
        const int g = e / (16 * 8 * NT), r = e % 16, m = (e / 16) % (8 * NT), n = ((int)blockIdx.x * groups + g) * 16 + r;
        if (m0 + m >= p.M || n >= p.N) continue;
        float v = 0.f;
        for (int i = 0; i < ks; ++i) v += part[g * ks + i][r][m];
        if (p.act == ACT_GLU_GELU) {
            if (r & 1) continue;
            float u = 0.f;
            for (int i = 0; i < ks; ++i) u += part[g * ks + i][r + 1][m];
            put<__nv_bfloat16, TO>(p, head, m0 + m, n >> 1, gelu_tanh_f(v) * u);
            continue;
        }
        if (p.bias) v += to_f(((const __nv_bfloat16*)p.bias)[n]);
        put<__nv_bfloat16, TO>(p, head, m0 + m, n, activate(v, p.act));
    }
}

template <typename T, typename TO>
__global__ void __launch_bounds__(256)
linear_tile_kernel(const LinParams p) {
    __shared__ float sx[16][64 + 4], sw[16][64 + 4];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, head = blockIdx.z;
    const T* x = (const T*)p.x + head * p.xh;
    const T* w = (const T*)p.w + head * p.wh;
    pdl_launch_dependents();
    pdl_wait();
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = tid + i * 256, r = e >> 4, kk = e & 15, k = k0 + kk;
            sx[kk][r] = (m0 + r < p.M && k < p.K) ? to_f(x[(long long)(m0 + r) * p.ldx + k]) : 0.f;
            sw[kk][r] = (n0 + r < p.N && k < p.K) ? to_f(w[(long long)(n0 + r) * p.ldw + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 16; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = sx[kk][ty * 4 + i]; b[i] = sw[kk][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= p.M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= p.N) continue;
            if (p.act == ACT_GLU_GELU) {
                if (j & 1) continue;
                put<T, TO>(p, head, m, n >> 1, gelu_tanh_f(acc[i][j]) * acc[i][j + 1 < 4 ? j + 1 : 3]);
                continue;
            }
            float v = acc[i][j];
            if (p.bias) v += to_f(((const T*)p.bias)[n]);
            put<T, TO>(p, head, m, n, activate(v, p.act));
        }
    }
}

template <typename T, typename TO>
int launch_rows(const LinParams& p, int heads, cudaStream_t stream) {
    const int groups = (p.N + 1) / 2, chunks = p.K >> 3;
    int ks = 1;   // more warps per row pair until the launch has about 24 warps per SM or a warp has less than one batch of loads
    while (ks < 8 && (long long)groups * heads * ks < 24ll * seq_sm_count() && chunks > 32 * ks) ks *= 2;
    const dim3 grid((groups + 8 / ks - 1) / (8 / ks), heads);
    if (p.M == 1) PLZ_LAUNCH_CHAIN((linear_rows_kernel<T, TO, 1>), grid, dim3(256), 0, stream, p, ks);
    else if (p.M <= 4) PLZ_LAUNCH_CHAIN((linear_rows_kernel<T, TO, 4>), grid, dim3(256), 0, stream, p, ks);
    else PLZ_LAUNCH_CHAIN((linear_rows_kernel<T, TO, 8>), grid, dim3(256), 0, stream, p, ks);
    return PLZ_OK;
}
template <typename TO>
int launch_skinny(const LinParams& p, int heads, cudaStream_t stream) {
    const int tiles = (p.N + 15) / 16;
    const int per = p.M <= 8 ? 8 : 16, groups = (p.M + per - 1) / per;
    int ks = 1;
    while (ks < 8 && (long long)tiles * heads * groups * ks < 16ll * seq_sm_count() && p.K > 128 * ks) ks *= 2;
    const dim3 grid((tiles + 8 / ks - 1) / (8 / ks), heads, groups);
    if (p.M <= 8) PLZ_LAUNCH_CHAIN((linear_skinny_kernel<TO, 1>), grid, dim3(256), 0, stream, p, ks);
    else PLZ_LAUNCH_CHAIN((linear_skinny_kernel<TO, 2>), grid, dim3(256), 0, stream, p, ks);
    return PLZ_OK;
}
template <typename T, typename TO>
int launch_tile(const LinParams& p, int heads, cudaStream_t stream) {
    const long long my = (p.M + 63) / 64;
    if (my > 65535) { set_last_error("linear: too many rows"); return PLZ_ERR_TOO_LARGE; }
    PLZ_LAUNCH_CHAIN((linear_tile_kernel<T, TO>), dim3((p.N + 63) / 64, (unsigned)my, heads), dim3(256), 0, stream, p);
    return PLZ_OK;
}

}  // namespace

int launch_seq_linear(int dtype, const void* x, long long ldx, int M, int K, const void* w, long long ldw, int N, const void* bias, int act,
                      void* y, long long ldy, int y_f32, cudaStream_t stream) {
    if (M <= 0) return PLZ_OK;
    if (N <= 0 || K <= 0 || act < 0 || act > ACT_GLU_GELU || (act == ACT_GLU_GELU && (N % 2 || bias))) {
        set_last_error("linear: bad shape M=%d N=%d K=%d act=%d", M, N, K, act); return PLZ_ERR_BAD_SHAPE;
    }
    if (!x || !w || !y) { set_last_error("linear: null pointer"); return PLZ_ERR_NULL; }
    LinParams p = {};
    p.x = x; p.ldx = ldx; p.w = w; p.ldw = ldw; p.bias = bias; p.y = y; p.ldy = ldy; p.M = M; p.N = N; p.K = K; p.act = act;
    const int per16 = dtype == 0 ? 8 : 4;
    const bool vec = K % 8 == 0 && ldx % per16 == 0 && ldw % per16 == 0 && !((uintptr_t)x & 15) && !((uintptr_t)w & 15);
    if (dtype == 0 && M > 1 && M <= 16 && vec) return y_f32 ? launch_skinny<float>(p, 1, stream) : launch_skinny<__nv_bfloat16>(p, 1, stream);
    if (M <= 8 && vec) {
        if (dtype == 1) return launch_rows<float, float>(p, 1, stream);
        return y_f32 ? launch_rows<__nv_bfloat16, float>(p, 1, stream) : launch_rows<__nv_bfloat16, __nv_bfloat16>(p, 1, stream);
    }
    const int out_cols = act == ACT_GLU_GELU ? N / 2 : N;
    if (dtype == 0 && !y_f32 && vec && N % 8 == 0 && out_cols % 8 == 0 && ldy % 8 == 0 && !((uintptr_t)y & 15) && !((uintptr_t)bias & 15)) {
        LutGemmArgs g = {};
        g.bmode = B_TMA_K; g.M = M; g.J = N; g.R = K;
        g.A = x; g.lda = ldx; g.Bdense = w; g.ldb = ldw;
        g.bias = bias; g.act = act; g.fuse = act == ACT_GLU_GELU ? 4 : ((bias || act) ? 3 : 0);
        g.out = y; g.ld_out = ldy; g.alpha = 1.0f;
        return launch_lut_gemm(g, stream);
    }
    if (dtype == 1) return launch_tile<float, float>(p, 1, stream);
    return y_f32 ? launch_tile<__nv_bfloat16, float>(p, 1, stream) : launch_tile<__nv_bfloat16, __nv_bfloat16>(p, 1, stream);
}

// one small product per head: y[m, h, :] = x[m, h, :] W_h^T
int launch_head_linear(int dtype, const HeadLinearArgs& a, cudaStream_t stream) {
    if (a.M <= 0) return PLZ_OK;
    LinParams p = {};
    p.x = a.x; p.ldx = a.ldx; p.xh = a.xh; p.w = a.w; p.ldw = a.K; p.wh = (long long)a.N * a.K; p.y = a.y; p.ldy = a.ldy; p.yh = a.yh;
    p.M = a.M; p.N = a.N; p.K = a.K; p.gate = a.gate; p.ldg = a.ldg; p.gh = a.N;
    const int per16 = dtype == 0 ? 8 : 4;
    const bool vec = a.K % 8 == 0 && a.ldx % per16 == 0 && a.xh % per16 == 0 && !((uintptr_t)a.x & 15) && !((uintptr_t)a.w & 15);
    if (vec && dtype == 0 && a.M > 1) return launch_skinny<__nv_bfloat16>(p, a.H, stream);
    if (vec && a.M <= 8) return dtype == 1 ? launch_rows<float, float>(p, a.H, stream) : launch_rows<__nv_bfloat16, __nv_bfloat16>(p, a.H, stream);
    return dtype == 1 ? launch_tile<float, float>(p, a.H, stream) : launch_tile<__nv_bfloat16, __nv_bfloat16>(p, a.H, stream);
}

}  // namespace plz
