// Attention whose keys and values are both the cached latent (the key and value matrices are folded into the queries and the output):
// every head of a token reads the same row c [R] | kr [dr] of a cached token, score = q . [c | kr] * scale, and the output is a weighted
// sum of c. A query row is one (token, head) pair; rows of a sequence are numbered t * H + h.
//
//   latent_rows_kernel      the CUDA-core form: fp32 products for both types, any size up to R = 1024. It is the 32-bit mode and serves
//                           bf16 sizes outside the tensor-core kernel's range (latent_attention_tc.cu).
//   latent_combine_kernel   merges the key splits of either form and adds the sink.
#include "latent_attention.cuh"

namespace plz {
namespace {

constexpr int kRows = 8, kKeys = 32;

struct RowsParams {
    LatentParams l;
    const void* q; long long ldq;
    const void* c; const void* kr; long long c_batch, r_batch;
    const int* pos;
};

// Block: 8 query rows, one key split, 128 threads. Scores: thread = (row, 2 of 32 keys); weighted sum: thread = RT latent columns.
template <typename T, int RT>
__global__ void __launch_bounds__(128)
latent_rows_kernel(const RowsParams p) {
    extern __shared__ float sm[];
    const int R = p.l.R, dr = p.l.dr, D = R + dr, pk = D | 1;
    float* sQ = sm;                       // [kRows][D]
    float* sC = sQ + kRows * D;           // [kKeys][pk]
    float* sP = sC + kKeys * pk;          // [kRows][kKeys]
    float* sA = sP + kRows * kKeys;       // [kRows] correction of the running sums
    const int tid = threadIdx.x, rr = tid >> 4, kk = tid & 15;
    const int r0 = (int)blockIdx.y * kRows, rows = p.l.n * p.l.H;
    const long long b = blockIdx.z;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *p.pos;
    for (int e = tid; e < kRows * D; e += 128) {
        const int r = e / D, c = e - r * D, g = r0 + r;
        sQ[e] = g < rows ? to_f(((const T*)p.q)[(b * p.l.n + g / p.l.H) * p.ldq + (long long)(g % p.l.H) * D + c]) : 0.f;
    }
    const int my_last = r0 + rr < rows ? pos + (r0 + rr) / p.l.H : -1;        // last key this thread's row sees
    const int last = pos + (min(rows, r0 + kRows) - 1) / p.l.H;
    const int total = last + 1;
    int chunk = (total + p.l.splits - 1) / p.l.splits;
    chunk = (chunk + kKeys - 1) / kKeys * kKeys;
    const int k0 = (int)blockIdx.x * chunk, k1 = min(total, k0 + chunk);
    float m = kLatNegBig, l = 0.f;
    float acc[kRows][RT];
#pragma unroll
    for (int r = 0; r < kRows; ++r)
#pragma unroll
        for (int i = 0; i < RT; ++i) acc[r][i] = 0.f;
    for (int j0 = k0; j0 < k1; j0 += kKeys) {
        __syncthreads();
        for (int e = tid; e < kKeys * D; e += 128) {
            const int r = e / D, c = e - r * D, j = j0 + r;
            float v = 0.f;
            if (j < k1) v = to_f(c < R ? ((const T*)p.c)[b * p.c_batch + (long long)j * R + c] : ((const T*)p.kr)[b * p.r_batch + (long long)j * dr + c - R]);
            sC[r * pk + c] = v;
        }
        __syncthreads();
        float s0 = 0.f, s1 = 0.f;
        for (int c = 0; c < D; ++c) {
            const float qv = sQ[rr * D + c];
            s0 = fmaf(qv, sC[kk * pk + c], s0);
            s1 = fmaf(qv, sC[(kk + 16) * pk + c], s1);
        }
        const bool in0 = j0 + kk < k1 && j0 + kk <= my_last, in1 = j0 + kk + 16 < k1 && j0 + kk + 16 <= my_last;
        s0 = in0 ? s0 * p.l.scale : kLatNegBig;
        s1 = in1 ? s1 * p.l.scale : kLatNegBig;
        float mt = fmaxf(s0, s1);
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xFFFFFFFFu, mt, o));
        const float mn = fmaxf(m, mt), corr = expf(m - mn);
        const float e0 = in0 ? expf(s0 - mn) : 0.f, e1 = in1 ? expf(s1 - mn) : 0.f;
        float ls = e0 + e1;
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) ls += __shfl_xor_sync(0xFFFFFFFFu, ls, o);
        l = l * corr + ls;
        m = mn;
        sP[rr * kKeys + kk] = e0;
        sP[rr * kKeys + kk + 16] = e1;
        if (kk == 0) sA[rr] = corr;
        __syncthreads();
#pragma unroll
        for (int r = 0; r < kRows; ++r) {
            const float a = sA[r];
#pragma unroll
            for (int i = 0; i < RT; ++i) acc[r][i] *= a;
        }
        for (int j = 0; j < kKeys; ++j) {
#pragma unroll
            for (int i = 0; i < RT; ++i) {
                const int c = tid + i * 128;
                const float cv = c < R ? sC[j * pk + c] : 0.f;
#pragma unroll
                for (int r = 0; r < kRows; ++r) acc[r][i] = fmaf(sP[r * kKeys + j], cv, acc[r][i]);
            }
        }
    }
    if (kk == 0 && r0 + rr < rows) {
        const long long slot = (b * rows + r0 + rr) * p.l.splits + blockIdx.x;
        p.l.ws_ml[slot * 2] = m * kLatLog2e;
        p.l.ws_ml[slot * 2 + 1] = l;
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        if (r0 + r >= rows) break;
        float* dst = p.l.ws_o + ((b * rows + r0 + r) * p.l.splits + blockIdx.x) * R;
#pragma unroll
        for (int i = 0; i < RT; ++i) {
            const int c = tid + i * 128;
            if (c < R) dst[c] = acc[r][i];
        }
    }
}

// One block per query row and 32 * V latent columns, V per lane; the four warps share the splits. Weights exp2(m_s - M) of the splits
// once. A split without keys has weight 0 and was not written: the first one, which always has some, is read in its place.
template <typename T, int V>
__global__ void __launch_bounds__(128)
latent_combine_kernel(const LatentParams p, T* __restrict__ o, long long ldo) {
    __shared__ float wgt[kLatMaxSplits];
    __shared__ float red[8];
    __shared__ float sum[4][32 * V];
    const long long row = blockIdx.x;                       // b * n * H + t * H + h
    const int h = (int)(row % p.H), t = threadIdx.x, lane = t & 31, w = t >> 5;
    pdl_launch_dependents();
    const float sink = p.sinks ? p.sinks[h] * kLatLog2e : kLatNegBig;
    pdl_wait();
    const float2 ml = t < p.splits ? *reinterpret_cast<const float2*>(p.ws_ml + (row * p.splits + t) * 2) : make_float2(kLatNegBig, 0.f);
    float M = fmaxf(ml.x, sink);
#pragma unroll
    for (int i = 16; i > 0; i >>= 1) M = fmaxf(M, __shfl_xor_sync(0xFFFFFFFFu, M, i));
    if (lane == 0) red[w] = M;
    __syncthreads();
    M = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    const float c = ml.y > 0.f ? exp2f(ml.x - M) : 0.f;
    wgt[t] = c;
    float ls = c * ml.y;
#pragma unroll
    for (int i = 16; i > 0; i >>= 1) ls += __shfl_xor_sync(0xFFFFFFFFu, ls, i);
    if (lane == 0) red[4 + w] = ls;
    __syncthreads();
    const float L = red[4] + red[5] + red[6] + red[7] + (p.sinks ? exp2f(sink - M) : 0.f);
    const float inv = L > 0.f ? 1.0f / L : 0.f;
    const int d = ((int)blockIdx.y * 32 + lane) * V;
    float acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = 0.f;
    if (d < p.R) {
        const float* src = p.ws_o + row * p.splits * p.R + d;
#pragma unroll 8
        for (int s = w; s < p.splits; s += 4) {
            const float f = wgt[s];
            const float* q = src + (f > 0.f ? (long long)s * p.R : 0ll);
            if (V == 4) {
                const float4 v = __ldcs(reinterpret_cast<const float4*>(q));
                acc[0] = fmaf(f, v.x, acc[0]); acc[1 % V] = fmaf(f, v.y, acc[1 % V]); acc[2 % V] = fmaf(f, v.z, acc[2 % V]); acc[3 % V] = fmaf(f, v.w, acc[3 % V]);
            } else {
                acc[0] = fmaf(f, __ldcs(q), acc[0]);
            }
        }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) sum[w][lane * V + e] = acc[e];
    __syncthreads();
    const int col = (int)blockIdx.y * 32 * V + t;
    if (t < 32 * V && col < p.R)
        o[(row / p.H) * ldo + (long long)h * p.R + col] = from_f<T>((sum[0][t] + sum[1][t] + sum[2][t] + sum[3][t]) * inv);
}

template <typename T>
int launch_combine(const LatentParams& l, long long rows, void* o, long long ldo, cudaStream_t stream) {
    const int V = l.R % 4 == 0 ? 4 : 1;
    const dim3 grid((unsigned)rows, (l.R + 32 * V - 1) / (32 * V));
    if (V == 4) PLZ_LAUNCH_CHAIN((latent_combine_kernel<T, 4>), grid, dim3(128), 0, stream, l, (T*)o, ldo);
    else PLZ_LAUNCH_CHAIN((latent_combine_kernel<T, 1>), grid, dim3(128), 0, stream, l, (T*)o, ldo);
    return PLZ_OK;
}

template <typename T, int RT>
int launch_rows_t(const RowsParams& p, dim3 grid, size_t smem, cudaStream_t stream) {
    auto kern = latent_rows_kernel<T, RT>;
    PLZ_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    PLZ_LAUNCH_CHAIN(kern, grid, dim3(128), smem, stream, p);
    return PLZ_OK;
}
template <typename T>
int launch_rows(const RowsParams& p, int B, cudaStream_t stream) {
    const int R = p.l.R, D = R + p.l.dr, rows = p.l.n * p.l.H;
    const size_t smem = (size_t)(kRows * D + kKeys * (D | 1) + kRows * kKeys + kRows) * sizeof(float);
    if (R > 1024 || smem > 220 * 1024) { set_last_error("latent attention: latent of %d + %d columns", R, p.l.dr); return PLZ_ERR_UNSUPPORTED; }
    const long long gy = (rows + kRows - 1) / kRows;
    if (gy > 65535) { set_last_error("latent attention: %d query rows", rows); return PLZ_ERR_TOO_LARGE; }
    const dim3 grid(p.l.splits, (unsigned)gy, B);
    if (R <= 128) return launch_rows_t<T, 1>(p, grid, smem, stream);
    if (R <= 256) return launch_rows_t<T, 2>(p, grid, smem, stream);
    if (R <= 512) return launch_rows_t<T, 4>(p, grid, smem, stream);
    return launch_rows_t<T, 8>(p, grid, smem, stream);
}

bool on_tensor_cores(int dtype, int R, int dr) { return dtype == 0 && latent_tc_fits(R, dr); }

// key splits of a launch over a cache of `cap` positions whose length may be known on the device only
int plan_splits(int dtype, int B, int n, int H, int R, int dr, int cap) {
    const bool tc = on_tensor_cores(dtype, R, dr);
    const int rows = n * H, step = tc ? kLatTile : kKeys, per = tc ? latent_tc_rows(rows, R, dr) : kRows;
    const long long groups = (long long)B * ((rows + per - 1) / per);
    const int tiles = (cap + step - 1) / step, sms = seq_sm_count(), most = tiles < kLatMaxSplits ? tiles : kLatMaxSplits;
    const long long slots = tc ? sms : 2ll * sms;        // CTAs at once
    // waves of CTAs times the tiles of each, one more tile's time for start and end
    int best = 1;
    long long best_cost = -1;
    for (int s = 1; s <= most; ++s) {
        const long long cost = ((groups * s + slots - 1) / slots) * ((tiles + s - 1) / s + 1);
        if (best_cost < 0 || cost < best_cost) { best = s; best_cost = cost; }
    }
    return best;
}

}  // namespace

long long latent_attn_ws_bytes(int dtype, int B, int n, int H, int R, int dr, int cap) {
    const long long slots = (long long)B * n * H * plan_splits(dtype, B, n, H, R, dr, cap);
    return ((slots * 2 + 3) / 4 * 4 + slots * R) * (long long)sizeof(float);
}

int launch_latent_attn(int dtype, const LatentAttnArgs& a, void* ws, long long ws_bytes, cudaStream_t stream) {
    const long long need = latent_attn_ws_bytes(dtype, a.B, a.n, a.H, a.R, a.dr, a.cap);
    if (!ws || ws_bytes < need) { set_last_error("latent attention: workspace of %lld bytes needed, %lld given", need, ws_bytes); return PLZ_ERR_TOO_LARGE; }
    LatentParams l = {};
    l.n = a.n; l.H = a.H; l.R = a.R; l.dr = a.dr; l.scale = a.scale; l.sinks = a.sinks;
    l.splits = plan_splits(dtype, a.B, a.n, a.H, a.R, a.dr, a.cap);
    const long long rows = (long long)a.B * a.n * a.H;
    l.ws_ml = (float*)ws;
    l.ws_o = l.ws_ml + (rows * l.splits * 2 + 3) / 4 * 4;
    int rc;
    const bool aligned = a.scale > 0.f && a.ldq % 8 == 0 && a.c_batch % 8 == 0 && a.r_batch % 8 == 0 && !((uintptr_t)a.q & 15) && !((uintptr_t)a.c & 15) && !((uintptr_t)a.kr & 15);
    if (on_tensor_cores(dtype, a.R, a.dr) && aligned) {
        rc = launch_latent_tc(a, l, stream);
    } else {
        RowsParams p = {};
        p.l = l; p.q = a.q; p.ldq = a.ldq; p.c = a.c; p.kr = a.kr; p.c_batch = a.c_batch; p.r_batch = a.r_batch; p.pos = a.pos;
        rc = dtype == 1 ? launch_rows<float>(p, a.B, stream) : launch_rows<__nv_bfloat16>(p, a.B, stream);
    }
    if (rc) return rc;
    return dtype == 1 ? launch_combine<float>(l, rows, a.o, a.ldo, stream) : launch_combine<__nv_bfloat16>(l, rows, a.o, a.ldo, stream);
}

}  // namespace plz
