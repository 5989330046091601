// Causal attention with a per-head bias by distance and a sink, against the key / value cache, on the CUDA cores: fp32 products
// and softmax for both types and any head sizes. It is the 32-bit mode, and serves bf16 head sizes outside the tensor-core kernel's
// range.  score(i, j) = q_i . k_j * scale + bias[h][i - j];  with a sink, the denominator starts at exp(its score).  The last key
// columns may come from a second tensor shared by all heads; the output may be multiplied by sigmoid(gate).
//
// Block = 32 queries of one head, 128 threads: thread = (query, one of four key slices). Keys and values pass through shared memory
// 32 at a time.
#include "seq_math.cuh"

namespace plz {
namespace {

constexpr int kQ = 32, kK = 32;

struct BiasParams {
    const void* q; long long ldq;                              // [B * n, H * dk]
    const void* k; const void* v; long long k_batch, v_batch;  // caches [B, T, G * dk], [B, T, G * dv]
    void* o; long long ldo;
    const float* bias; long long ldb; int n_bias;              // [H, ldb], entry d: bias at distance d, the last one for all beyond; or null
    const int* pos;
    int n, H, G, dk, dv, sink;
    float scale;
    const float* sinks;
    long long k_tok, v_tok;
    const void* k2; long long k2_batch; int dk2;               // [B, T, dk2]
    const void* gate; long long ldg;
};

template <typename T, int DVT>   // DVT: value columns per thread (dv <= 4 * DVT)
__global__ void __launch_bounds__(128)
attn_bias_kernel(const BiasParams p) {
    extern __shared__ float sm[];
    const int pk = p.dk + 1;
    float* sQ = sm;                          // [kQ][pk]
    float* sK = sQ + kQ * pk;                // [kK][pk]
    float* sV = sK + kK * pk;                // [kK][dv]
    float* sP = sV + kK * p.dv;              // [kQ][kK + 1]
    const int tid = threadIdx.x, qi = tid >> 2, sl = tid & 3;
    const int h = blockIdx.y, hk = h / (p.H / p.G);
    const long long b = blockIdx.z;
    const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kQ;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *p.pos;
    for (int e = tid; e < kQ * p.dk; e += 128) {
        const int r = e / p.dk, c = e - r * p.dk;
        sQ[r * pk + c] = q0 + r < p.n ? to_f(((const T*)p.q)[(b * p.n + q0 + r) * p.ldq + (long long)h * p.dk + c]) : 0.f;
    }
    const int i = pos + q0 + qi;                                   // absolute position of this thread's query
    const int last = pos + min(p.n, q0 + kQ) - 1;                  // largest key any query of the block sees
    const int dk1 = p.dk - p.dk2;
    float m = p.sink ? (p.sinks ? p.sinks[h] : 0.f) : -INFINITY, l = p.sink ? 1.f : 0.f;
    float acc[DVT];
#pragma unroll
    for (int d = 0; d < DVT; ++d) acc[d] = 0.f;
    const float* brow = p.bias ? p.bias + (long long)h * p.ldb : nullptr;
    for (int j0 = 0; j0 <= last; j0 += kK) {
        __syncthreads();
        for (int e = tid; e < kK * p.dk; e += 128) {
            const int r = e / p.dk, c = e - r * p.dk;
            float v = 0.f;
            if (j0 + r <= last)
                v = to_f(c < dk1 ? ((const T*)p.k)[b * p.k_batch + (j0 + r) * p.k_tok + hk * dk1 + c]
                                 : ((const T*)p.k2)[b * p.k2_batch + (long long)(j0 + r) * p.dk2 + c - dk1]);
            sK[r * pk + c] = v;
        }
        for (int e = tid; e < kK * p.dv; e += 128) {
            const int r = e / p.dv, c = e - r * p.dv;
            sV[e] = j0 + r <= last ? to_f(((const T*)p.v)[b * p.v_batch + (j0 + r) * p.v_tok + hk * p.dv + c]) : 0.f;
        }
        __syncthreads();
        float s[8];
        float mt = -INFINITY;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int j = sl + 4 * u;
            float d = 0.f;
            for (int c = 0; c < p.dk; ++c) d = fmaf(sQ[qi * pk + c], sK[j * pk + c], d);
            d *= p.scale;
            const int dist = i - (j0 + j);
            if (dist >= 0) { if (brow) d += brow[min(dist, p.n_bias - 1)]; }
            else d = -INFINITY;
            s[u] = d;
            mt = fmaxf(mt, d);
        }
        mt = fmaxf(mt, __shfl_xor_sync(0xFFFFFFFFu, mt, 1));
        mt = fmaxf(mt, __shfl_xor_sync(0xFFFFFFFFu, mt, 2));
        const float mn = fmaxf(m, mt);
        const float corr = m == -INFINITY ? 0.f : expf(m - mn);
        float ls = 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const float e = s[u] == -INFINITY ? 0.f : expf(s[u] - mn);
            sP[qi * (kK + 1) + sl + 4 * u] = e;
            ls += e;
        }
        ls += __shfl_xor_sync(0xFFFFFFFFu, ls, 1);
        ls += __shfl_xor_sync(0xFFFFFFFFu, ls, 2);
        l = l * corr + ls;
        m = mn;
        __syncwarp();
#pragma unroll
        for (int d = 0; d < DVT; ++d) acc[d] *= corr;
        for (int j = 0; j < kK; ++j) {
            const float e = sP[qi * (kK + 1) + j];
#pragma unroll
            for (int d = 0; d < DVT; ++d) {
                const int c = sl + 4 * d;
                if (c < p.dv) acc[d] = fmaf(e, sV[j * p.dv + c], acc[d]);
            }
        }
        __syncwarp();
    }
    if (q0 + qi < p.n) {
        const float inv = l > 0.f ? 1.0f / l : 0.f;
        T* dst = (T*)p.o + (b * p.n + q0 + qi) * p.ldo + (long long)h * p.dv;
        const T* gate = p.gate ? (const T*)p.gate + (b * p.n + q0 + qi) * p.ldg + (long long)h * p.dv : nullptr;
#pragma unroll
        for (int d = 0; d < DVT; ++d) {
            const int c = sl + 4 * d;
            if (c < p.dv) dst[c] = from_f<T>(acc[d] * inv * (gate ? sigmoid_f(to_f(gate[c])) : 1.f));
        }
    }
}

template <typename T, int DVT>
int launch_b(const BiasParams& p, int B, cudaStream_t stream) {
    const size_t smem = (size_t)((kQ + kK) * (p.dk + 1) + kK * p.dv + kQ * (kK + 1)) * sizeof(float);
    auto kern = attn_bias_kernel<T, DVT>;
    PLZ_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    PLZ_LAUNCH_CHAIN(kern, dim3((p.n + kQ - 1) / kQ, p.H, B), dim3(128), smem, stream, p);
    return PLZ_OK;
}
template <typename T>
int launch_any(const BiasParams& p, int B, cudaStream_t stream) {
    if (p.dk > 512) { set_last_error("attention: query / key size %d (at most 512)", p.dk); return PLZ_ERR_UNSUPPORTED; }
    if (p.dv <= 64) return launch_b<T, 16>(p, B, stream);
    if (p.dv <= 128) return launch_b<T, 32>(p, B, stream);
    if (p.dv <= 256) return launch_b<T, 64>(p, B, stream);
    set_last_error("attention: value size %d (at most 256)", p.dv);
    return PLZ_ERR_UNSUPPORTED;
}

}  // namespace

int launch_attn_bias_simt(int dtype, const AttnBiasArgs& a, cudaStream_t stream) {
    if (a.B <= 0 || a.n <= 0) return PLZ_OK;
    BiasParams p = {};
    p.q = a.q; p.ldq = a.ldq; p.k = a.k; p.v = a.v; p.k_batch = a.k_batch; p.v_batch = a.v_batch; p.o = a.o; p.ldo = a.ldo;
    p.bias = a.bias; p.ldb = a.ldb; p.n_bias = a.n_bias; p.pos = a.pos;
    p.n = a.n; p.H = a.H; p.G = a.G; p.dk = a.dk; p.dv = a.dv; p.sink = a.sink || a.sinks; p.scale = a.scale;
    p.sinks = a.sinks; p.k_tok = a.k_tok; p.v_tok = a.v_tok; p.k2 = a.k2; p.k2_batch = a.k2_batch; p.dk2 = a.dk2; p.gate = a.gate; p.ldg = a.ldg;
    return dtype == 1 ? launch_any<float>(p, a.B, stream) : launch_any<__nv_bfloat16>(p, a.B, stream);
}

}  // namespace plz
