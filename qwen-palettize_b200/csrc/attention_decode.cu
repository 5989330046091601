// Attention of one new token per sequence against a key / value cache (token decode), and the embedding-row gather that
// opens a forward pass. Both are single passes bound by HBM: a decode step reads every cached key and value once
// (B * T * Hkv * 128 * 2 * 2 bytes per layer), no tensor core involved.
//
//   attn_decode_partial_kernel  grid (splits, Hkv, B), 4 warps. The sequence is cut into `splits` contiguous chunks so that
//     the launch has a few CTAs per SM whatever B is. Inside a CTA a warp takes 8 tokens per step: 16 lanes per token, each
//     lane the 16 bytes (8 dims) of the key and of the value row that belong to it, so one load instruction of a warp covers
//     two whole 256-byte rows, and four such loads for K and four for V are in flight per lane before anything is used. The
//     up-to-4 query heads of the group share every key / value byte. The 16 partial scores of a step (4 heads x 4 token
//     slots) are summed over the 16 lanes by recursive halving (15 shuffles, after which lane i owns score i), so exp2 is
//     evaluated once per score; online softmax (running max and sum per head) across steps; the warps' partial results meet in
//     shared memory. With one split the CTA writes the bf16 output itself, else an unnormalised fp32 partial (o, max, sum).
//   attn_decode_combine_kernel  merges the splits.
//
// Template parameters widen it: element type (bf16, fp32), lanes per token (8, 16, 32: head sizes up to 64, 128, 256, key and value
// sizes independent), and EXT, which takes the length from device memory (a captured step replays at any position), adds a bias by
// distance to the scores and a sink (score 0, no value) to the denominator.
//
// The reference has no attention code (it calls the HuggingFace layer, scripts/qwen_model.py:454 selects SDPA); semantics are
// those of transformers' Qwen3Attention at q_len = 1 with a DynamicCache: softmax over all T cached positions, no mask.
#include "plz_launch.h"

namespace plz {
namespace {

constexpr float kLog2eDec = 1.4426950408889634f;
constexpr float kNegBig = -1.0e30f;
constexpr int kDecWarps = 4;
constexpr int kStepTokens = 8;                     // tokens of one warp step
constexpr int kCtaStep = kDecWarps * kStepTokens;  // tokens a CTA advances per step of its warps
constexpr int kMaxSplits = 128;

struct DecParams {
    const void* q; long long ldq;
    const void* k; const void* v; long long k_batch, v_batch, k_tok, v_tok;   // elements between sequences / positions
    void* out; long long ldo;
    float* ws_o; float* ws_ml;       // [B, Hq, splits, dv] and [B, Hq, splits, 2]
    int T, Hq, Hkv, chunk, splits;
    int group, passes;                       // Hq / Hkv; launches of up to four query heads of a group, side by side in the grid
    float scale_log2e;
    // EXT only: head sizes, device-side length, bias by distance, sink
    int dk, dv;
    const int* pos;                          // the new token's position; T = *pos + 1
    const float* bias; long long ldb; int n_bias;
    int sink;
};

__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// eight consecutive cached elements of a lane
template <typename T> struct Chunk;
template <> struct Chunk<__nv_bfloat16> {
    uint4 r;
    __device__ __forceinline__ void zero() { r = make_uint4(0u, 0u, 0u, 0u); }
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { r = __ldcs(reinterpret_cast<const uint4*>(p)); }
    __device__ __forceinline__ void unpack(float (&f)[8]) const {
        const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u); }
    }
};
template <> struct Chunk<float> {
    float4 a, b;
    __device__ __forceinline__ void zero() { a = make_float4(0.f, 0.f, 0.f, 0.f); b = a; }
    __device__ __forceinline__ void load(const float* p) { a = __ldcs(reinterpret_cast<const float4*>(p)); b = __ldcs(reinterpret_cast<const float4*>(p + 4)); }
    __device__ __forceinline__ void unpack(float (&f)[8]) const {
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    }
};
__device__ __forceinline__ void store_elem(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_elem(float* p, float v) { *p = v; }

// T: element type; LPT: lanes per token (head sizes up to 8 * LPT); EXT: the head sizes, bias, sink and length of the params
template <typename T, int LPT, bool EXT>
__global__ void __launch_bounds__(kDecWarps * 32)
attn_decode_partial_kernel(const DecParams p) {
    constexpr int U = LPT / 4;                      // token groups of a step: U * (32 / LPT) = 8 tokens
    constexpr int D = 8 * LPT;
    __shared__ float sm_o[kDecWarps][4][D];
    __shared__ float sm_ml[kDecWarps][4][2];
    const int split = blockIdx.x, hk = blockIdx.y / p.passes, g0 = (blockIdx.y % p.passes) * 4, b = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tl = lane / LPT, dl = lane % LPT;
    const int G = min(4, p.group - g0);
    const int head0 = hk * p.group + g0;            // first q head of this CTA's part of the group
    const int dk = EXT ? p.dk : 128, dv = EXT ? p.dv : 128;
    const bool in_k = !EXT || dl * 8 < dk, in_v = !EXT || dl * 8 < dv;
    pdl_launch_dependents();
    pdl_wait();
    const int T_all = EXT ? *p.pos + 1 : p.T;
    int chunk = p.chunk;
    if (EXT) chunk = ((T_all + p.splits - 1) / p.splits + kCtaStep - 1) / kCtaStep * kCtaStep;
    const int t0 = split * chunk, t1 = min(T_all, t0 + chunk);

    float q[4][8];
#pragma unroll
    for (int g = 0; g < 4; ++g) {
        Chunk<T> r;
        r.zero();
        if (g < G && in_k) r.load((const T*)p.q + (long long)b * p.ldq + (long long)(head0 + g) * dk + dl * 8);
        r.unpack(q[g]);
#pragma unroll
        for (int d = 0; d < 8; ++d) q[g][d] *= p.scale_log2e;
    }
    float o[4][8];
#pragma unroll
    for (int g = 0; g < 4; ++g)
#pragma unroll
        for (int d = 0; d < 8; ++d) o[g][d] = 0.f;
    float m_own = kNegBig, l_own = 0.f;             // of head dl / U, this lane's share of the sum
    const T* kb = (const T*)p.k + (long long)b * p.k_batch + (long long)hk * dk + dl * 8;
    const T* vb = (const T*)p.v + (long long)b * p.v_batch + (long long)hk * dv + dl * 8;
    const int u_own = dl % U, g_own = dl / U;
    const float* brow = nullptr;
    if (EXT && p.bias && g_own < G) brow = p.bias + (long long)(head0 + g_own) * p.ldb;

    for (int base = t0 + warp * kStepTokens; base < t1; base += kCtaStep) {
        Chunk<T> kr[U], vr[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int t = base + (32 / LPT) * u + tl;
            kr[u].zero(); vr[u].zero();
            if (t < t1) {
                if (in_k) kr[u].load(kb + (long long)t * p.k_tok);
                if (in_v) vr[u].load(vb + (long long)t * p.v_tok);
            }
        }
        float val[LPT];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            float kf[8];
            kr[u].unpack(kf);
#pragma unroll
            for (int g = 0; g < 4; ++g) {
                float s = 0.f;
#pragma unroll
                for (int d = 0; d < 8; ++d) s = fmaf(q[g][d], kf[d], s);
                val[g * U + u] = s;
            }
        }
        // sum over the LPT lanes of a token by recursive halving: afterwards lane dl holds the total of val[dl]
#pragma unroll
        for (int half = LPT / 2; half >= 1; half >>= 1) {
            const bool up = (dl & half) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float send = up ? val[i] : val[i + half];
                const float keep = up ? val[i + half] : val[i];
                val[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, half);
            }
        }
        const int t_own = base + (32 / LPT) * u_own + tl;
        const bool ok = t_own < t1;
        float s = ok ? val[0] : kNegBig;
        if (EXT && ok && brow) s = fmaf(__ldg(brow + min(T_all - 1 - t_own, p.n_bias - 1)), kLog2eDec, s);
        float mx = s;
#pragma unroll
        for (int i = 1; i < U; i <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, i));
#pragma unroll
        for (int i = LPT; i < 32; i <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, i));
        const float m_new = fmaxf(m_own, mx);
        const float corr = ex2(m_own - m_new);
        const float pr = ok ? ex2(s - m_new) : 0.f;
        l_own = l_own * corr + pr;
        m_own = m_new;
#pragma unroll
        for (int g = 0; g < 4; ++g) {
            const float cg = __shfl_sync(0xFFFFFFFFu, corr, g * U);
#pragma unroll
            for (int d = 0; d < 8; ++d) o[g][d] *= cg;
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            float vf[8];
            vr[u].unpack(vf);
#pragma unroll
            for (int g = 0; g < 4; ++g) {
                const float pgu = __shfl_sync(0xFFFFFFFFu, pr, tl * LPT + g * U + u);
#pragma unroll
                for (int d = 0; d < 8; ++d) o[g][d] = fmaf(pgu, vf[d], o[g][d]);
            }
        }
    }
    // the token slots of a warp, then the sum of a head over its lanes
#pragma unroll
    for (int i = LPT; i < 32; i <<= 1) {
#pragma unroll
        for (int g = 0; g < 4; ++g)
#pragma unroll
            for (int d = 0; d < 8; ++d) o[g][d] += __shfl_xor_sync(0xFFFFFFFFu, o[g][d], i);
        l_own += __shfl_xor_sync(0xFFFFFFFFu, l_own, i);
    }
#pragma unroll
    for (int i = 1; i < U; i <<= 1) l_own += __shfl_xor_sync(0xFFFFFFFFu, l_own, i);
    if (tl == 0) {
#pragma unroll
        for (int g = 0; g < 4; ++g)
#pragma unroll
            for (int d = 0; d < 8; ++d) sm_o[warp][g][dl * 8 + d] = o[g][d];
        if (u_own == 0) { sm_ml[warp][g_own][0] = m_own; sm_ml[warp][g_own][1] = l_own; }
    }
    __syncthreads();
    // merge the warps: thread d takes dimension d (and d + 128) of every head
    for (int d = threadIdx.x; d < dv; d += kDecWarps * 32) {
        for (int g = 0; g < G; ++g) {
            float M = kNegBig;
#pragma unroll
            for (int w = 0; w < kDecWarps; ++w) M = fmaxf(M, sm_ml[w][g][0]);
            const bool sink = EXT && p.sink && p.splits == 1;
            if (sink) M = fmaxf(M, 0.f);
            float acc = 0.f, l = sink ? ex2(-M) : 0.f;
#pragma unroll
            for (int w = 0; w < kDecWarps; ++w) {
                const float c = ex2(sm_ml[w][g][0] - M);
                acc = fmaf(c, sm_o[w][g][d], acc);
                l = fmaf(c, sm_ml[w][g][1], l);
            }
            const int head = head0 + g;
            if (p.splits == 1) {
                store_elem((T*)p.out + (long long)b * p.ldo + (long long)head * dv + d, l > 0.f ? acc / l : 0.f);
            } else {
                const long long slot = ((long long)b * p.Hq + head) * p.splits + split;
                p.ws_o[slot * dv + d] = acc;
                if (d == 0) { p.ws_ml[slot * 2] = M; p.ws_ml[slot * 2 + 1] = l; }
            }
        }
    }
}

// Merge of the splits: one block per (head, sequence), thread d = dimension d (and d + 128). The weights exp2(m_s - M) of the
// splits are computed once (thread s for split s, at most kMaxSplits of them) and shared; the sum over splits then has
// independent loads.
template <typename T>
__global__ void __launch_bounds__(128)
attn_decode_combine_kernel(const float* __restrict__ ws_o, const float* __restrict__ ws_ml, int splits, int Hq, int dv, int sink,
                           T* __restrict__ out, long long ldo) {
    __shared__ float wgt[kMaxSplits];
    __shared__ float red[8];
    const int head = blockIdx.x, b = blockIdx.y, t = threadIdx.x, lane = t & 31, wib = t >> 5;
    const long long slot0 = ((long long)b * Hq + head) * splits;
    pdl_launch_dependents();
    pdl_wait();
    const float m = t < splits ? ws_ml[(slot0 + t) * 2] : kNegBig;
    const float l = t < splits ? ws_ml[(slot0 + t) * 2 + 1] : 0.f;
    float M = m;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xFFFFFFFFu, M, o));
    if (lane == 0) red[wib] = M;
    __syncthreads();
    M = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    if (sink) M = fmaxf(M, 0.f);
    const float c = ex2(m - M);
    wgt[t] = c;
    float ls = c * l;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ls += __shfl_xor_sync(0xFFFFFFFFu, ls, o);
    if (lane == 0) red[4 + wib] = ls;
    __syncthreads();
    const float L = red[4] + red[5] + red[6] + red[7] + (sink ? ex2(-M) : 0.f);
    for (int d = t; d < dv; d += 128) {
        float acc = 0.f;
        const float* src = ws_o + slot0 * dv + d;
#pragma unroll 8
        for (int s = 0; s < splits; ++s) acc = fmaf(wgt[s], __ldcs(src + (long long)s * dv), acc);
        store_elem(out + (long long)b * ldo + (long long)head * dv + d, L > 0.f ? acc / L : 0.f);
    }
}

// out[i, :] = table[ids[i], :] (bf16 rows of `width`, width % 8 == 0); an id outside [0, vocab) gives a zero row and sets *bad
__global__ void __launch_bounds__(256)
embed_gather_kernel(const __nv_bfloat16* __restrict__ table, long long ldt, const long long* __restrict__ ids, long long n, int width,
                    long long vocab, __nv_bfloat16* __restrict__ out, long long ldo, int* __restrict__ bad) {
    const int vec = width >> 3;
    const long long total = n * vec;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / vec;
        const int c = (int)(i - r * vec) << 3;
        const long long id = ids[r];
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (id >= 0 && id < vocab) v = __ldg(reinterpret_cast<const uint4*>(table + id * ldt + c));
        else if (bad && c == 0) *bad = 1;
        *reinterpret_cast<uint4*>(out + r * ldo + c) = v;
    }
}

int sm_count_now() {
    int dev = 0, sms = 1;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    return sms;
}

// tokens per split (a multiple of the CTA step) and the number of splits for a launch of B * Hkv groups over T tokens
void decode_split(int B, int Hkv, int T, int* chunk, int* splits) {
    const int want_ctas = 2 * sm_count_now();
    int s = (want_ctas + B * Hkv - 1) / (B * Hkv);
    const int max_s = (T + kCtaStep - 1) / kCtaStep;
    if (s > max_s) s = max_s;
    if (s > kMaxSplits) s = kMaxSplits;
    if (s < 1) s = 1;
    int c = (T + s - 1) / s;
    c = ((c + kCtaStep - 1) / kCtaStep) * kCtaStep;
    *chunk = c;
    *splits = (T + c - 1) / c;
}

}  // namespace

long long attn_decode_ws_bytes(int B, int T, int Hq, int Hkv) {
    int chunk = 0, splits = 1;
    decode_split(B, Hkv, T, &chunk, &splits);
    return splits == 1 ? 0 : (long long)B * Hq * splits * 130 * (long long)sizeof(float);
}

int launch_attn_decode(const AttnDecodeArgs& a, cudaStream_t stream) {
    if (a.B <= 0) return PLZ_OK;
    DecParams p = {};
    decode_split(a.B, a.Hkv, a.T, &p.chunk, &p.splits);
    const long long need = p.splits == 1 ? 0 : (long long)a.B * a.Hq * p.splits * 130 * (long long)sizeof(float);
    if (need > a.ws_bytes) { set_last_error("attn_decode: workspace of %lld bytes needed, %lld given", need, a.ws_bytes); return PLZ_ERR_TOO_LARGE; }
    p.q = a.q; p.ldq = a.ldq;
    p.k = a.k; p.v = a.v; p.k_batch = p.v_batch = a.batch_stride; p.k_tok = p.v_tok = a.tok_stride;
    p.out = a.out; p.ldo = a.ldo;
    p.ws_o = (float*)a.ws;
    p.ws_ml = p.ws_o ? p.ws_o + (long long)a.B * a.Hq * p.splits * 128 : nullptr;
    p.T = a.T; p.Hq = a.Hq; p.Hkv = a.Hkv; p.group = a.Hq / a.Hkv; p.passes = (p.group + 3) / 4;
    p.scale_log2e = a.scale * kLog2eDec;
    PLZ_LAUNCH_CHAIN((attn_decode_partial_kernel<__nv_bfloat16, 16, false>), dim3(p.splits, a.Hkv * p.passes, a.B), dim3(kDecWarps * 32), 0, stream, p);
    if (p.splits > 1) {
        PLZ_LAUNCH_CHAIN(attn_decode_combine_kernel<__nv_bfloat16>, dim3(a.Hq, a.B), dim3(128), 0, stream, (const float*)p.ws_o, (const float*)p.ws_ml,
                         p.splits, a.Hq, 128, 0, (__nv_bfloat16*)p.out, p.ldo);
    }
    return PLZ_OK;
}

// splits for a cache of `cap` positions whose length is known on the device only
static int ext_splits(int B, int groups, int cap) {
    int chunk = 0, splits = 1;
    decode_split(B, groups, cap, &chunk, &splits);
    return splits;
}
long long attn_bias_decode_ws_bytes(int B, int H, int G, int dv, int cap) {
    const int passes = (H / G + 3) / 4, splits = ext_splits(B, G * passes, cap);
    return splits == 1 ? 0 : (long long)B * H * splits * (dv + 2) * (long long)sizeof(float);
}
template <typename T>
static int launch_attn_bias_decode_t(const AttnBiasArgs& a, int cap, float* ws, cudaStream_t stream) {
    DecParams p = {};
    p.group = a.H / a.G; p.passes = (p.group + 3) / 4;
    p.splits = ext_splits(a.B, a.G * p.passes, cap);
    p.q = a.q; p.ldq = a.ldq; p.k = a.k; p.v = a.v; p.k_batch = a.k_batch; p.v_batch = a.v_batch;
    p.k_tok = (long long)a.G * a.dk; p.v_tok = (long long)a.G * a.dv;
    p.out = a.o; p.ldo = a.ldo; p.ws_o = ws; p.ws_ml = ws ? ws + (long long)a.B * a.H * p.splits * a.dv : nullptr;
    p.Hq = a.H; p.Hkv = a.G; p.scale_log2e = a.scale * kLog2eDec;
    p.dk = a.dk; p.dv = a.dv; p.pos = a.pos; p.bias = a.bias; p.ldb = a.ldb; p.n_bias = a.n_bias; p.sink = a.sink;
    const dim3 grid(p.splits, a.G * p.passes, a.B), block(kDecWarps * 32);
    const int d = a.dk > a.dv ? a.dk : a.dv;
    if (d <= 64) PLZ_LAUNCH_CHAIN((attn_decode_partial_kernel<T, 8, true>), grid, block, 0, stream, p);
    else if (d <= 128) PLZ_LAUNCH_CHAIN((attn_decode_partial_kernel<T, 16, true>), grid, block, 0, stream, p);
    else PLZ_LAUNCH_CHAIN((attn_decode_partial_kernel<T, 32, true>), grid, block, 0, stream, p);
    if (p.splits > 1) {
        PLZ_LAUNCH_CHAIN(attn_decode_combine_kernel<T>, dim3(a.H, a.B), dim3(128), 0, stream, (const float*)p.ws_o, (const float*)p.ws_ml, p.splits, a.H,
                         a.dv, a.sink, (T*)p.out, p.ldo);
    }
    return PLZ_OK;
}
int launch_attn_bias_decode(int dtype, const AttnBiasArgs& a, int cap, void* ws, long long ws_bytes, cudaStream_t stream) {
    if (a.B <= 0) return PLZ_OK;
    if (a.n != 1) { set_last_error("attention decode: one token per sequence (%d given)", a.n); return PLZ_ERR_BAD_SHAPE; }
    const long long need = attn_bias_decode_ws_bytes(a.B, a.H, a.G, a.dv, cap);
    if (need > ws_bytes) { set_last_error("attention decode: workspace of %lld bytes needed, %lld given", need, ws_bytes); return PLZ_ERR_TOO_LARGE; }
    return dtype == 1 ? launch_attn_bias_decode_t<float>(a, cap, (float*)ws, stream) : launch_attn_bias_decode_t<__nv_bfloat16>(a, cap, (float*)ws, stream);
}

int launch_embed_gather(const void* table, long long ldt, const long long* ids, long long n, int width, long long vocab, void* out,
                        long long ldo, int* bad, cudaStream_t stream) {
    if (n <= 0) return PLZ_OK;
    long long blocks = (n * (width >> 3) + 255) / 256;
    const long long cap = (long long)sm_count_now() * 16;
    if (blocks > cap) blocks = cap;
    embed_gather_kernel<<<(unsigned)blocks, 256, 0, stream>>>((const __nv_bfloat16*)table, ldt, ids, n, width, vocab, (__nv_bfloat16*)out, ldo, bad);
    PLZ_LAUNCH_CHECK();
    return PLZ_OK;
}

}  // namespace plz
