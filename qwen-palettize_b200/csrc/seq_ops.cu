// Row-wise steps of the hybrid decoders around their Linears, recurrences and attention: embedding with a scale or a norm, the norm on a
// sublayer's output fused with the fp32 residual update and the norm ahead of the next sublayer, the norm + gate that closes a recurrent mixer, the short causal
// convolution with its activation, unit norm and decay, the query / key norm that feeds the cache, and token sampling.
//
// Rows are b * n + t: B sequences advance in lockstep by n tokens each; *pos (device memory, so that a captured step can be
// replayed at later positions) is the position of the first of them. The residual stream, statistics, decays and gates are fp32.
#include "seq_math.cuh"

namespace plz {
namespace {

// x[r, :] = table[ids[r], :] * scale (fp32), then (NORM) over its root mean square times w + w_offset; x2 the same, xb the same in T
// (bf16 models: the operand of the first Linear)
struct EmbedParams {
    const void* table; long long ldt; const long long* ids; int W; long long vocab; float scale;
    const float* w; float w_offset, eps;
    float* x; float* x2; void* xb; int* bad;
};
template <typename T>
__global__ void __launch_bounds__(256)
embed_scale_kernel(const EmbedParams p) {
    __shared__ float part[8];
    const long long r = blockIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const long long id = p.ids[r];
    const bool ok = id >= 0 && id < p.vocab;
    if (!ok && p.bad && threadIdx.x == 0) *p.bad = 1;
    const T* row = (const T*)p.table + (ok ? id : 0) * p.ldt;
    float rs = 1.f;
    if (p.w) {
        float s = 0.f;
        for (int c = threadIdx.x; c < p.W; c += 256) { const float v = ok ? to_f(row[c]) * p.scale : 0.f; s = fmaf(v, v, s); }
        rs = 1.0f / sqrtf(block_sum<8>(s, part) / (float)p.W + p.eps);
    }
    for (int c = threadIdx.x; c < p.W; c += 256) {
        float v = ok ? to_f(row[c]) * p.scale : 0.f;
        if (p.w) v = v * rs * (p.w[c] + p.w_offset);
        p.x[r * p.W + c] = v;
        if (p.x2) p.x2[r * p.W + c] = v;
        if (p.xb) ((T*)p.xb)[r * p.W + c] = from_f<T>(v);
    }
}

// x += mult * y / rms(y) * (w + w_offset);  x += add_rows + add_vec;  out = T(x), or T(x / rms(x) * (w_next + w_offset))
struct StreamParams {
    const void* y; long long ldy; const float* w; float w_offset, mult, eps; int W;
    float* x; const float* add_rows; const float* add_vec; const float* w_next; void* out;
};
template <typename T>
__global__ void __launch_bounds__(256)
stream_kernel(const StreamParams p) {
    __shared__ float part[8];
    const long long r = blockIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const T* yr = (const T*)p.y + r * p.ldy;
    float* xr = p.x + r * p.W;
    const float* er = p.add_rows ? p.add_rows + r * p.W : nullptr;
    T* out = (T*)p.out + (p.out ? r * p.W : 0);
    float rs = 0.f;
    if (p.y) {
        float s = 0.f;
        for (int c = threadIdx.x; c < p.W; c += 256) { const float v = to_f(yr[c]); s = fmaf(v, v, s); }
        rs = 1.0f / sqrtf(block_sum<8>(s, part) / (float)p.W + p.eps);
    }
    float sx = 0.f;
    for (int c = threadIdx.x; c < p.W; c += 256) {
        float v = xr[c];
        if (p.y) v += p.mult * (to_f(yr[c]) * rs * (p.w[c] + p.w_offset));
        if (er) v += er[c];
        if (p.add_vec) v += p.add_vec[c];
        xr[c] = v;
        sx = fmaf(v, v, sx);
        if (p.out && !p.w_next) out[c] = from_f<T>(v);
    }
    if (p.out && p.w_next) {
        const float rx = 1.0f / sqrtf(block_sum<8>(sx, part) / (float)p.W + p.eps);
        for (int c = threadIdx.x; c < p.W; c += 256) out[c] = from_f<T>(xr[c] * rx * (p.w_next[c] + p.w_offset));   // this thread's own x
    }
}
// the same for W % 4 == 0 and 16-byte aligned rows, four columns per access, y and x kept in registers (W <= 1024 * NQ)
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xFFFF0000u), __uint_as_float(r.y << 16), __uint_as_float(r.y & 0xFFFF0000u));
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w)); }
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ float dot4(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }
template <typename T, int NQ>
__global__ void __launch_bounds__(256, NQ <= 2 ? 8 : (NQ <= 4 ? 6 : 3))
stream4_kernel(const StreamParams p) {
    __shared__ float part[8];
    const long long r = blockIdx.x;
    const int n4 = p.W >> 2;
    pdl_launch_dependents();
    pdl_wait();
    const T* yr = (const T*)p.y + r * p.ldy;
    float* xr = p.x + r * p.W;
    const float* er = p.add_rows ? p.add_rows + r * p.W : nullptr;
    T* out = (T*)p.out + (p.out ? r * p.W : 0);
    float4 x[NQ];                  // the sublayer's output, then the stream
    float s = 0.f, rs = 0.f;
    if (p.y) {
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
            const int c = threadIdx.x + i * 256;
            if (c < n4) { x[i] = load4(yr + c * 4); s += dot4(x[i]); }
        }
        rs = p.mult / sqrtf(block_sum<8>(s, part) / (float)p.W + p.eps);
    }
    float sx = 0.f;
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
        const int c = threadIdx.x + i * 256;
        if (c < n4) {
            float4 a = load4(xr + c * 4);
            if (p.y) {
                const float4 g = __ldg(reinterpret_cast<const float4*>(p.w + c * 4));
                a.x += x[i].x * rs * (g.x + p.w_offset); a.y += x[i].y * rs * (g.y + p.w_offset);
                a.z += x[i].z * rs * (g.z + p.w_offset); a.w += x[i].w * rs * (g.w + p.w_offset);
            }
            if (er) { const float4 e = load4(er + c * 4); a.x += e.x; a.y += e.y; a.z += e.z; a.w += e.w; }
            if (p.add_vec) { const float4 e = __ldg(reinterpret_cast<const float4*>(p.add_vec + c * 4)); a.x += e.x; a.y += e.y; a.z += e.z; a.w += e.w; }
            store4(xr + c * 4, a);
            if (p.out && !p.w_next) store4(out + c * 4, a);
            sx += dot4(a);
            x[i] = a;
        }
    }
    if (p.out && p.w_next) {
        const float rx = 1.0f / sqrtf(block_sum<8>(sx, part) / (float)p.W + p.eps);
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
            const int c = threadIdx.x + i * 256;
            if (c < n4) {
                const float4 g = __ldg(reinterpret_cast<const float4*>(p.w_next + c * 4));
                store4(out + c * 4, make_float4(x[i].x * rx * (g.x + p.w_offset), x[i].y * rx * (g.y + p.w_offset), x[i].z * rx * (g.z + p.w_offset),
                                                x[i].w * rx * (g.w + p.w_offset)));
            }
        }
    }
}

// out[i, :] = x[idx[i], :] / rms * (w + w_offset) in T (idx null: row i)
template <typename T>
__global__ void __launch_bounds__(256)
rows_norm_kernel(const float* __restrict__ x, const long long* __restrict__ idx, const float* __restrict__ w, float w_offset, float eps, int W,
                 T* __restrict__ out) {
    __shared__ float part[8];
    pdl_launch_dependents();
    pdl_wait();
    const long long i = blockIdx.x, r = idx ? idx[i] : i;
    float s = 0.f;
    for (int c = threadIdx.x; c < W; c += 256) { const float v = x[r * W + c]; s = fmaf(v, v, s); }
    s = block_sum<8>(s, part);
    const float rs = 1.0f / sqrtf(s / (float)W + eps);
    for (int c = threadIdx.x; c < W; c += 256) out[i * W + c] = from_f<T>(x[r * W + c] * rs * (w[c] + w_offset));
}

// out[r, g * L + c] = o / rms(o over the L values of the group) * w[c] * sigmoid(gate); a block per (row, several groups), a warp
// per group when L is small, the whole block otherwise
template <typename T, bool BLOCK>
__global__ void __launch_bounds__(256)
norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long ldg, const float* __restrict__ w, float eps, int groups, int L,
                 T* __restrict__ out) {
    __shared__ float part[8];
    const long long r = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = BLOCK ? (int)blockIdx.y : (int)blockIdx.y * 8 + warp;
    const int t = BLOCK ? (int)threadIdx.x : lane, team = BLOCK ? 256 : 32;
    pdl_launch_dependents();
    pdl_wait();
    if (!BLOCK && g >= groups) return;
    const long long W = (long long)groups * L;
    const float* og = o + r * W + (long long)g * L;
    const T* gg = gate + r * ldg + (long long)g * L;
    float s = 0.f;
    for (int c = t; c < L; c += team) s = fmaf(og[c], og[c], s);
    s = BLOCK ? block_sum<8>(s, part) : warp_sum(s);
    const float rs = 1.0f / sqrtf(s / (float)L + eps);
    T* dst = out + r * W + (long long)g * L;
    for (int c = t; c < L; c += team) dst[c] = from_f<T>(og[c] * rs * w[c] * sigmoid_f(to_f(gg[c])));
}

// ---- gated delta rule: everything between the projections and the recurrence ------------------------------------------
struct DeltaPrep {
    const void* proj; long long ldp; int off_q, off_k, off_v, off_b;   // raw projections of this step
    const void* a; long long lda;                                      // decay pre-activation [rows, H * dk]
    const float* taps;                                                 // [channels, n_taps], channels = q | k | v
    const float* A_log; const float* dt_bias;                          // [H], [H * dk]
    void* conv; int n_taps;                                            // [B, n_taps - 1, channels] inputs before this step, oldest first
    int B, n, H, G, dk, dv;
    float q_scale;
    float* q; float* k; float* v; float* logg; float* beta;            // [rows, G * dk] x 2, [rows, H * dv], [rows, H * dk], [rows, H]
    int update;                                                        // n == 1: shift this token into `conv`
};

// One warp per item of a row: G query heads, G key heads, H value heads, H decay heads (lane 0 of the last also does beta).
template <typename T>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const DeltaPrep p) {
    const long long r = blockIdx.x;
    const int lane = threadIdx.x & 31, item = (int)blockIdx.y * 8 + (threadIdx.x >> 5);
    const int t = (int)(r % p.n);
    const long long b = r / p.n;
    pdl_launch_dependents();
    pdl_wait();
    if (item >= 2 * p.G + 2 * p.H) return;
    if (item >= 2 * p.G + p.H) {
        const int h = item - 2 * p.G - p.H;
        const float rate = expf(p.A_log[h]);
        const T* ar = (const T*)p.a + r * p.lda + (long long)h * p.dk;
        float* gr = p.logg + (r * p.H + h) * p.dk;
        for (int c = lane; c < p.dk; c += 32) gr[c] = -rate * softplus_f(to_f(ar[c]) + p.dt_bias[h * p.dk + c]);
        if (lane == 0) p.beta[r * p.H + h] = sigmoid_f(to_f(((const T*)p.proj)[r * p.ldp + p.off_b + h]));
        return;
    }
    const int kind = item < p.G ? 0 : (item < 2 * p.G ? 1 : 2);
    const int head = kind == 0 ? item : (kind == 1 ? item - p.G : item - 2 * p.G);
    const int L = kind == 2 ? p.dv : p.dk;
    const int off = (kind == 0 ? p.off_q : (kind == 1 ? p.off_k : p.off_v)) + head * L;       // column of the projection
    const int ch0 = (kind == 0 ? 0 : (kind == 1 ? p.G * p.dk : 2 * p.G * p.dk)) + head * L;   // convolution channel
    const int C = 2 * p.G * p.dk + p.H * p.dv, keep = p.n_taps - 1;
    T* cs = (T*)p.conv + b * (long long)keep * C;
    float* dst = kind == 0 ? p.q + (r * p.G + head) * p.dk : (kind == 1 ? p.k + (r * p.G + head) * p.dk : p.v + (r * p.H + head) * p.dv);
    float ss = 0.f;
    for (int c = lane; c < L; c += 32) {
        const float* w = p.taps + (long long)(ch0 + c) * p.n_taps;
        const T cur = ((const T*)p.proj)[r * p.ldp + off + c];
        float s = 0.f;
        for (int j = 0; j < keep; ++j) {             // tap j looks back keep - j tokens
            const int tt = t - (keep - j);
            const T in = tt >= 0 ? ((const T*)p.proj)[(r - (keep - j)) * p.ldp + off + c] : cs[(long long)(tt + keep) * C + ch0 + c];
            s = fmaf(w[j], to_f(in), s);
        }
        s = fmaf(w[keep], to_f(cur), s);
        if (p.update && keep > 0) {
            for (int j = 0; j + 1 < keep; ++j) cs[(long long)j * C + ch0 + c] = cs[(long long)(j + 1) * C + ch0 + c];
            cs[(long long)(keep - 1) * C + ch0 + c] = cur;
        }
        s = silu_f(s);
        dst[c] = s;
        ss = fmaf(s, s, ss);
    }
    if (kind == 2) return;
    ss = warp_sum(ss);
    const float f = (kind == 0 ? p.q_scale : 1.0f) / sqrtf(ss + 1e-6f);
    for (int c = lane; c < L; c += 32) dst[c] *= f;      // this lane's own elements
}

// The same for portions: a warp takes one item over kPrepRows consecutive tokens, four channels per lane (head sizes up to 128, a
// multiple of 4), the convolution's inputs sliding through registers. Up to four taps (missing ones count as zero weights).
constexpr int kPrepRows = 16;
template <typename T>
__global__ void __launch_bounds__(256)
delta_prep_rows_kernel(const DeltaPrep p) {
    const int lane = threadIdx.x & 31, item = (int)blockIdx.y * 8 + (threadIdx.x >> 5);
    const int blocks = (p.n + kPrepRows - 1) / kPrepRows;
    const long long b = blockIdx.x / blocks;
    const int t0 = (int)(blockIdx.x % blocks) * kPrepRows, t1 = min(p.n, t0 + kPrepRows);
    const long long r0 = b * p.n;
    pdl_launch_dependents();
    pdl_wait();
    if (item >= 2 * p.G + 2 * p.H) return;
    const int c = lane * 4;
    if (item >= 2 * p.G + p.H) {
        const int h = item - 2 * p.G - p.H;
        const float rate = -expf(p.A_log[h]);
        float4 bias = make_float4(0.f, 0.f, 0.f, 0.f);
        const bool in = c < p.dk;
        if (in) bias = make_float4(p.dt_bias[h * p.dk + c], p.dt_bias[h * p.dk + c + 1], p.dt_bias[h * p.dk + c + 2], p.dt_bias[h * p.dk + c + 3]);
        for (int tb = t0; tb < t1; tb += 4) {
            float4 x[4];
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (in && tb + u < t1) x[u] = load4((const T*)p.a + (r0 + tb + u) * p.lda + (long long)h * p.dk + c);
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (in && tb + u < t1)
                    *reinterpret_cast<float4*>(p.logg + ((r0 + tb + u) * p.H + h) * p.dk + c) =
                        make_float4(rate * softplus_f(x[u].x + bias.x), rate * softplus_f(x[u].y + bias.y), rate * softplus_f(x[u].z + bias.z),
                                    rate * softplus_f(x[u].w + bias.w));
        }
        if (lane < kPrepRows && t0 + lane < t1)
            p.beta[(r0 + t0 + lane) * p.H + h] = sigmoid_f(to_f(((const T*)p.proj)[(r0 + t0 + lane) * p.ldp + p.off_b + h]));
        return;
    }
    const int kind = item < p.G ? 0 : (item < 2 * p.G ? 1 : 2);
    const int head = kind == 0 ? item : (kind == 1 ? item - p.G : item - 2 * p.G);
    const int L = kind == 2 ? p.dv : p.dk;
    const int off = (kind == 0 ? p.off_q : (kind == 1 ? p.off_k : p.off_v)) + head * L;
    const int ch0 = (kind == 0 ? 0 : (kind == 1 ? p.G * p.dk : 2 * p.G * p.dk)) + head * L;
    const int C = 2 * p.G * p.dk + p.H * p.dv, keep = p.n_taps - 1;
    const bool in = c < L;
    float w[4][4];                                    // [tap looking back 3 - j tokens][channel]
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int k = j - (4 - p.n_taps);         // stored column of this tap
            w[j][e] = in && k >= 0 ? p.taps[(long long)(ch0 + c + e) * p.n_taps + k] : 0.f;
        }
    auto input = [&](int t) {                         // tokens before the portion come from the kept inputs, before those zero
        if (!in) return make_float4(0.f, 0.f, 0.f, 0.f);
        if (t >= 0) return load4((const T*)p.proj + (r0 + t) * p.ldp + off + c);
        if (t + keep < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
        return load4((const T*)p.conv + (b * keep + t + keep) * (long long)C + ch0 + c);
    };
    float4 x0 = input(t0 - 3), x1 = input(t0 - 2), x2 = input(t0 - 1);
    float* dst = kind == 0 ? p.q + head * p.dk : (kind == 1 ? p.k + head * p.dk : p.v + head * p.dv);
    const long long ldd = kind == 2 ? (long long)p.H * p.dv : (long long)p.G * p.dk;
    for (int tb = t0; tb < t1; tb += 4) {
        float4 nx[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) nx[u] = tb + u < t1 ? input(tb + u) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const float4 x3 = nx[u];
            float4 y;
            y.x = silu_f(w[0][0] * x0.x + w[1][0] * x1.x + w[2][0] * x2.x + w[3][0] * x3.x);
            y.y = silu_f(w[0][1] * x0.y + w[1][1] * x1.y + w[2][1] * x2.y + w[3][1] * x3.y);
            y.z = silu_f(w[0][2] * x0.z + w[1][2] * x1.z + w[2][2] * x2.z + w[3][2] * x3.z);
            y.w = silu_f(w[0][3] * x0.w + w[1][3] * x1.w + w[2][3] * x2.w + w[3][3] * x3.w);
            x0 = x1; x1 = x2; x2 = x3;
            float f = 1.f;
            if (kind != 2) {
                const float ss = warp_sum(y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w);
                f = (kind == 0 ? p.q_scale : 1.0f) / sqrtf(ss + 1e-6f);
            }
            if (in && tb + u < t1) *reinterpret_cast<float4*>(dst + (r0 + tb + u) * ldd + c) = make_float4(y.x * f, y.y * f, y.z * f, y.w * f);
        }
    }
}

// the last n_taps - 1 inputs after a portion of n tokens (n >= 1)
template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const T* __restrict__ proj, long long ldp, int off_q, int off_k, int off_v, int qk, int C, int keep, int n, T* __restrict__ conv) {
    const long long b = blockIdx.y;
    const int ch = (int)blockIdx.x * 256 + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (ch >= C) return;
    const int col = ch < qk ? off_q + ch : (ch < 2 * qk ? off_k + ch - qk : off_v + ch - 2 * qk);
    T* cs = conv + b * (long long)keep * C + ch;
    for (int j = 0; j < keep; ++j) {             // ascending: a slot is read (as j + n) before it is overwritten
        const int t = n - keep + j;
        cs[(long long)j * C] = t >= 0 ? proj[(b * n + t) * ldp + col] : cs[(long long)(j + n) * C];
    }
}

// ---- attention: norm over the whole query / key projection, value mixing, cache write ----------------------------------
struct AttnPrep {
    const void* proj; long long ldp; int off_q, off_k, off_v;
    const float* wq; const float* wk;              // [H * dk], [G * dk]
    const float* mix;                              // [1] or null; v <- (1 - mix) v + mix v_first
    void* v_first; int v_first_write;              // [rows, G * dv]
    void* q;                                       // [rows, H * dk]
    void* kc; void* vc; long long k_batch, v_batch;   // caches [B, T, G * dk], [B, T, G * dv]; elements per sequence
    const int* pos;
    int n, qw, kw, vw, cap;
    float eps;
};
template <typename T>
__global__ void __launch_bounds__(256)
attn_prep_kernel(const AttnPrep p) {
    __shared__ float part[8];
    const long long r = blockIdx.x, b = r / p.n;
    pdl_launch_dependents();
    pdl_wait();
    const int at = *p.pos + (int)(r % p.n);
    if (at >= p.cap) return;                       // the host checks the capacity; never write past it
    const T* row = (const T*)p.proj + r * p.ldp;
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x; c < p.qw; c += 256) { const float v = to_f(row[p.off_q + c]); sq = fmaf(v, v, sq); }
    for (int c = threadIdx.x; c < p.kw; c += 256) { const float v = to_f(row[p.off_k + c]); sk = fmaf(v, v, sk); }
    sq = block_sum<8>(sq, part);
    sk = block_sum<8>(sk, part);
    const float rq = 1.0f / sqrtf(sq / (float)p.qw + p.eps), rk = 1.0f / sqrtf(sk / (float)p.kw + p.eps);
    T* qo = (T*)p.q + r * p.qw;
    T* ko = (T*)p.kc + b * p.k_batch + (long long)at * p.kw;
    T* vo = (T*)p.vc + b * p.v_batch + (long long)at * p.vw;
    for (int c = threadIdx.x; c < p.qw; c += 256) qo[c] = from_f<T>(to_f(row[p.off_q + c]) * rq * p.wq[c]);
    for (int c = threadIdx.x; c < p.kw; c += 256) ko[c] = from_f<T>(to_f(row[p.off_k + c]) * rk * p.wk[c]);
    const float lam = p.mix ? *p.mix : 0.f;
    T* vf = (T*)p.v_first + (p.v_first ? r * p.vw : 0);
    for (int c = threadIdx.x; c < p.vw; c += 256) {
        T v = row[p.off_v + c];
        if (p.v_first_write) vf[c] = v;
        if (p.mix) v = from_f<T>((1.0f - lam) * to_f(v) + lam * to_f(vf[c]));
        vo[c] = v;
    }
}

__global__ void advance_kernel(int* pos, int n) {
    pdl_wait();
    *pos += n;
}

// ---- sampling: one block per row ------------------------------------------------------------------------------------------
// temperature == 0: index of the largest logit, the first of equals. Else the largest of logit / temperature + Gumbel noise
// among the top_k logits (top_k <= 0: all), the noise from a counter hash of (seed, *pos, row, index).
__device__ __forceinline__ uint32_t mix32(uint32_t h) {
    h ^= h >> 16; h *= 0x85EBCA6Bu; h ^= h >> 13; h *= 0xC2B2AE35u; h ^= h >> 16;
    return h;
}
__global__ void __launch_bounds__(256)
sample_kernel(const float* __restrict__ logits, long long ld, int V, float temperature, int top_k, uint32_t seed, const int* __restrict__ pos,
              long long* __restrict__ out) {
    __shared__ float sv[8];
    __shared__ int si[8];
    __shared__ int cnt;
    const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    pdl_launch_dependents();
    pdl_wait();
    const float* lr = logits + (long long)row * ld;
    uint32_t floor_key = 0;              // smallest admitted key
    auto key_of = [](float v) { const uint32_t u = __float_as_uint(v); return (u & 0x80000000u) ? ~u : (u | 0x80000000u); };
    if (temperature > 0.f && top_k > 0 && top_k < V) {
        // largest key that at least top_k logits reach, bit by bit
        for (int bit = 31; bit >= 0; --bit) {
            const uint32_t trial = floor_key | (1u << bit);
            if (threadIdx.x == 0) cnt = 0;
            __syncthreads();
            int c = 0;
            for (int i = threadIdx.x; i < V; i += 256) c += key_of(lr[i]) >= trial;
            c = __reduce_add_sync(0xFFFFFFFFu, c);
            if (lane == 0) atomicAdd(&cnt, c);
            __syncthreads();
            if (cnt >= top_k) floor_key = trial;
            __syncthreads();
        }
    }
    const uint32_t base = mix32(seed ^ mix32((uint32_t)*pos * 0x9E3779B1u + (uint32_t)row));
    float best = -INFINITY;
    int bi = V;
    for (int i = threadIdx.x; i < V; i += 256) {
        float v = lr[i];
        if (temperature > 0.f) {
            if (key_of(v) < floor_key) continue;
            const float u = ((float)(mix32(base ^ mix32((uint32_t)i + 0x7F4A7C15u)) >> 8) + 0.5f) * (1.0f / 16777216.0f);
            v = v / temperature - logf(-logf(u));
        }
        if (v > best || bi == V) { best = v; bi = i; }
    }
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xFFFFFFFFu, best, o);
        const int oi = __shfl_xor_sync(0xFFFFFFFFu, bi, o);
        if (oi < V && (bi == V || ov > best || (ov == best && oi < bi))) { best = ov; bi = oi; }
    }
    if (lane == 0) { sv[warp] = best; si[warp] = bi; }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < 8; ++w)
            if (si[w] < V && (bi == V || sv[w] > best || (sv[w] == best && si[w] < bi))) { best = sv[w]; bi = si[w]; }
        out[row] = bi < V ? bi : 0;
    }
}

typedef __nv_bfloat16 bf;

}  // namespace

int launch_seq_embed(int dtype, const void* table, long long ldt, const long long* ids, long long rows, int W, long long vocab, float scale,
                     const float* norm_w, float norm_offset, float eps, float* x, float* x2, void* xb, int* bad, cudaStream_t stream) {
    if (rows <= 0) return PLZ_OK;
    const EmbedParams p = {table, ldt, ids, W, vocab, scale, norm_w, norm_offset, eps, x, x2, xb, bad};
    if (dtype == 1) PLZ_LAUNCH_CHAIN(embed_scale_kernel<float>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    else PLZ_LAUNCH_CHAIN(embed_scale_kernel<bf>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    return PLZ_OK;
}

template <typename T>
static int stream_t_(const StreamArgs& a, cudaStream_t s) {
    const StreamParams p = {a.y, a.ldy, a.w, a.w_offset, a.mult, a.eps, a.W, a.x, a.add_rows, a.add_vec, a.w_next, a.out};
    const uintptr_t ptrs = (uintptr_t)a.y | (uintptr_t)a.w | (uintptr_t)a.x | (uintptr_t)a.add_rows | (uintptr_t)a.add_vec | (uintptr_t)a.w_next | (uintptr_t)a.out;
    const bool vec = a.W % 4 == 0 && a.ldy % 4 == 0 && !(ptrs & 15);
    const dim3 grid((unsigned)a.rows), block(256);
    if (vec && a.W <= 2048) PLZ_LAUNCH_CHAIN((stream4_kernel<T, 2>), grid, block, 0, s, p);
    else if (vec && a.W <= 3072) PLZ_LAUNCH_CHAIN((stream4_kernel<T, 3>), grid, block, 0, s, p);
    else if (vec && a.W <= 4096) PLZ_LAUNCH_CHAIN((stream4_kernel<T, 4>), grid, block, 0, s, p);
    else if (vec && a.W <= 8192) PLZ_LAUNCH_CHAIN((stream4_kernel<T, 8>), grid, block, 0, s, p);
    else PLZ_LAUNCH_CHAIN(stream_kernel<T>, grid, block, 0, s, p);
    return PLZ_OK;
}
int launch_seq_stream(int dtype, const StreamArgs& a, cudaStream_t stream) {
    if (a.rows <= 0) return PLZ_OK;
    return dtype == 1 ? stream_t_<float>(a, stream) : stream_t_<bf>(a, stream);
}

int launch_seq_rows_norm(int dtype, const float* x, const long long* idx, const float* w, float w_offset, float eps, long long rows, int W, void* out,
                         cudaStream_t stream) {
    if (rows <= 0) return PLZ_OK;
    if (dtype == 1) PLZ_LAUNCH_CHAIN(rows_norm_kernel<float>, dim3((unsigned)rows), dim3(256), 0, stream, x, idx, w, w_offset, eps, W, (float*)out);
    else PLZ_LAUNCH_CHAIN(rows_norm_kernel<bf>, dim3((unsigned)rows), dim3(256), 0, stream, x, idx, w, w_offset, eps, W, (bf*)out);
    return PLZ_OK;
}

int launch_seq_norm_gate(int dtype, const float* o, const void* gate, long long ldg, const float* w, float eps, long long rows, int groups, int L,
                         void* out, cudaStream_t stream) {
    if (rows <= 0) return PLZ_OK;
    const bool block = L > 256;
    const dim3 grid((unsigned)rows, block ? groups : (groups + 7) / 8);
    if (dtype == 1) {
        if (block) PLZ_LAUNCH_CHAIN((norm_gate_kernel<float, true>), grid, dim3(256), 0, stream, o, (const float*)gate, ldg, w, eps, groups, L, (float*)out);
        else PLZ_LAUNCH_CHAIN((norm_gate_kernel<float, false>), grid, dim3(256), 0, stream, o, (const float*)gate, ldg, w, eps, groups, L, (float*)out);
    } else {
        if (block) PLZ_LAUNCH_CHAIN((norm_gate_kernel<bf, true>), grid, dim3(256), 0, stream, o, (const bf*)gate, ldg, w, eps, groups, L, (bf*)out);
        else PLZ_LAUNCH_CHAIN((norm_gate_kernel<bf, false>), grid, dim3(256), 0, stream, o, (const bf*)gate, ldg, w, eps, groups, L, (bf*)out);
    }
    return PLZ_OK;
}

int launch_delta_prep(int dtype, const DeltaPrepArgs& a, cudaStream_t stream) {
    const long long rows = (long long)a.B * a.n;
    if (rows <= 0) return PLZ_OK;
    DeltaPrep p;
    p.proj = a.proj; p.ldp = a.ldp; p.off_q = a.off_q; p.off_k = a.off_k; p.off_v = a.off_v; p.off_b = a.off_b; p.a = a.a; p.lda = a.lda;
    p.taps = a.taps; p.A_log = a.A_log; p.dt_bias = a.dt_bias; p.conv = a.conv; p.n_taps = a.n_taps;
    p.B = a.B; p.n = a.n; p.H = a.H; p.G = a.G; p.dk = a.dk; p.dv = a.dv; p.q_scale = a.q_scale;
    p.q = a.q; p.k = a.k; p.v = a.v; p.logg = a.logg; p.beta = a.beta;
    p.update = a.n == 1;
    const dim3 grid((unsigned)rows, (2 * a.G + 2 * a.H + 7) / 8);
    const int C4 = 2 * a.G * a.dk + a.H * a.dv;
    const bool rows4 = a.n >= 8 && a.n_taps <= 4 && a.dk % 4 == 0 && a.dv % 4 == 0 && a.dk <= 128 && a.dv <= 128 && C4 % 4 == 0 && a.ldp % 4 == 0 && a.lda % 4 == 0 &&
                       a.off_q % 4 == 0 && a.off_k % 4 == 0 && a.off_v % 4 == 0 && !(((uintptr_t)a.proj | (uintptr_t)a.a | (uintptr_t)a.conv | (uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.logg) & 15);
    if (rows4) {
        const dim3 g4((unsigned)((long long)a.B * ((a.n + kPrepRows - 1) / kPrepRows)), grid.y);
        if (dtype == 1) PLZ_LAUNCH_CHAIN(delta_prep_rows_kernel<float>, g4, dim3(256), 0, stream, p);
        else PLZ_LAUNCH_CHAIN(delta_prep_rows_kernel<bf>, g4, dim3(256), 0, stream, p);
    } else if (dtype == 1) PLZ_LAUNCH_CHAIN(delta_prep_kernel<float>, grid, dim3(256), 0, stream, p);
    else PLZ_LAUNCH_CHAIN(delta_prep_kernel<bf>, grid, dim3(256), 0, stream, p);
    if (a.n > 1 && a.n_taps > 1) {
        const int qk = a.G * a.dk, C = 2 * qk + a.H * a.dv;
        const dim3 g2((C + 255) / 256, a.B);
        if (dtype == 1) PLZ_LAUNCH_CHAIN(conv_state_kernel<float>, g2, dim3(256), 0, stream, (const float*)a.proj, a.ldp, a.off_q, a.off_k, a.off_v, qk, C, a.n_taps - 1, a.n, (float*)a.conv);
        else PLZ_LAUNCH_CHAIN(conv_state_kernel<bf>, g2, dim3(256), 0, stream, (const bf*)a.proj, a.ldp, a.off_q, a.off_k, a.off_v, qk, C, a.n_taps - 1, a.n, (bf*)a.conv);
    }
    return PLZ_OK;
}

int launch_attn_prep(int dtype, const AttnPrepArgs& a, cudaStream_t stream) {
    const long long rows = (long long)a.B * a.n;
    if (rows <= 0) return PLZ_OK;
    AttnPrep p;
    p.proj = a.proj; p.ldp = a.ldp; p.off_q = a.off_q; p.off_k = a.off_k; p.off_v = a.off_v; p.wq = a.wq; p.wk = a.wk; p.mix = a.mix;
    p.v_first = a.v_first; p.v_first_write = a.v_first_write; p.q = a.q; p.kc = a.kc; p.vc = a.vc; p.k_batch = a.k_batch; p.v_batch = a.v_batch;
    p.pos = a.pos; p.n = a.n; p.qw = a.qw; p.kw = a.kw; p.vw = a.vw; p.cap = a.cap; p.eps = a.eps;
    if (dtype == 1) PLZ_LAUNCH_CHAIN(attn_prep_kernel<float>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    else PLZ_LAUNCH_CHAIN(attn_prep_kernel<bf>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    return PLZ_OK;
}

int launch_advance(int* pos, int n, cudaStream_t stream) {
    PLZ_LAUNCH_CHAIN(advance_kernel, dim3(1), dim3(1), 0, stream, pos, n);
    return PLZ_OK;
}

int launch_sample(const float* logits, long long ld, int rows, int V, float temperature, int top_k, uint32_t seed, const int* pos, long long* out,
                  cudaStream_t stream) {
    if (rows <= 0) return PLZ_OK;
    PLZ_LAUNCH_CHAIN(sample_kernel, dim3(rows), dim3(256), 0, stream, logits, ld, V, temperature, top_k, seed, pos, out);
    return PLZ_OK;
}

}  // namespace plz
