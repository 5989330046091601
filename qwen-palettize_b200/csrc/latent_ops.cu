// Row-wise steps of attention over cached latents: the norms of the two latents and the cache write, and rotary positions on pairs of
// neighbouring columns. Frequencies are double precision and the angle is reduced to one turn before it is rounded to fp32, so that
// positions far out keep the accuracy of the near ones.
#include "seq_math.cuh"

namespace plz {
namespace {

// cos and sin of position * frequency
__device__ __forceinline__ float2 turn(int pos, double freq) {
    const double a = (double)pos * freq;
    const double r = a - 6.283185307179586476925287 * rint(a * 0.159154943091895335768884);
    float s, c;
    sincosf((float)r, &s, &c);
    return make_float2(c, s);
}

struct LatentPrep {
    const void* proj; long long ldp; int off_q, off_c, off_r;
    const float* wq; const float* wc;
    void* cq; void* c; void* kr; long long c_batch, r_batch;
    const int* pos; const double* freq; int pairs; float m;
    int n, q_rank, R, dr, cap;
    float eps;
};

// one block per token; 256 threads
template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const LatentPrep p) {
    __shared__ float part[8];
    const long long r = blockIdx.x, b = r / p.n;
    pdl_launch_dependents();
    pdl_wait();
    const int at = *p.pos + (int)(r % p.n);
    if (at >= p.cap) return;                       // the host checks the capacity; never write past it
    const T* row = (const T*)p.proj + r * p.ldp;
    float sq = 0.f, sc = 0.f;
    for (int c = threadIdx.x; c < p.q_rank; c += 256) { const float v = to_f(row[p.off_q + c]); sq = fmaf(v, v, sq); }
    for (int c = threadIdx.x; c < p.R; c += 256) { const float v = to_f(row[p.off_c + c]); sc = fmaf(v, v, sc); }
    sq = block_sum<8>(sq, part);
    sc = block_sum<8>(sc, part);
    const float rq = 1.0f / sqrtf(sq / (float)p.q_rank + p.eps), rc = 1.0f / sqrtf(sc / (float)p.R + p.eps);
    T* qo = (T*)p.cq + r * p.q_rank;
    T* co = (T*)p.c + b * p.c_batch + (long long)at * p.R;
    for (int c = threadIdx.x; c < p.q_rank; c += 256) qo[c] = from_f<T>(to_f(row[p.off_q + c]) * rq * p.wq[c]);
    for (int c = threadIdx.x; c < p.R; c += 256) co[c] = from_f<T>(to_f(row[p.off_c + c]) * rc * p.wc[c]);
    if (p.dr > 0) {
        T* ko = (T*)p.kr + b * p.r_batch + (long long)at * p.dr;
        for (int i = threadIdx.x; i < p.pairs; i += 256) {
            const float2 t = turn(at, p.freq[i]);
            const float u = to_f(row[p.off_r + 2 * i]), v = to_f(row[p.off_r + 2 * i + 1]);
            ko[2 * i] = from_f<T>(p.m * (u * t.x - v * t.y));
            ko[2 * i + 1] = from_f<T>(p.m * (v * t.x + u * t.y));
        }
        for (int c = 2 * p.pairs + threadIdx.x; c < p.dr; c += 256) ko[c] = row[p.off_r + c];
    }
}

__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ float dot8(const float (&f)[8]) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s = fmaf(f[i], f[i], s);
    return s;
}

// The same for sizes that are multiples of 8 and 16-byte aligned rows (q_rank + R <= 16 * NT): a row's values stay in registers between
// the sums and the store, the key part is turned by the threads that the latents leave idle, or by the last ones.
template <typename T, int NT>
__global__ void __launch_bounds__(NT)
latent_prep8_kernel(const LatentPrep p) {
    constexpr int NW = NT / 32;
    __shared__ float part[2][NW];
    const long long r = blockIdx.x, b = r / p.n;
    const int tid = threadIdx.x, nq = p.q_rank >> 3, nc = nq + (p.R >> 3);
    float w[2][8];
#pragma unroll
    for (int i = 0; i < 2; ++i) {                  // norm weights do not depend on the previous kernel
        const int c = tid + i * NT;
        if (c < nc) load8(c < nq ? p.wq + c * 8 : p.wc + (c - nq) * 8, w[i]);
    }
    const int pair = NT - 1 - tid;                 // of the key part
    const double freq = pair < p.pairs ? p.freq[pair] : 0.0;
    pdl_launch_dependents();
    pdl_wait();
    const int at = *p.pos + (int)(r % p.n);
    if (at >= p.cap) return;                       // the host checks the capacity; never write past it
    const T* row = (const T*)p.proj + r * p.ldp;
    float x[2][8], sq = 0.f, sc = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int c = tid + i * NT;
        if (c < nc) {
            load8(c < nq ? row + p.off_q + c * 8 : row + p.off_c + (c - nq) * 8, x[i]);
            (c < nq ? sq : sc) += dot8(x[i]);
        }
    }
    T* ko = (T*)p.kr + b * p.r_batch + (long long)at * p.dr;
    if (pair < p.pairs) {
        const float u = to_f(row[p.off_r + 2 * pair]), v = to_f(row[p.off_r + 2 * pair + 1]);
        const float2 t = turn(at, freq);
        ko[2 * pair] = from_f<T>(p.m * (u * t.x - v * t.y));
        ko[2 * pair + 1] = from_f<T>(p.m * (v * t.x + u * t.y));
    }
    for (int c = 2 * p.pairs + tid; c < p.dr; c += NT) ko[c] = row[p.off_r + c];
    sq = warp_sum(sq);
    sc = warp_sum(sc);
    if ((tid & 31) == 0) { part[0][tid >> 5] = sq; part[1][tid >> 5] = sc; }
    __syncthreads();
    sq = sc = 0.f;
#pragma unroll
    for (int i = 0; i < NW; ++i) { sq += part[0][i]; sc += part[1][i]; }
    const float rq = 1.0f / sqrtf(sq / (float)p.q_rank + p.eps), rc = 1.0f / sqrtf(sc / (float)p.R + p.eps);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int c = tid + i * NT;
        if (c < nc) {
            const float f = c < nq ? rq : rc;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[i][e] = x[i][e] * f * w[i][e];
            if (c < nq) store8((T*)p.cq + r * p.q_rank + c * 8, x[i]);
            else store8((T*)p.c + b * p.c_batch + (long long)at * p.R + (c - nq) * 8, x[i]);
        }
    }
}

struct Rotate {
    const void* x; long long ldx, xh;
    void* out; long long ldo, oh;
    const int* pos; const double* freq; int pairs; float m;
    int n, H, dr;
};

// one block per token: the turns are computed once and serve all heads
template <typename T>
__global__ void __launch_bounds__(256)
rotate_kernel(const Rotate p) {
    extern __shared__ float2 cs[];
    const long long r = blockIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const int at = *p.pos + (int)(r % p.n);
    for (int i = threadIdx.x; i < p.pairs; i += 256) {
        const float2 t = turn(at, p.freq[i]);
        cs[i] = make_float2(p.m * t.x, p.m * t.y);
    }
    __syncthreads();
    const T* x = (const T*)p.x + r * p.ldx;
    T* o = (T*)p.out + r * p.ldo;
    const int half = (p.dr + 1) / 2;
    for (int e = threadIdx.x; e < p.H * half; e += 256) {
        const int h = e / half, i = e - h * half;
        const T* xi = x + h * p.xh + 2 * i;
        T* oi = o + h * p.oh + 2 * i;
        if (i < p.pairs) {
            const float u = to_f(xi[0]), v = to_f(xi[1]);
            oi[0] = from_f<T>(u * cs[i].x - v * cs[i].y);
            oi[1] = from_f<T>(v * cs[i].x + u * cs[i].y);
        } else {
            oi[0] = xi[0];
            if (2 * i + 1 < p.dr) oi[1] = xi[1];
        }
    }
}

// the same for parts that are multiples of 8 and 16-byte aligned: four pairs at a time
template <typename T>
__global__ void __launch_bounds__(256)
rotate8_kernel(const Rotate p) {
    extern __shared__ float2 cs[];
    const long long r = blockIdx.x;
    const double freq = (int)threadIdx.x < p.pairs ? p.freq[threadIdx.x] : 0.0;
    pdl_launch_dependents();
    pdl_wait();
    const int at = *p.pos + (int)(r % p.n), per = p.dr >> 3;
    for (int i = threadIdx.x; i < 4 * per; i += 256) {
        float2 t = make_float2(1.f, 0.f);
        if (i < p.pairs) {
            t = turn(at, i < 256 ? freq : p.freq[i]);
            t.x *= p.m; t.y *= p.m;
        }
        cs[i] = t;
    }
    __syncthreads();
    const T* x = (const T*)p.x + r * p.ldx;
    T* o = (T*)p.out + r * p.ldo;
    for (int e = threadIdx.x; e < p.H * per; e += 256) {
        const int h = e / per, i = e - h * per;
        float f[8], g[8];
        load8(x + h * p.xh + 8 * i, f);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 t = cs[4 * i + k];
            g[2 * k] = f[2 * k] * t.x - f[2 * k + 1] * t.y;
            g[2 * k + 1] = f[2 * k + 1] * t.x + f[2 * k] * t.y;
        }
        store8(o + h * p.oh + 8 * i, g);
    }
}

typedef __nv_bfloat16 bf;

}  // namespace

int launch_latent_prep(int dtype, const LatentPrepArgs& a, cudaStream_t stream) {
    const long long rows = (long long)a.B * a.n;
    if (rows <= 0) return PLZ_OK;
    const LatentPrep p = {a.proj, a.ldp, a.off_q, a.off_c, a.off_r, a.wq, a.wc, a.cq, a.c, a.kr, a.c_batch, a.r_batch, a.pos, a.freq, a.pairs, a.m,
                          a.n, a.q_rank, a.R, a.dr, a.cap, a.eps};
    const int per16 = dtype == 0 ? 8 : 4, both = a.q_rank + a.R;
    const uintptr_t ptrs = (uintptr_t)a.proj | (uintptr_t)a.wq | (uintptr_t)a.wc | (uintptr_t)a.cq | (uintptr_t)a.c;
    const bool vec = a.q_rank % 8 == 0 && a.R % 8 == 0 && a.off_q % 8 == 0 && a.off_c % 8 == 0 && a.ldp % per16 == 0 && a.c_batch % per16 == 0 && !(ptrs & 15);
    const dim3 grid((unsigned)rows);
    if (vec && both <= 16 * 128 && a.pairs <= 128) {
        if (dtype == 1) PLZ_LAUNCH_CHAIN((latent_prep8_kernel<float, 128>), grid, dim3(128), 0, stream, p);
        else PLZ_LAUNCH_CHAIN((latent_prep8_kernel<bf, 128>), grid, dim3(128), 0, stream, p);
    } else if (vec && both <= 16 * 256 && a.pairs <= 256) {
        if (dtype == 1) PLZ_LAUNCH_CHAIN((latent_prep8_kernel<float, 256>), grid, dim3(256), 0, stream, p);
        else PLZ_LAUNCH_CHAIN((latent_prep8_kernel<bf, 256>), grid, dim3(256), 0, stream, p);
    } else if (dtype == 1) PLZ_LAUNCH_CHAIN(latent_prep_kernel<float>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    else PLZ_LAUNCH_CHAIN(latent_prep_kernel<bf>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    return PLZ_OK;
}

int launch_rotate(int dtype, const RotateArgs& a, cudaStream_t stream) {
    const long long rows = (long long)a.B * a.n;
    if (rows <= 0) return PLZ_OK;
    const Rotate p = {a.x, a.ldx, a.xh, a.out, a.ldo, a.oh, a.pos, a.freq, a.pairs, a.m, a.n, a.H, a.dr};
    const size_t smem = (size_t)(a.dr / 2 + 1) * sizeof(float2);
    if (smem > 48 * 1024) { set_last_error("rotate: %d columns", a.dr); return PLZ_ERR_UNSUPPORTED; }
    const int per16 = dtype == 0 ? 8 : 4;
    const bool vec = a.dr % 8 == 0 && a.ldx % per16 == 0 && a.xh % per16 == 0 && a.ldo % per16 == 0 && a.oh % per16 == 0 && !(((uintptr_t)a.x | (uintptr_t)a.out) & 15);
    if (vec) {
        if (dtype == 1) PLZ_LAUNCH_CHAIN(rotate8_kernel<float>, dim3((unsigned)rows), dim3(256), smem, stream, p);
        else PLZ_LAUNCH_CHAIN(rotate8_kernel<bf>, dim3((unsigned)rows), dim3(256), smem, stream, p);
    } else if (dtype == 1) PLZ_LAUNCH_CHAIN(rotate_kernel<float>, dim3((unsigned)rows), dim3(256), smem, stream, p);
    else PLZ_LAUNCH_CHAIN(rotate_kernel<bf>, dim3((unsigned)rows), dim3(256), smem, stream, p);
    return PLZ_OK;
}

}  // namespace plz
