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

typedef __nv_bfloat16 bf;

}  // namespace

int launch_latent_prep(int dtype, const LatentPrepArgs& a, cudaStream_t stream) {
    const long long rows = (long long)a.B * a.n;
    if (rows <= 0) return PLZ_OK;
    const LatentPrep p = {a.proj, a.ldp, a.off_q, a.off_c, a.off_r, a.wq, a.wc, a.cq, a.c, a.kr, a.c_batch, a.r_batch, a.pos, a.freq, a.pairs, a.m,
                          a.n, a.q_rank, a.R, a.dr, a.cap, a.eps};
    if (dtype == 1) PLZ_LAUNCH_CHAIN(latent_prep_kernel<float>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    else PLZ_LAUNCH_CHAIN(latent_prep_kernel<bf>, dim3((unsigned)rows), dim3(256), 0, stream, p);
    return PLZ_OK;
}

int launch_rotate(int dtype, const RotateArgs& a, cudaStream_t stream) {
    const long long rows = (long long)a.B * a.n;
    if (rows <= 0) return PLZ_OK;
    const Rotate p = {a.x, a.ldx, a.xh, a.out, a.ldo, a.oh, a.pos, a.freq, a.pairs, a.m, a.n, a.H, a.dr};
    const size_t smem = (size_t)a.pairs * sizeof(float2);
    if (smem > 48 * 1024) { set_last_error("rotate: %d pairs", a.pairs); return PLZ_ERR_UNSUPPORTED; }
    if (dtype == 1) PLZ_LAUNCH_CHAIN(rotate_kernel<float>, dim3((unsigned)rows), dim3(256), smem, stream, p);
    else PLZ_LAUNCH_CHAIN(rotate_kernel<bf>, dim3((unsigned)rows), dim3(256), smem, stream, p);
    return PLZ_OK;
}

}  // namespace plz
