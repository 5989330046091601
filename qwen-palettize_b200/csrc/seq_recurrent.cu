// Token-by-token form of the two linear recurrences, state fp32 [B, H, dk, dv] in HBM, read and written once per call:
//
//   decayed linear attention   S <- lambda_h S + k v^T ;                                   o = S^T q   (q, k, v = silu of the projections)
//   gated delta rule           S <- g S (rows) ; u = beta (v - S^T k) ; S <- S + k u^T ;   o = S^T q
//
// This form serves token decode (bound by streaming the state), short portions and the 32-bit mode. A warp holds 8 value columns
// x dk key rows in registers: lane = 8 * (key row group) + column, row group g owning rows g, g + 4, g + 8, ..., so a warp's access
// to the state is whole 32-byte sectors, a token's key and query are conflict-free broadcasts from shared memory, and the sums
// over the key dimension take two shuffles.
#include "seq_math.cuh"

namespace plz {
namespace {

constexpr int kTok = 8;      // tokens staged in shared memory at a time

struct RecParams {
    // DELTA: q, k [rows, G * dk], v [rows, H * dv], logg [rows, H * dk], beta [rows, H], all fp32.  else: T slices of the projections
    const void* q; const void* k; const void* v; long long ldq, ldk, ldv;
    const float* logg; const float* beta; const float* decay;
    float* S;
    float* o;                // [rows, H * dv]
    int n, H, G, dk, dv;
};

// RK: key rows of a thread (dk <= 4 * RK). T: type of q, k, v.
template <typename T, bool DELTA, int RK>
__global__ void __launch_bounds__(128)
recurrent_kernel(const RecParams p) {
    extern __shared__ float sm[];
    constexpr int DK = 4 * RK;
    float* sq = sm;                      // [kTok][DK], zero past dk
    float* sk = sq + kTok * DK;
    float* sg = sk + kTok * DK;          // DELTA only
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, kg = lane >> 3;
    const int col = (int)blockIdx.x * 32 + warp * 8 + (lane & 7);
    const int h = blockIdx.y;
    const long long b = blockIdx.z;
    const int hk = DELTA ? h / (p.H / p.G) : h;
    const bool live = col < p.dv;
    float* Sp = p.S + ((b * p.H + h) * p.dk) * (long long)p.dv + col;
    pdl_launch_dependents();
    pdl_wait();
    float s[RK];
#pragma unroll
    for (int i = 0; i < RK; ++i) {
        const int r = i * 4 + kg;
        s[i] = (live && r < p.dk) ? Sp[(long long)r * p.dv] : 0.f;
    }
    const float lam = DELTA ? 0.f : p.decay[h];
    for (int t0 = 0; t0 < p.n; t0 += kTok) {
        const int nt = min(kTok, p.n - t0);
        __syncthreads();
        for (int e = threadIdx.x; e < nt * DK; e += 128) {
            const int t = e / DK, c = e - t * DK;
            const long long row = b * p.n + t0 + t;
            float q = 0.f, k = 0.f, g = 0.f;
            if (c < p.dk) {
                q = to_f(((const T*)p.q)[row * p.ldq + (long long)hk * p.dk + c]);
                k = to_f(((const T*)p.k)[row * p.ldk + (long long)hk * p.dk + c]);
                if (DELTA) g = expf(p.logg[(row * p.H + h) * p.dk + c]);
                else { q = silu_f(q); k = silu_f(k); }
            }
            sq[t * DK + c] = q;
            sk[t * DK + c] = k;
            if (DELTA) sg[t * DK + c] = g;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const long long row = b * p.n + t0 + t;
            float v = live ? to_f(((const T*)p.v)[row * p.ldv + (long long)h * p.dv + col]) : 0.f;
            float acc = 0.f;
            if (DELTA) {
                float pred = 0.f;
#pragma unroll
                for (int i = 0; i < RK; ++i) {
                    s[i] *= sg[t * DK + i * 4 + kg];
                    pred = fmaf(s[i], sk[t * DK + i * 4 + kg], pred);
                }
                pred += __shfl_xor_sync(0xFFFFFFFFu, pred, 8);
                pred += __shfl_xor_sync(0xFFFFFFFFu, pred, 16);
                const float u = p.beta[row * p.H + h] * (v - pred);
#pragma unroll
                for (int i = 0; i < RK; ++i) {
                    s[i] = fmaf(sk[t * DK + i * 4 + kg], u, s[i]);
                    acc = fmaf(s[i], sq[t * DK + i * 4 + kg], acc);
                }
            } else {
                v = silu_f(v);
#pragma unroll
                for (int i = 0; i < RK; ++i) {
                    s[i] = fmaf(sk[t * DK + i * 4 + kg], v, lam * s[i]);
                    acc = fmaf(s[i], sq[t * DK + i * 4 + kg], acc);
                }
            }
            acc += __shfl_xor_sync(0xFFFFFFFFu, acc, 8);
            acc += __shfl_xor_sync(0xFFFFFFFFu, acc, 16);
            if (live && kg == 0) p.o[(row * p.H + h) * (long long)p.dv + col] = acc;
        }
    }
#pragma unroll
    for (int i = 0; i < RK; ++i) {
        const int r = i * 4 + kg;
        if (live && r < p.dk) Sp[(long long)r * p.dv] = s[i];
    }
}

template <typename T, bool DELTA, int RK>
int launch_rk(const RecParams& p, int B, cudaStream_t stream) {
    const size_t smem = (size_t)(DELTA ? 3 : 2) * kTok * 4 * RK * sizeof(float);
    PLZ_LAUNCH_CHAIN((recurrent_kernel<T, DELTA, RK>), dim3((p.dv + 31) / 32, p.H, B), dim3(128), smem, stream, p);
    return PLZ_OK;
}
template <typename T, bool DELTA>
int launch_any(const RecParams& p, int B, cudaStream_t stream) {
    if (p.dk <= 32) return launch_rk<T, DELTA, 8>(p, B, stream);
    if (p.dk <= 64) return launch_rk<T, DELTA, 16>(p, B, stream);
    if (p.dk <= 128) return launch_rk<T, DELTA, 32>(p, B, stream);
    if (p.dk <= 256) return launch_rk<T, DELTA, 64>(p, B, stream);
    set_last_error("recurrence: key size %d (at most 256)", p.dk);
    return PLZ_ERR_UNSUPPORTED;
}

}  // namespace

int launch_recurrent_decay(int dtype, const DecayAttnArgs& a, cudaStream_t stream) {
    if (a.B <= 0 || a.n <= 0) return PLZ_OK;
    RecParams p = {};
    p.q = a.q; p.k = a.k; p.v = a.v; p.ldq = p.ldk = p.ldv = a.ld; p.decay = a.decay; p.S = a.state; p.o = a.o;
    p.n = a.n; p.H = a.H; p.G = a.H; p.dk = a.dk; p.dv = a.dv;
    return dtype == 1 ? launch_any<float, false>(p, a.B, stream) : launch_any<__nv_bfloat16, false>(p, a.B, stream);
}

int launch_recurrent_delta(const DeltaRuleArgs& a, cudaStream_t stream) {
    if (a.B <= 0 || a.n <= 0) return PLZ_OK;
    RecParams p = {};
    p.q = a.q; p.k = a.k; p.v = a.v; p.ldq = p.ldk = (long long)a.G * a.dk; p.ldv = (long long)a.H * a.dv;
    p.logg = a.logg; p.beta = a.beta; p.S = a.state; p.o = a.o;
    p.n = a.n; p.H = a.H; p.G = a.G; p.dk = a.dk; p.dv = a.dv;
    return launch_any<float, true>(p, a.B, stream);
}

}  // namespace plz
