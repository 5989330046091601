// Workspace between the two launches of the chunked recurrences: per (sequence, head, chunk of 64 tokens) the operands of the scan as
// ready-made shared-memory images (bf16, 128-byte swizzle, hi and lo planes), so that the scan brings them in with two bulk copies.
#pragma once
#include "seq_math.cuh"

namespace plz {

constexpr int kC = 64;                     // tokens per chunk

// (x, y) -> bf16 pairs hi, lo with x ~ hi.x + lo.x
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16x2(x, y);
    lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}

// KB: 64-column blocks of the key dimension (1 or 2); R: rows of the first tile, 128 = -W over Q~, 64 = Q~ alone
//   A  [hi, lo][KB][R][64]   K-major B operand of S^T x (-W | Q~)^T
//      e^{b_C} fp32 [64 KB]
//   B  M [hi, lo][64][64] K-major, K~ [hi, lo][KB][64][64] MN-major
//   U0 fp32 [64][dvp]
template <int KB, int R>
struct ChunkWs {
    static constexpr uint32_t DK = 64 * KB;
    static constexpr uint32_t A_BLOCK = R * 128, A_PLANE = KB * A_BLOCK, A_BYTES = 2 * A_PLANE, DEC_BYTES = DK * 4;
    static constexpr uint32_t M_PLANE = kC * 128, K_PLANE = KB * kC * 128, B_BYTES = 2 * (M_PLANE + K_PLANE);
    static constexpr uint32_t OFF_DEC = A_BYTES, OFF_B = OFF_DEC + DEC_BYTES, OFF_K = OFF_B + 2 * M_PLANE, OFF_U = OFF_B + B_BYTES;
    static __host__ __device__ long long bytes(int dvp) { return (long long)OFF_U + (long long)kC * dvp * 4; }
    // byte of column c, row r of a tile with `rows` rows per 64-column block
    static __device__ __forceinline__ uint32_t at(uint32_t rows, uint32_t r, uint32_t c) {
        return (c >> 6) * (rows * 128u) + r * 128u + ((((c & 63u) >> 3) ^ (r & 7u)) << 4) + (c & 7u) * 2u;
    }
};
// columns c, c + 1 (c even) / c .. c + 3 (c a multiple of four) of one row, both planes
__device__ __forceinline__ void put_split(uint8_t* p, uint32_t plane, float x, float y) {
    uint32_t h, l;
    split2(x, y, h, l);
    *reinterpret_cast<uint32_t*>(p) = h;
    *reinterpret_cast<uint32_t*>(p + plane) = l;
}
__device__ __forceinline__ void put_split4(uint8_t* p, uint32_t plane, float x, float y, float z, float w) {
    uint2 h, l;
    split2(x, y, h.x, l.x);
    split2(z, w, h.y, l.y);
    *reinterpret_cast<uint2*>(p) = h;
    *reinterpret_cast<uint2*>(p + plane) = l;
}

struct ScanArgs {
    const uint8_t* ws; long long ws_stride;
    float* state; float* o;
    int B, n, t_begin, chunks, H, dk, dv, dvp;
};
// has_w: the gated delta rule; kb: key blocks of the workspace
int launch_chunk_scan(const ScanArgs& a, bool has_w, int kb, cudaStream_t stream);

}  // namespace plz
