// Shared by the two forms of attention over cached latents (latent_attention.cu, latent_attention_tc.cu).
#pragma once
#include "seq_math.cuh"

namespace plz {

constexpr float kLatLog2e = 1.4426950408889634f;
constexpr float kLatNegBig = -1.0e30f;
constexpr int kLatMaxSplits = 128;
constexpr int kLatTile = 128;          // keys per tile of the tensor-core form

struct LatentParams {
    int n, H, R, dr, splits;
    float scale;
    const float* sinks;
    // per query row (b * n * H + t * H + h) and split: unnormalised sum [R]; (running maximum in log2 units, sum of weights)
    float* ws_o; float* ws_ml;
};

bool latent_tc_fits(int R, int dr);
int latent_tc_rows(int rows, int R, int dr);          // query rows of one CTA of the tensor-core form
int launch_latent_tc(const LatentAttnArgs& a, const LatentParams& l, cudaStream_t stream);

}  // namespace plz
