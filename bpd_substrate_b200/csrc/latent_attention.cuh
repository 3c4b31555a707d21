// Attention over a cache of latents: keys and values of all heads are linear maps of one latent row per token, and one
// rotated key part per token is shared by the heads.
#pragma once
#include "decoder_device.cuh"

namespace bpdq {

// Cache row of a token: [latent, rank_pad | rotated key part, rot_pad], activation type.
struct LatentShape {
    int heads, dim_pad, value_pad, rank, rank_pad, rot_dims, rot_pad;
    int q_rank, q_rank_pad;
    const float* rot_freq;      // [rot_dims / 2]
    float scale, eps;
    __host__ __device__ int row() const { return rank_pad + rot_pad; }
    __host__ __device__ int q_head() const { return dim_pad + rot_pad; }
};

// u [T][ld_u] = [query latent, q_rank_pad | latent, rank_pad | rotated key part, rot_pad]: RMS norms with weights, the key
// part rotated; the query latent to cq [T][q_rank_pad], the rest to cache rows *pos + t (cache null: queries only).
int latent_prepare(const LatentShape& p, const void* u, int ld_u, const float* q_norm, const float* kv_norm, void* cq, void* cache,
                   const int* pos, int T, bool act_bf16, cudaStream_t s);

// Buffers of one attention call.
struct LatentBuffers {
    void* q_latent;             // [T][heads][row()]
    float* partial;             // latent_partial_floats()
    void* expanded;             // [context][heads * (dim_pad + value_pad)]
};
// q [T][heads * q_head()] (not rotated yet) against cache rows 0 .. *pos + t; o [T][heads * value_pad].
// w_uk [heads * dim_pad][rank_pad], then w_uv [heads * value_pad][rank_pad].  context = *pos + T where keys
// and values are expanded (latent_expands); otherwise it is not used, the kernels read *pos.
int latent_attention(const LatentShape& p, void* q, const bf16* w_ukv, const void* cache, void* o, const LatentBuffers& b, const int* pos,
                     int T, int context, bool act_bf16, cudaStream_t s);

bool latent_expands(const LatentShape& p, int T, bool act_bf16);
size_t latent_partial_floats(const LatentShape& p, int T, bool act_bf16);

}  // namespace bpdq
