// Attention with key and value heads shared by groups of query heads, over cached rows.
#pragma once
#include "decoder_device.cuh"

namespace bpdq {

// A position sees itself and what came before, with `chunk` only from the start of its chunk on (chunks of that many
// positions from position 0).  score = scale q.k, with `cap` then cap tanh(score / cap); `sink` adds a score of 0 without a
// value to the softmax.  Position i is cached in row i mod rows: [groups][dim_pad] keys, then [groups][value_pad] values.
struct GroupedShape {
    int heads, groups, dim, dim_pad, value_pad, chunk, rows, sink;
    float scale, cap, eps;
    __host__ __device__ int row() const { return groups * (dim_pad + value_pad); }
    __host__ __device__ int share() const { return heads / groups; }
    __host__ __device__ int q_width() const { return heads * dim_pad; }
    __host__ __device__ int first_seen(int i) const { return chunk > 0 ? i / chunk * chunk : 0; }
};

// u [T][ld_u] = queries [heads][dim_pad], then (cache given) keys [groups][dim_pad] and values [groups][value_pad]: queries and
// keys over their root mean square (per head, over dim), queries in place, keys and values to cache rows of *pos + t.
int grouped_prepare(const GroupedShape& p, void* u, int ld_u, void* cache, const int* pos, int T, bool act_bf16, cudaStream_t s);

// Normed queries of u against the cache, which holds positions up to *pos + T - 1; o [T][heads * value_pad].
int grouped_attention(const GroupedShape& p, const void* u, int ld_u, const void* cache, void* o, const int* pos, int T, bool act_bf16,
                      cudaStream_t s);

}  // namespace bpdq
