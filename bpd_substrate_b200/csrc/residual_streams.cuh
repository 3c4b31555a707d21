// Residual streams joined by hyper-connections, and the RMS norm that reads them.
#pragma once
#include "decoder_device.cuh"
#include "../../include/bpdq.h"

namespace bpdq {

static_assert(kMaxStreams == BPDQ_MAX_STREAMS, "descriptors and kernels agree");

// Per token: the sublayer's output y enters the streams x [T][m.n][width_pad] (or, with a table, the streams start as
// embed_scale times the token's row); u = sum_t next[t] x_t goes to `u` (fp32) and its RMS norm with norm_w to `h`
// (activation type), each when given.
struct StreamStep {
    const float* y;             // [T][width_pad]
    const bf16* table;          // [vocab][width_pad] or null
    const int32_t* tokens;      // [T]
    float embed_scale;
    int vocab;
    float* x;
    StreamMix m;
    const float* norm_w;
    float eps;
    int width, width_pad;
    void* h;                    // [T][width_pad]
    float* u;                   // [T][width_pad]
};
// The descriptor's matrix and shares, with `next` the weights of the sublayer that reads afterwards.
static inline StreamMix stream_mix(const bpdq_stream_mix& d, int streams, const float* next)
{
    StreamMix m = {};
    m.n = streams;
    for (int i = 0; i < streams; i++) {
        for (int j = 0; j < streams; j++) m.mix[i][j] = d.mix[i * BPDQ_MAX_STREAMS + j];
        m.out[i] = d.out[i];
        m.next[i] = next[i];
    }
    return m;
}
int stream_step(const StreamStep& p, int T, bool act_bf16, cudaStream_t s);

// out [T][width] = sum of the streams.
int stream_sum(const float* x, int streams, int width, int width_pad, float* out, int T, cudaStream_t s);

}  // namespace bpdq
