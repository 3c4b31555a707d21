// Residual streams: one CTA per token carries a sublayer's output into all streams, forms the next sublayer's input from
// them and norms it, so that a prompt's streams go through HBM once per sublayer.  (One-token steps do the first two in the
// epilogue of the product that ends the sublayer and the norm in the product that begins the next one: linear.cu.)
#include "residual_streams.cuh"
#include "launch.cuh"
#include "../../include/bpdq.h"

namespace bpdq {

// Thread = four columns, NJ times; NS: the most streams.
template <typename A, int NS, int NJ>
__global__ void __launch_bounds__(1024) k_stream_step(const __grid_constant__ StreamStep p, int* err)
{
    __shared__ float s_sum[32];
    pdl_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = p.m.n;
    float4 w[NJ];
#pragma unroll
    for (int j = 0; j < NJ; j++) {
        const int c = 4 * (tid + blockDim.x * j);
        w[j] = (p.h && c < p.width_pad) ? *reinterpret_cast<const float4*>(p.norm_w + c) : make_float4(0, 0, 0, 0);
    }
    pdl_wait();
    float* x = p.x + (size_t)t * n * p.width_pad;
    const bf16* row = nullptr;
    if (p.table) {
        const int tok = p.tokens[t];
        if (tok >= 0 && tok < p.vocab) row = p.table + (size_t)tok * p.width_pad;
        else if (tid == 0 && err) atomicCAS(err, 0, 21);        // no such row: nothing is read, code 21 is recorded
    }
    float4 u[NJ];
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; j++) {
        const int c = 4 * (tid + blockDim.x * j);
        u[j] = make_float4(0, 0, 0, 0);
        if (c >= p.width_pad) continue;
        float4 old[NS], y = make_float4(0, 0, 0, 0);
        if (p.table) {
            if (row) y = act_load4(row + c);
            y = make_float4(y.x * p.embed_scale, y.y * p.embed_scale, y.z * p.embed_scale, y.w * p.embed_scale);
        } else {
            y = *reinterpret_cast<const float4*>(p.y + (size_t)t * p.width_pad + c);
#pragma unroll
            for (int i = 0; i < NS; i++)
                old[i] = i < n ? *reinterpret_cast<const float4*>(x + (size_t)i * p.width_pad + c) : make_float4(0, 0, 0, 0);
        }
#pragma unroll
        for (int i = 0; i < NS; i++) {
            if (i >= n) break;
            float4 r = y;
            if (!p.table) {
                const float o = p.m.out[i];
                r = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
                for (int k = 0; k < NS; k++) {
                    const float f = p.m.mix[k][i];      // zero beyond the last stream
                    r.x = fmaf(f, old[k].x, r.x); r.y = fmaf(f, old[k].y, r.y); r.z = fmaf(f, old[k].z, r.z); r.w = fmaf(f, old[k].w, r.w);
                }
            }
            *reinterpret_cast<float4*>(x + (size_t)i * p.width_pad + c) = r;
            const float g = p.m.next[i];
            u[j].x = fmaf(g, r.x, u[j].x); u[j].y = fmaf(g, r.y, u[j].y); u[j].z = fmaf(g, r.z, u[j].z); u[j].w = fmaf(g, r.w, u[j].w);
        }
        if (p.u) *reinterpret_cast<float4*>(p.u + (size_t)t * p.width_pad + c) = u[j];
        sum = fmaf(u[j].x, u[j].x, sum); sum = fmaf(u[j].y, u[j].y, sum); sum = fmaf(u[j].z, u[j].z, sum); sum = fmaf(u[j].w, u[j].w, sum);
    }
    if (!p.h) return;
    sum = warp_sum(sum);
    if (lane == 0) s_sum[warp] = sum;
    __syncthreads();
    sum = warp_sum(lane < (int)(blockDim.x >> 5) ? s_sum[lane] : 0.0f);
    const float f = 1.0f / sqrtf(sum / (float)p.width + p.eps);
#pragma unroll
    for (int j = 0; j < NJ; j++) {
        const int c = 4 * (tid + blockDim.x * j);
        if (c < p.width_pad)
            act_store4(reinterpret_cast<A*>(p.h) + (size_t)t * p.width_pad + c,
                       make_float4(u[j].x * f * w[j].x, u[j].y * f * w[j].y, u[j].z * f * w[j].z, u[j].w * f * w[j].w));
    }
}

template <typename A, int NJ>
static int launch_stream_step(const StreamStep& p, int T, cudaStream_t s)
{
    int threads = (p.width_pad / 4 + 32 * NJ - 1) / (32 * NJ) * 32;
    if (threads > 1024) return latch(BPDQ_ERR_RANGE);
    if (p.m.n <= 2) return launch_ordered(k_stream_step<A, 2, NJ>, T, threads, 0, s, p, device_error_flag());
    if (p.m.n <= 4) return launch_ordered(k_stream_step<A, 4, NJ>, T, threads, 0, s, p, device_error_flag());
    return launch_ordered(k_stream_step<A, kMaxStreams, NJ>, T, threads, 0, s, p, device_error_flag());
}

int stream_step(const StreamStep& p, int T, bool act_bf16, cudaStream_t s)
{
    if (T < 1 || p.m.n < 1 || p.m.n > kMaxStreams || p.width < 1 || p.width_pad < p.width || p.width_pad % 4 || !p.x || (p.h && !p.norm_w) ||
        (p.table ? !p.tokens : !p.y))
        return latch(BPDQ_ERR_ARG);
    if (p.width_pad <= 4096) return act_bf16 ? launch_stream_step<bf16, 1>(p, T, s) : launch_stream_step<float, 1>(p, T, s);
    return act_bf16 ? launch_stream_step<bf16, 4>(p, T, s) : launch_stream_step<float, 4>(p, T, s);
}

__global__ void __launch_bounds__(256) k_stream_sum(const float* x, int streams, int width, int width_pad, float* out, int T)
{
    pdl_launch_dependents();
    pdl_wait();
    const long total = (long)T * width;
    for (long u = (long)blockIdx.x * blockDim.x + threadIdx.x; u < total; u += (long)gridDim.x * blockDim.x) {
        const long t = u / width;
        const float* p = x + (size_t)t * streams * width_pad + (u - t * width);
        float v = 0.0f;
        for (int i = 0; i < streams; i++) v += p[(size_t)i * width_pad];
        out[u] = v;
    }
}

int stream_sum(const float* x, int streams, int width, int width_pad, float* out, int T, cudaStream_t s)
{
    return launch_ordered(k_stream_sum, grid_1d((long)T * width), 256, 0, s, x, streams, width, width_pad, out, T);
}

}  // namespace bpdq

using namespace bpdq;

extern "C" {

int bpd_stream_step_cuda(const float* y, float* x, const bpdq_stream_mix* mix, int streams, const float* norm_w, float eps, int n_tokens, int width,
                         int width_pad, void* h, float* u, int act_bf16, void* stream)
{
    if (n_tokens < 0 || !mix || !y || !x) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (streams < 1 || streams > kMaxStreams) return latch(BPDQ_ERR_RANGE);
    StreamStep p = {};
    p.y = y;
    p.x = x;
    p.m = stream_mix(*mix, streams, mix->in);
    p.norm_w = norm_w;
    p.eps = eps;
    p.width = width;
    p.width_pad = width_pad;
    p.h = h;
    p.u = u;
    return stream_step(p, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

}  // extern "C"
