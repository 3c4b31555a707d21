// Latent attention.
//
// Two orders of the same products.  Few queries (decoding, short portions) and fp32 runs work on the latents
// themselves: W_uk is applied to the queries, scores and weighted sums run over the cached rows (read once for all
// heads), W_uv is applied to the sums.  A long portion of a prompt expands the context's keys and values once (one
// matrix product) and attends head by head.
//
//   k_latent_prepare       norms of the two latents, rotation of the key part, cache rows
//   k_latent_queries       q . W_uk per head, rotation of the query part
//   k_latent_attn_mma      bf16: rows = (token, head) pairs in tiles of 16 or 32, keys split over CTAs, mma.sync; scores and
//                          softmax fp32, weights enter the product as the sum of two bf16 numbers
//   k_latent_attn_rows     fp32 (and bf16 sizes beyond the tile kernel's shared memory): a warp per row
//   k_latent_values        joins the splits and applies W_uv
//   k_expanded_attn_mma    bf16 prompts: 64 queries of a head per CTA against expanded keys and values
#include "latent_attention.cuh"
#include "launch.cuh"
#include "mma_device.cuh"
#include "../../include/bpdq.h"

namespace bpdq {

constexpr float kLog2e = 1.44269504088896340736f;
constexpr int kKeyBlock = 64;

// ------------------------------------------------------------------ latents and cache rows

// Query latents of up to 2048 and latents of up to 1024: one CTA per token, the row in registers, the norms' weights fetched
// before the launch ahead has finished, the key part turned while the sums are joined.
template <typename A>
__global__ void __launch_bounds__(256) k_latent_prepare_regs(LatentShape p, const A* u, int ld_u, const float* __restrict__ q_norm,
                                                             const float* __restrict__ kv_norm, A* cq, A* cache, const int* pos_p)
{
    __shared__ float2 s_sum[8];
    pdl_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x;
    float q[8], qw[8], c[4], cw[4];
#pragma unroll
    for (int j = 0; j < 8; j++) qw[j] = tid + 256 * j < p.q_rank ? q_norm[tid + 256 * j] : 0.0f;
#pragma unroll
    for (int j = 0; j < 4; j++) cw[j] = (cache && tid + 256 * j < p.rank) ? kv_norm[tid + 256 * j] : 0.0f;
    const bool turns = cache && tid < p.rot_pad / 2 && 2 * tid < p.rot_dims;
    const float freq = turns ? p.rot_freq[tid] : 0.0f;
    pdl_wait();
    const int pos = *pos_p + t;
    const A* row = u + (size_t)t * ld_u;
    const A* lat = row + p.q_rank_pad;
    float a = 0.0f, b = 0.0f;
#pragma unroll
    for (int j = 0; j < 8; j++) q[j] = tid + 256 * j < p.q_rank ? act_load(row + tid + 256 * j) : 0.0f;
#pragma unroll
    for (int j = 0; j < 4; j++) c[j] = (cache && tid + 256 * j < p.rank) ? act_load(lat + tid + 256 * j) : 0.0f;
    if (turns) {
        a = act_load(lat + p.rank_pad + 2 * tid);
        b = act_load(lat + p.rank_pad + 2 * tid + 1);
    }
    float sq = 0.0f, sc = 0.0f;
#pragma unroll
    for (int j = 0; j < 8; j++) sq = fmaf(q[j], q[j], sq);
#pragma unroll
    for (int j = 0; j < 4; j++) sc = fmaf(c[j], c[j], sc);
    sq = warp_sum(sq);
    sc = warp_sum(sc);
    if ((tid & 31) == 0) s_sum[tid >> 5] = make_float2(sq, sc);
    if (turns) {
        float sn, cs;
        sincosf((float)pos * freq, &sn, &cs);
        const float x = a;
        a = x * cs - b * sn;
        b = b * cs + x * sn;
    }
    A* dst = cache ? cache + (size_t)pos * p.row() : nullptr;
    if (cache && tid < p.rot_pad / 2) {
        dst[p.rank_pad + 2 * tid] = act_from<A>(a);
        dst[p.rank_pad + 2 * tid + 1] = act_from<A>(b);
    }
    __syncthreads();
    sq = sc = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) { sq += s_sum[i].x; sc += s_sum[i].y; }
    const float fq = 1.0f / sqrtf(sq / (float)p.q_rank + p.eps), fc = 1.0f / sqrtf(sc / (float)p.rank + p.eps);
#pragma unroll
    for (int j = 0; j < 8; j++)
        if (tid + 256 * j < p.q_rank_pad) cq[(size_t)t * p.q_rank_pad + tid + 256 * j] = act_from<A>(q[j] * fq * qw[j]);
    if (!cache) return;
#pragma unroll
    for (int j = 0; j < 4; j++)
        if (tid + 256 * j < p.rank_pad) dst[tid + 256 * j] = act_from<A>(c[j] * fc * cw[j]);
}

// Any sizes: one CTA per token.
template <typename A>
__global__ void __launch_bounds__(256) k_latent_prepare(LatentShape p, const A* u, int ld_u, const float* __restrict__ q_norm,
                                                        const float* __restrict__ kv_norm, A* cq, A* cache, const int* pos_p)
{
    __shared__ float s_q[8], s_c[8];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, pos = *pos_p + t;
    const A* row = u + (size_t)t * ld_u;
    const A* lat = row + p.q_rank_pad;
    float sq = 0.0f, sc = 0.0f;
#pragma unroll 8
    for (int i = tid; i < p.q_rank; i += 256) { const float v = act_load(row + i); sq = fmaf(v, v, sq); }
    if (cache)
#pragma unroll 4
        for (int i = tid; i < p.rank; i += 256) { const float v = act_load(lat + i); sc = fmaf(v, v, sc); }
    sq = warp_sum(sq);
    sc = warp_sum(sc);
    if ((tid & 31) == 0) { s_q[tid >> 5] = sq; s_c[tid >> 5] = sc; }
    __syncthreads();
    sq = sc = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) { sq += s_q[i]; sc += s_c[i]; }
    const float fq = 1.0f / sqrtf(sq / (float)p.q_rank + p.eps);
#pragma unroll 8
    for (int i = tid; i < p.q_rank_pad; i += 256)
        cq[(size_t)t * p.q_rank_pad + i] = act_from<A>(i < p.q_rank ? act_load(row + i) * fq * q_norm[i] : 0.0f);
    if (!cache) return;
    const float fc = 1.0f / sqrtf(sc / (float)p.rank + p.eps);
    A* dst = cache + (size_t)pos * p.row();
    for (int i = tid; i < p.rank_pad; i += 256) dst[i] = act_from<A>(i < p.rank ? act_load(lat + i) * fc * kv_norm[i] : 0.0f);
    const A* rot = lat + p.rank_pad;
    for (int i = tid; i < p.rot_pad / 2; i += 256) {
        float a = 0.0f, b = 0.0f;
        if (2 * i < p.rot_dims) {
            float sn, cs;
            sincosf((float)pos * p.rot_freq[i], &sn, &cs);
            const float x = act_load(rot + 2 * i), y = act_load(rot + 2 * i + 1);
            a = x * cs - y * sn;
            b = y * cs + x * sn;
        }
        dst[p.rank_pad + 2 * i] = act_from<A>(a);
        dst[p.rank_pad + 2 * i + 1] = act_from<A>(b);
    }
}

int latent_prepare(const LatentShape& p, const void* u, int ld_u, const float* q_norm, const float* kv_norm, void* cq, void* cache,
                   const int* pos, int T, bool act_bf16, cudaStream_t s)
{
    if (p.q_rank_pad <= 2048 && p.rank_pad <= 1024 && p.rot_pad <= 512) {
        if (act_bf16) return launch_ordered(k_latent_prepare_regs<bf16>, T, 256, 0, s, p, (const bf16*)u, ld_u, q_norm, kv_norm, (bf16*)cq, (bf16*)cache, pos);
        return launch_ordered(k_latent_prepare_regs<float>, T, 256, 0, s, p, (const float*)u, ld_u, q_norm, kv_norm, (float*)cq, (float*)cache, pos);
    }
    if (act_bf16) return launch_ordered(k_latent_prepare<bf16>, T, 256, 0, s, p, (const bf16*)u, ld_u, q_norm, kv_norm, (bf16*)cq, (bf16*)cache, pos);
    return launch_ordered(k_latent_prepare<float>, T, 256, 0, s, p, (const float*)u, ld_u, q_norm, kv_norm, (float*)cq, (float*)cache, pos);
}

// ------------------------------------------------------------------ queries in latent space

// grid (rank columns / 128, heads, tokens / TT), 256 threads: sixteen lanes read 128 columns of a row of W_uk, sixteen
// rows at a time; the first eight rounds of weights are requested before the launch ahead has finished.
template <typename A, int TT>
__global__ void __launch_bounds__(256) k_latent_queries(LatentShape p, const A* q, const bf16* __restrict__ w_uk, A* out, const int* pos_p, int T)
{
    extern __shared__ float sq[];       // [TT][dim_pad], then [16][132] partial sums
    float* red = sq + TT * p.dim_pad;
    pdl_launch_dependents();
    const int h = blockIdx.y, t0 = blockIdx.z * TT, tid = threadIdx.x;
    const int n_t = T - t0 < TT ? T - t0 : TT;
    const int c = blockIdx.x * 128 + 8 * (tid & 15), phase = tid >> 4;
    const bool live = c < p.rank_pad;
    const bf16* w = w_uk + (size_t)h * p.dim_pad * p.rank_pad + (live ? c : 0);
    constexpr int kAhead = 8;
    uint4 u[kAhead];
    const int rounds = p.dim_pad / 16;
#pragma unroll
    for (int i = 0; i < kAhead; i++)
        u[i] = (live && i < rounds) ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)(phase + 16 * i) * p.rank_pad)) : make_uint4(0, 0, 0, 0);
    pdl_wait();
    const int ldq = p.heads * p.q_head();
    for (int i = tid; i < TT * p.dim_pad; i += 256) {
        const int t = i / p.dim_pad, d = i - t * p.dim_pad;
        sq[i] = t < n_t ? act_load(q + (size_t)(t0 + t) * ldq + h * p.q_head() + d) : 0.0f;
    }
    __syncthreads();
    float acc[TT][8] = {};
    auto add = [&](const uint4& v, int d) {
        const float f[8] = {bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y), bf_lo(v.z), bf_hi(v.z), bf_lo(v.w), bf_hi(v.w)};
#pragma unroll
        for (int t = 0; t < TT; t++) {
            const float x = sq[t * p.dim_pad + d];
#pragma unroll
            for (int j = 0; j < 8; j++) acc[t][j] = fmaf(f[j], x, acc[t][j]);
        }
    };
#pragma unroll
    for (int i = 0; i < kAhead; i++)
        if (i < rounds) add(u[i], phase + 16 * i);
    for (int i = kAhead; i < rounds; i++)
        add(live ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)(phase + 16 * i) * p.rank_pad)) : make_uint4(0, 0, 0, 0), phase + 16 * i);
#pragma unroll
    for (int t = 0; t < TT; t++) {
        if (t >= n_t) break;
        *reinterpret_cast<float4*>(red + phase * 132 + 8 * (tid & 15)) = make_float4(acc[t][0], acc[t][1], acc[t][2], acc[t][3]);
        *reinterpret_cast<float4*>(red + phase * 132 + 8 * (tid & 15) + 4) = make_float4(acc[t][4], acc[t][5], acc[t][6], acc[t][7]);
        __syncthreads();
        const int col = blockIdx.x * 128 + tid;
        if (tid < 128 && col < p.rank_pad) {
            float v = 0.0f;
#pragma unroll
            for (int i = 0; i < 16; i++) v += red[i * 132 + tid];
            out[((size_t)(t0 + t) * p.heads + h) * p.row() + col] = act_from<A>(v);
        }
        __syncthreads();
    }
    if (blockIdx.x == 0) {
        const int pairs = p.rot_pad / 2;
        for (int i = tid; i < n_t * pairs; i += 256) {
            const int t = i / pairs, j = i - t * pairs;
            const A* src = q + (size_t)(t0 + t) * ldq + h * p.q_head() + p.dim_pad + 2 * j;
            A* dst = out + ((size_t)(t0 + t) * p.heads + h) * p.row() + p.rank_pad + 2 * j;
            float a = 0.0f, b = 0.0f;
            if (2 * j < p.rot_dims) {
                float sn, cs;
                sincosf((float)(*pos_p + t0 + t) * p.rot_freq[j], &sn, &cs);
                const float x = act_load(src), y = act_load(src + 1);
                a = x * cs - y * sn;
                b = y * cs + x * sn;
            }
            dst[0] = act_from<A>(a);
            dst[1] = act_from<A>(b);
        }
    }
}

template <typename A, int TT>
static int launch_latent_queries(const LatentShape& p, const void* q, const bf16* w_uk, void* out, const int* pos, int T, cudaStream_t s)
{
    return launch_ordered(k_latent_queries<A, TT>, dim3((p.rank_pad + 127) / 128, p.heads, (T + TT - 1) / TT), 256,
                          (size_t)(TT * p.dim_pad + 16 * 132) * 4, s, p, (const A*)q, w_uk, (A*)out, pos, T);
}

// ------------------------------------------------------------------ attention over latents

// Keys are dealt to `splits` CTAs in whole blocks; short contexts leave the last CTAs without any.
__device__ __forceinline__ int keys_per_split(int context, int splits)
{
    const int blocks = (context + kKeyBlock - 1) / kKeyBlock;
    return (blocks + splits - 1) / splits * kKeyBlock;
}

// Partial results of (row, split): maximum (log2 units) and sum of weights of all splits side by side, then [rank_pad]
// unnormalised sums per split.
__host__ __device__ inline size_t partial_stride(int splits, int rank_pad) { return (size_t)splits * (rank_pad + 2) + 2 * (splits & 1); }
__device__ __forceinline__ float2* partial_stats(float* partial, long row, int splits, int rank_pad)
{
    return reinterpret_cast<float2*>(partial + (size_t)row * partial_stride(splits, rank_pad));
}
__device__ __forceinline__ float* partial_sums(float* partial, long row, int split, int splits, int rank_pad)
{
    return partial + (size_t)row * partial_stride(splits, rank_pad) + 2 * (splits + (splits & 1)) + (size_t)split * rank_pad;
}

template <int MT, int NTC>
struct LatentTile {
    static constexpr int kRows = 16 * MT, kCols = 64 * NTC, kLdP = kKeyBlock + 8, kLdS = kKeyBlock + 4;
    static size_t smem(int row)
    {
        return (size_t)(2 * kKeyBlock + kRows) * (row + 8) * 2 + (size_t)kRows * kLdS * 4 + 2 * (size_t)kRows * kLdP * 2 + 3 * kRows * 4;
    }
};

// grid (row tiles, splits, column slices of kCols).  Eight warps; scores: warp w takes keys 8 w .. 8 w + 7 of a block; sums: warp w
// takes columns 8 NTC w .. of the slice.
template <int MT, int NTC>
__global__ void __launch_bounds__(256, 1) k_latent_attn_mma(LatentShape p, const bf16* q, const bf16* cache, float* partial, const int* pos_p, int T)
{
    using S = LatentTile<MT, NTC>;
    constexpr int M = S::kRows, LDP = S::kLdP, LDS = S::kLdS, TPR = 256 / M;     // threads per row in the softmax
    extern __shared__ __align__(128) uint8_t smem[];
    const int row = p.row(), LD = row + 8;
    bf16* sK[2] = {reinterpret_cast<bf16*>(smem), reinterpret_cast<bf16*>(smem) + kKeyBlock * LD};
    bf16* sQ = sK[1] + kKeyBlock * LD;
    float* sS = reinterpret_cast<float*>(sQ + M * LD);
    bf16* sPh = reinterpret_cast<bf16*>(sS + M * LDS);
    bf16* sPl = sPh + M * LDP;
    float* sMax = reinterpret_cast<float*>(sPl + M * LDP);
    float* sSum = sMax + M;
    float* sAlpha = sSum + M;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
    const long rows = (long)T * p.heads, r0 = (long)blockIdx.x * M;
    const int col0 = blockIdx.z * S::kCols, splits = gridDim.y, split = blockIdx.y;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *pos_p;
    const int per = keys_per_split(pos + T, splits), k_begin = split * per;
    // the last key any row of this tile may see
    const long r_last = (r0 + M < rows ? r0 + M : rows) - 1;
    int k_end = pos + (int)(r_last / p.heads) + 1;
    if (k_end > k_begin + per) k_end = k_begin + per;
    const int units = row / 8;
    auto load_keys = [&](int k0, int b) {
        for (int i = tid; i < kKeyBlock * units; i += 256) {
            const int r = i / units, u = i - r * units, k = k0 + r;
            cp_async16(sK[b] + r * LD + 8 * u, cache + (size_t)(k < k_end ? k : k_end - 1) * row + 8 * u, k < k_end);
        }
        cp_async_commit();
    };
    if (k_begin < k_end) {
        for (int i = tid; i < M * units; i += 256) {
            const int r = i / units, u = i - r * units;
            const long g = r0 + r;
            cp_async16(sQ + r * LD + 8 * u, q + (size_t)(g < rows ? g : rows - 1) * row + 8 * u, g < rows);
        }
        load_keys(k_begin, 0);
    }
    if (tid < M) { sMax[tid] = -INFINITY; sSum[tid] = 0.0f; }
    float o[MT][NTC][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int n = 0; n < NTC; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[m][n][e] = 0.0f;
    const float scale = p.scale * kLog2e;
    int b = 0;
    for (int k0 = k_begin; k0 < k_end; k0 += kKeyBlock, b ^= 1) {
        cp_async_wait_all();
        __syncthreads();
        if (k0 + kKeyBlock < k_end) load_keys(k0 + kKeyBlock, b ^ 1);
        {
            float acc[MT][4];
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[m][e] = 0.0f;
            const bf16* kp = sK[b] + (8 * warp + (lane & 7)) * LD + 8 * (lane >> 3);
            const bf16* qp = sQ + (lane & 15) * LD + 8 * (lane >> 4);
            int d = 0;
            for (; d + 32 <= row; d += 32) {
                uint32_t bk[4];
                ldsm4(bk, kp + d);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    uint32_t a0[4], a1[4];
                    ldsm4(a0, qp + 16 * m * LD + d);
                    ldsm4(a1, qp + 16 * m * LD + d + 16);
                    mma_bf16(acc[m], a0, bk[0], bk[1]);
                    mma_bf16(acc[m], a1, bk[2], bk[3]);
                }
            }
            if (d < row) {      // sixteen left: the fragment's upper half would lie beyond the row
                uint32_t bk[4];
                ldsm4(bk, sK[b] + (8 * warp + (lane & 7)) * LD + d + 8 * ((lane >> 3) & 1));
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    uint32_t a0[4];
                    ldsm4(a0, qp + 16 * m * LD + d);
                    mma_bf16(acc[m], a0, bk[0], bk[1]);
                }
            }
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int e = 0; e < 4; e++) sS[(16 * m + g4 + 8 * (e >> 1)) * LDS + 8 * warp + 2 * t4 + (e & 1)] = acc[m][e];
        }
        __syncthreads();
        {
            const int r = tid / TPR, j = tid % TPR;
            const long g = r0 + r;
            const int last = g < rows ? pos + (int)(g / p.heads) : -1;      // the row's own position
            constexpr int KPT = kKeyBlock / TPR;
            float v[KPT], mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < KPT; i++) {
                const int k = k0 + KPT * j + i;
                v[i] = (k <= last && k < k_end) ? sS[r * LDS + KPT * j + i] * scale : -INFINITY;
                mx = fmaxf(mx, v[i]);
            }
#pragma unroll
            for (int w = 1; w < TPR; w <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, w));
            const float before = sMax[r], now = fmaxf(before, mx);
            const float base = now == -INFINITY ? 0.0f : now;
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < KPT; i += 2) {
                const float e0 = exp2f(v[i] - base), e1 = exp2f(v[i + 1] - base);
                uint32_t hi, lo;
                split_bf16(e0, e1, hi, lo);
                *reinterpret_cast<uint32_t*>(sPh + r * LDP + KPT * j + i) = hi;
                *reinterpret_cast<uint32_t*>(sPl + r * LDP + KPT * j + i) = lo;
                sum += e0 + e1;
            }
#pragma unroll
            for (int w = 1; w < TPR; w <<= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, w);
            __syncwarp();
            if (j == 0) {
                const float alpha = exp2f(before - base);
                sAlpha[r] = alpha;
                sSum[r] = sSum[r] * alpha + sum;
                sMax[r] = now;
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; m++) {
            const float a0 = sAlpha[16 * m + g4], a1 = sAlpha[16 * m + g4 + 8];
#pragma unroll
            for (int n = 0; n < NTC; n++) { o[m][n][0] *= a0; o[m][n][1] *= a0; o[m][n][2] *= a1; o[m][n][3] *= a1; }
        }
        const int c0 = col0 + 8 * NTC * warp;
#pragma unroll
        for (int kk = 0; kk < kKeyBlock / 16; kk++) {
            uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
            for (int m = 0; m < MT; m++) {
                ldsm4(ph[m], sPh + (16 * m + (lane & 15)) * LDP + 16 * kk + 8 * (lane >> 4));
                ldsm4(pl[m], sPl + (16 * m + (lane & 15)) * LDP + 16 * kk + 8 * (lane >> 4));
            }
#pragma unroll
            for (int n = 0; n < NTC; n += 2) {
                if (c0 + 8 * n >= p.rank_pad) break;
                uint32_t bv[4];
                ldsm4_t(bv, sK[b] + (16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * LD + c0 + 8 * n + 8 * (lane >> 4));
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    mma_bf16(o[m][n], ph[m], bv[0], bv[1]);
                    mma_bf16(o[m][n], pl[m], bv[0], bv[1]);
                    mma_bf16(o[m][n + 1], ph[m], bv[2], bv[3]);
                    mma_bf16(o[m][n + 1], pl[m], bv[2], bv[3]);
                }
            }
        }
    }
    cp_async_wait_all();
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const long g = r0 + 16 * m + g4 + 4 * e;
            if (g >= rows) continue;
            float* dst = partial_sums(partial, g, split, splits, p.rank_pad);
#pragma unroll
            for (int n = 0; n < NTC; n++) {
                const int c = col0 + 8 * NTC * warp + 8 * n + 2 * t4;
                if (c < p.rank_pad && k_begin < k_end) *reinterpret_cast<float2*>(dst + c) = make_float2(o[m][n][e], o[m][n][e + 1]);
            }
        }
    if (tid < M && r0 + tid < rows && blockIdx.z == 0)
        partial_stats(partial, r0 + tid, splits, p.rank_pad)[split] = make_float2(sMax[tid], sSum[tid]);
}

// Plain form: eight rows per CTA, one per warp; lane = key for the scores, lane = column for the sums.
constexpr int kRowKeys = 32, kRowCols = 32;     // up to 32 * 32 latent columns

template <typename A>
__global__ void __launch_bounds__(256) k_latent_attn_rows(LatentShape p, const A* q, const A* cache, float* partial, const int* pos_p, int T)
{
    extern __shared__ float sf[];               // keys [32][row + 1], queries [8][row]
    const int row = p.row(), LD = row + 1;
    float* sk = sf;
    float* sq = sf + kRowKeys * LD;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const long rows = (long)T * p.heads, r0 = (long)blockIdx.x * 8, g = r0 + warp;
    const int splits = gridDim.y, split = blockIdx.y;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *pos_p;
    const int per = keys_per_split(pos + T, splits), k_begin = split * per;
    const long r_last = (r0 + 8 < rows ? r0 + 8 : rows) - 1;
    int k_end = pos + (int)(r_last / p.heads) + 1;
    if (k_end > k_begin + per) k_end = k_begin + per;
    const int last = g < rows ? pos + (int)(g / p.heads) : -1;
    for (int i = tid; i < 8 * row; i += 256) {
        const long gr = r0 + i / row;
        sq[i] = gr < rows ? act_load(q + (size_t)gr * row + i % row) : 0.0f;
    }
    float acc[kRowCols];
#pragma unroll
    for (int i = 0; i < kRowCols; i++) acc[i] = 0.0f;
    float mx = -INFINITY, sum = 0.0f;
    const float scale = p.scale * kLog2e;
    for (int k0 = k_begin; k0 < k_end; k0 += kRowKeys) {
        __syncthreads();
        const int n = k_end - k0 < kRowKeys ? k_end - k0 : kRowKeys;
        for (int i = tid; i < n * row; i += 256) {
            const int r = i / row, c = i - r * row;
            sk[r * LD + c] = act_load(cache + (size_t)(k0 + r) * row + c);
        }
        __syncthreads();
        float v = -INFINITY;
        if (lane < n && k0 + lane <= last) {
            float s0 = 0.0f, s1 = 0.0f, s2 = 0.0f, s3 = 0.0f;
            const float *a = sk + lane * LD, *b = sq + warp * row;
            for (int c = 0; c < row; c += 4) {
                s0 = fmaf(a[c], b[c], s0);
                s1 = fmaf(a[c + 1], b[c + 1], s1);
                s2 = fmaf(a[c + 2], b[c + 2], s2);
                s3 = fmaf(a[c + 3], b[c + 3], s3);
            }
            v = ((s0 + s1) + (s2 + s3)) * scale;
        }
        const float now = fmaxf(mx, warp_max(v)), base = now == -INFINITY ? 0.0f : now;
        const float w = exp2f(v - base), alpha = exp2f(mx - base);
        sum = sum * alpha + warp_sum(w);
        mx = now;
#pragma unroll
        for (int i = 0; i < kRowCols; i++) acc[i] *= alpha;
        for (int j = 0; j < n; j++) {
            const float wj = __shfl_sync(0xFFFFFFFFu, w, j);
#pragma unroll
            for (int i = 0; i < kRowCols; i++)
                if (lane + 32 * i < p.rank_pad) acc[i] = fmaf(wj, sk[j * LD + lane + 32 * i], acc[i]);
        }
    }
    if (g < rows) {
        float* dst = partial_sums(partial, g, split, splits, p.rank_pad);
        if (k_begin < k_end)
#pragma unroll
            for (int i = 0; i < kRowCols; i++)
                if (lane + 32 * i < p.rank_pad) dst[lane + 32 * i] = acc[i];
        if (lane == 0) partial_stats(partial, g, splits, p.rank_pad)[split] = make_float2(mx, sum);
    }
}

// grid (value columns / 32, heads, tokens): joins the splits (every CTA of a head again; the sums sit in L2), then W_uv: a
// warp per four value columns, whose weights are requested before the launch ahead has finished.
template <typename A>
__global__ void __launch_bounds__(256) k_latent_values(LatentShape p, float* partial, int splits, const bf16* __restrict__ w_uv, A* o,
                                                       const int* pos_p, int T)
{
    extern __shared__ __align__(16) float lat[];      // [2][rank_pad], then [splits] weights
    float* sw = lat + 2 * p.rank_pad;
    const int h = blockIdx.y, t = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const long row = (long)t * p.heads + h;
    pdl_launch_dependents();
    const int c0 = blockIdx.x * 32 + 4 * warp;
    const bf16* w = w_uv + ((size_t)h * p.value_pad + c0) * p.rank_pad;
    uint4 u[4][2];                                     // the first 512 latent columns
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int k = 8 * lane + 256 * i;
            u[j][i] = (c0 + j < p.value_pad && k < p.rank_pad) ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)j * p.rank_pad + k)) : make_uint4(0, 0, 0, 0);
        }
    pdl_wait();
    const int context = *pos_p + T, per = keys_per_split(context, splits);
    const int used = (context + per - 1) / per;
    const float2* stats = partial_stats(partial, row, splits, p.rank_pad);
    if (warp == 0) {
        // at most 148 splits: five per lane
        float2 st[5];
        float mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < 5; i++) {
            st[i] = lane + 32 * i < used ? stats[lane + 32 * i] : make_float2(-INFINITY, 0.0f);
            mx = fmaxf(mx, st[i].x);
        }
        mx = warp_max(mx);
        float sum = 0.0f;
#pragma unroll
        for (int i = 0; i < 5; i++) {
            st[i].x = st[i].x == -INFINITY ? 0.0f : exp2f(st[i].x - mx);
            sum = fmaf(st[i].x, st[i].y, sum);
        }
        const float inv = 1.0f / warp_sum(sum);
#pragma unroll
        for (int i = 0; i < 5; i++)
            if (lane + 32 * i < used) sw[lane + 32 * i] = st[i].x * inv;
    }
    __syncthreads();
    // even and odd splits by the two halves of the CTA, four columns per thread
    const float* sums = partial_sums(partial, row, 0, splits, p.rank_pad);
    for (int c = 4 * (tid & 127); c < p.rank_pad; c += 512) {
        float4 v = make_float4(0, 0, 0, 0);
#pragma unroll 8
        for (int i = tid >> 7; i < used; i += 2) {
            const float f = sw[i];
            const float4 a = *reinterpret_cast<const float4*>(sums + (size_t)i * p.rank_pad + c);
            if (f != 0.0f) {                           // a split without keys for this row holds no sums
                v.x = fmaf(f, a.x, v.x); v.y = fmaf(f, a.y, v.y); v.z = fmaf(f, a.z, v.z); v.w = fmaf(f, a.w, v.w);
            }
        }
        *reinterpret_cast<float4*>(lat + (tid >> 7) * p.rank_pad + c) = v;
    }
    __syncthreads();
    for (int c = tid; c < p.rank_pad; c += 256) lat[c] += lat[p.rank_pad + c];
    __syncthreads();
    float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    auto add = [&](const uint4& q, int k, float& v) {
        const float4 a = *reinterpret_cast<const float4*>(lat + k), b = *reinterpret_cast<const float4*>(lat + k + 4);
        v = fmaf(bf_lo(q.x), a.x, v); v = fmaf(bf_hi(q.x), a.y, v); v = fmaf(bf_lo(q.y), a.z, v); v = fmaf(bf_hi(q.y), a.w, v);
        v = fmaf(bf_lo(q.z), b.x, v); v = fmaf(bf_hi(q.z), b.y, v); v = fmaf(bf_lo(q.w), b.z, v); v = fmaf(bf_hi(q.w), b.w, v);
    };
#pragma unroll
    for (int i = 0; i < 2; i++)
        if (8 * lane + 256 * i < p.rank_pad)
#pragma unroll
            for (int j = 0; j < 4; j++) add(u[j][i], 8 * lane + 256 * i, acc[j]);
    for (int k = 8 * lane + 512; k < p.rank_pad; k += 256)
#pragma unroll
        for (int j = 0; j < 4; j++)
            if (c0 + j < p.value_pad) add(__ldg(reinterpret_cast<const uint4*>(w + (size_t)j * p.rank_pad + k)), k, acc[j]);
#pragma unroll
    for (int j = 0; j < 4; j++) {
        const float v = warp_sum(acc[j]);
        if (lane == 0 && c0 + j < p.value_pad) o[((size_t)t * p.heads + h) * p.value_pad + c0 + j] = act_from<A>(v);
    }
}

// ------------------------------------------------------------------ expanded keys and values (long portions)

// Rotates the query parts in place.
__global__ void __launch_bounds__(256) k_rotate_queries(LatentShape p, bf16* q, const int* pos_p, int T)
{
    pdl_launch_dependents();
    pdl_wait();
    const int pairs = p.rot_dims / 2;
    const long total = (long)T * p.heads * pairs;
    const int pos = *pos_p;
    for (long u = (long)blockIdx.x * blockDim.x + threadIdx.x; u < total; u += (long)gridDim.x * blockDim.x) {
        const int i = (int)(u % pairs);
        const long th = u / pairs;
        const int t = (int)(th / p.heads);
        bf16* x = q + (size_t)th * p.q_head() + p.dim_pad + 2 * i;
        float sn, cs;
        sincosf((float)(pos + t) * p.rot_freq[i], &sn, &cs);
        const uint32_t w = *reinterpret_cast<const uint32_t*>(x);
        *reinterpret_cast<uint32_t*>(x) = pack_bf16(bf_lo(w) * cs - bf_hi(w) * sn, bf_hi(w) * cs + bf_lo(w) * sn);
    }
}

constexpr int kQueryTile = 64;

static size_t expanded_smem(int q_head, int dv)
{
    return (size_t)kQueryTile * (q_head + 8) * 2 + 2 * (size_t)kKeyBlock * ((q_head + 8) + (dv + 8)) * 2;
}

// grid (query tiles, heads, value slices of DV); four warps of 16 queries.
template <int DV>
__global__ void __launch_bounds__(128) k_expanded_attn_mma(LatentShape p, const bf16* q, const bf16* expanded, const bf16* cache, bf16* o,
                                                           const int* pos_p, int T)
{
    constexpr int LDV = DV + 8;
    extern __shared__ __align__(128) uint8_t smem[];
    const int dq = p.q_head(), LDQ = dq + 8;
    bf16* sQ = reinterpret_cast<bf16*>(smem);
    bf16* sK[2] = {sQ + kQueryTile * LDQ, sQ + (kQueryTile + kKeyBlock) * LDQ};
    bf16* sV[2] = {sQ + (kQueryTile + 2 * kKeyBlock) * LDQ, sQ + (kQueryTile + 2 * kKeyBlock) * LDQ + kKeyBlock * LDV};
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
    const int tile = gridDim.x - 1 - blockIdx.x;            // the longest rows first
    const int h = blockIdx.y, v0 = blockIdx.z * DV;
    const int v_n = p.value_pad - v0 < DV ? p.value_pad - v0 : DV;
    const int ld_e = p.heads * (p.dim_pad + p.value_pad), row = p.row();
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *pos_p, t0 = tile * kQueryTile;
    const int n_t = T - t0 < kQueryTile ? T - t0 : kQueryTile;
    const int k_end = pos + t0 + n_t;
    const bf16* gk = expanded + h * p.dim_pad;
    const bf16* gv = expanded + (size_t)p.heads * p.dim_pad + h * p.value_pad + v0;
    const int uq = dq / 8, ud = p.dim_pad / 8, uv = DV / 8;
    auto load_keys = [&](int k0, int b) {
        for (int i = tid; i < kKeyBlock * uq; i += 128) {
            const int r = i / uq, u = i - r * uq, k = k0 + r, kc = k < k_end ? k : k_end - 1;
            const bf16* src = u < ud ? gk + (size_t)kc * ld_e + 8 * u : cache + (size_t)kc * row + p.rank_pad + 8 * (u - ud);
            cp_async16(sK[b] + r * LDQ + 8 * u, src, k < k_end);
        }
        for (int i = tid; i < kKeyBlock * uv; i += 128) {
            const int r = i / uv, u = i - r * uv, k = k0 + r, kc = k < k_end ? k : k_end - 1;
            const bool ok = k < k_end && 8 * u < v_n;
            cp_async16(sV[b] + r * LDV + 8 * u, gv + (size_t)kc * ld_e + (8 * u < v_n ? 8 * u : 0), ok);
        }
        cp_async_commit();
    };
    for (int i = tid; i < kQueryTile * uq; i += 128) {
        const int r = i / uq, u = i - r * uq, t = r < n_t ? t0 + r : t0;
        cp_async16(sQ + r * LDQ + 8 * u, q + ((size_t)t * p.heads + h) * dq + 8 * u, r < n_t);
    }
    load_keys(0, 0);
    float acc[DV / 8][4] = {};
    float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
    const float scale = p.scale * kLog2e;
    int b = 0;
    for (int k0 = 0; k0 < k_end; k0 += kKeyBlock, b ^= 1) {
        cp_async_wait_all();
        __syncthreads();
        if (k0 + kKeyBlock < k_end) load_keys(k0 + kKeyBlock, b ^ 1);
        float s[8][4] = {};
        for (int d = 0; d < dq; d += 16) {
            uint32_t a[4];
            ldsm4(a, sQ + (16 * warp + (lane & 15)) * LDQ + d + 8 * (lane >> 4));
#pragma unroll
            for (int n = 0; n < 8; n += 2) {
                uint32_t bk[4];
                ldsm4(bk, sK[b] + (8 * n + (lane & 7) + 8 * (lane >> 4)) * LDQ + d + 8 * ((lane >> 3) & 1));
                mma_bf16(s[n], a, bk[0], bk[1]);
                mma_bf16(s[n + 1], a, bk[2], bk[3]);
            }
        }
        const int i0 = pos + t0 + 16 * warp + g4;       // positions of this lane's two queries: i0, i0 + 8
        const bool edge = k0 + kKeyBlock > pos + t0 + 16 * warp;
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float m = mx[e];
#pragma unroll
            for (int n = 0; n < 8; n++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    float v = s[n][2 * e + c] * scale;
                    if (edge && k0 + 8 * n + 2 * t4 + c > i0 + 8 * e) v = -INFINITY;
                    s[n][2 * e + c] = v;
                    m = fmaxf(m, v);
                }
            m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, 1));
            m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, 2));
            const float base = m == -INFINITY ? 0.0f : m, alpha = exp2f(mx[e] - base);
            mx[e] = m;
            float w = 0.0f;
#pragma unroll
            for (int n = 0; n < 8; n++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    s[n][2 * e + c] = exp2f(s[n][2 * e + c] - base);
                    w += s[n][2 * e + c];
                }
            sum[e] = sum[e] * alpha + w;
#pragma unroll
            for (int n = 0; n < DV / 8; n++) {
                acc[n][2 * e] *= alpha;
                acc[n][2 * e + 1] *= alpha;
            }
        }
#pragma unroll
        for (int kk = 0; kk < kKeyBlock / 16; kk++) {
            uint32_t ph[4], pl[4];
            split_bf16(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
            split_bf16(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
            split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
            split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int n = 0; n < DV / 8; n += 2) {
                uint32_t bv[4];
                ldsm4_t(bv, sV[b] + (16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * LDV + 8 * n + 8 * (lane >> 4));
                mma_bf16(acc[n], ph, bv[0], bv[1]);
                mma_bf16(acc[n], pl, bv[0], bv[1]);
                mma_bf16(acc[n + 1], ph, bv[2], bv[3]);
                mma_bf16(acc[n + 1], pl, bv[2], bv[3]);
            }
        }
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        float w = sum[e];
        w += __shfl_xor_sync(0xFFFFFFFFu, w, 1);
        w += __shfl_xor_sync(0xFFFFFFFFu, w, 2);
        const float inv = 1.0f / w;
        const int r = 16 * warp + g4 + 8 * e;
        if (r >= n_t) continue;
        bf16* dst = o + ((size_t)(t0 + r) * p.heads + h) * p.value_pad + v0;
#pragma unroll
        for (int n = 0; n < DV / 8; n++) {
            const int c = 8 * n + 2 * t4;
            if (c < v_n) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(acc[n][2 * e] * inv, acc[n][2 * e + 1] * inv);
        }
    }
}

// ------------------------------------------------------------------ host side

// Expanding costs context * heads * (dim + value) * rank products, once per portion; attending in latent space costs
// 2 rank - dim - value more products per (query, key, head).  They meet at this many queries.
bool latent_expands(const LatentShape& p, int T, bool act_bf16)
{
    if (!act_bf16) return false;
    if (expanded_smem(p.q_head(), p.value_pad <= 64 ? 64 : 128) > 220 * 1024) return false;
    const long extra = 2L * p.rank_pad - p.dim_pad - p.value_pad, once = (long)(p.dim_pad + p.value_pad) * p.rank_pad;
    if (T < kQueryTile) return false;
    return extra <= 0 ? T >= 2 * kQueryTile : T * extra >= once;
}

static int latent_mt(const LatentShape& p, int T) { return (long)T * p.heads <= 16 ? 1 : 2; }
static bool latent_mma_fits(const LatentShape& p, int T)
{
    const size_t smem = latent_mt(p, T) == 1 ? LatentTile<1, 2>::smem(p.row()) : LatentTile<2, 2>::smem(p.row());
    return smem <= 220 * 1024;
}
static int latent_splits(const LatentShape& p, int T, bool mma)
{
    const long tile = mma ? 16 * latent_mt(p, T) : 8;
    const long tiles = ((long)T * p.heads + tile - 1) / tile;
    const long want = sm_count() / tiles;
    return (int)(want < 1 ? 1 : want > 148 ? 148 : want);
}

size_t latent_partial_floats(const LatentShape& p, int T, bool act_bf16)
{
    if (latent_expands(p, T, act_bf16)) return 0;
    const int splits = latent_splits(p, T, act_bf16 && latent_mma_fits(p, T));
    return (size_t)T * p.heads * partial_stride(splits, p.rank_pad);
}

template <int MT, int NTC>
static int launch_latent_mma(const LatentShape& p, const bf16* q, const bf16* cache, float* partial, const int* pos, int T, int splits,
                             cudaStream_t s)
{
    using S = LatentTile<MT, NTC>;
    int rc = allow_smem<k_latent_attn_mma<MT, NTC>>(220 * 1024);
    if (rc) return rc;
    const long rows = (long)T * p.heads;
    const dim3 grid((unsigned)((rows + S::kRows - 1) / S::kRows), splits, (p.rank_pad + S::kCols - 1) / S::kCols);
    return launch_ordered(k_latent_attn_mma<MT, NTC>, grid, 256, S::smem(p.row()), s, p, q, cache, partial, pos, T);
}

template <typename A>
static int attend_latents(const LatentShape& p, const void* q, const bf16* w_ukv, const void* cache, void* o, const LatentBuffers& b,
                          const int* pos, int T, cudaStream_t s)
{
    constexpr bool kBf16 = sizeof(A) == 2;
    int rc = T == 1 ? launch_latent_queries<A, 1>(p, q, w_ukv, b.q_latent, pos, T, s) : launch_latent_queries<A, 4>(p, q, w_ukv, b.q_latent, pos, T, s);
    if (rc) return rc;
    const bool mma = kBf16 && latent_mma_fits(p, T);
    const int splits = latent_splits(p, T, mma);
    if (mma) {
        const bf16 *ql = (const bf16*)b.q_latent, *c = (const bf16*)cache;
        if (latent_mt(p, T) == 1) {
            if (p.rank_pad <= 128) rc = launch_latent_mma<1, 2>(p, ql, c, b.partial, pos, T, splits, s);
            else if (p.rank_pad <= 256) rc = launch_latent_mma<1, 4>(p, ql, c, b.partial, pos, T, splits, s);
            else rc = launch_latent_mma<1, 8>(p, ql, c, b.partial, pos, T, splits, s);
        } else {
            if (p.rank_pad <= 128) rc = launch_latent_mma<2, 2>(p, ql, c, b.partial, pos, T, splits, s);
            else if (p.rank_pad <= 256) rc = launch_latent_mma<2, 4>(p, ql, c, b.partial, pos, T, splits, s);
            else rc = launch_latent_mma<2, 8>(p, ql, c, b.partial, pos, T, splits, s);
        }
    } else {
        const size_t smem = ((size_t)kRowKeys * (p.row() + 1) + 8 * (size_t)p.row()) * 4;
        if (smem > 220 * 1024 || p.rank_pad > 32 * kRowCols) return latch(BPDQ_ERR_RANGE);
        if ((rc = allow_smem<k_latent_attn_rows<A>>(220 * 1024))) return rc;
        rc = launch_ordered(k_latent_attn_rows<A>, dim3((unsigned)(((long)T * p.heads + 7) / 8), splits), 256, smem, s, p, (const A*)b.q_latent,
                            (const A*)cache, b.partial, pos, T);
    }
    if (rc) return rc;
    const bf16* w_uv = w_ukv + (size_t)p.heads * p.dim_pad * p.rank_pad;
    return launch_ordered(k_latent_values<A>, dim3((p.value_pad + 31) / 32, p.heads, T), 256, (size_t)(2 * p.rank_pad + splits) * 4, s, p,
                          b.partial, splits, w_uv, (A*)o, pos, T);
}

int latent_attention(const LatentShape& p, void* q, const bf16* w_ukv, const void* cache, void* o, const LatentBuffers& b, const int* pos,
                     int T, int context, bool act_bf16, cudaStream_t s)
{
    if (!latent_expands(p, T, act_bf16))
        return act_bf16 ? attend_latents<bf16>(p, q, w_ukv, cache, o, b, pos, T, s) : attend_latents<float>(p, q, w_ukv, cache, o, b, pos, T, s);
    Linear l = {};
    l.W = w_ukv;
    l.in = cache;
    l.N = p.heads * (p.dim_pad + p.value_pad);
    l.K = p.rank_pad;
    l.ld_in = p.row();
    l.mode = kLinAct;
    l.out = b.expanded;
    l.ld_out = l.N;
    int rc = linear_forward(l, context, true, s);
    if (rc) return rc;
    if ((rc = launch_ordered(k_rotate_queries, grid_1d((long)T * p.heads * p.rot_dims / 2), 256, 0, s, p, (bf16*)q, pos, T))) return rc;
    const dim3 tiles((T + kQueryTile - 1) / kQueryTile, p.heads, p.value_pad <= 64 ? 1 : (p.value_pad + 127) / 128);
    const bf16 *e = (const bf16*)b.expanded, *c = (const bf16*)cache;
    if (p.value_pad <= 64) {
        if ((rc = allow_smem<k_expanded_attn_mma<64>>(220 * 1024))) return rc;
        return launch_ordered(k_expanded_attn_mma<64>, tiles, 128, expanded_smem(p.q_head(), 64), s, p, (const bf16*)q, e, c, (bf16*)o, pos, T);
    }
    if ((rc = allow_smem<k_expanded_attn_mma<128>>(220 * 1024))) return rc;
    return launch_ordered(k_expanded_attn_mma<128>, tiles, 128, expanded_smem(p.q_head(), 128), s, p, (const bf16*)q, e, c, (bf16*)o, pos, T);
}

}  // namespace bpdq

using namespace bpdq;

extern "C" {

static LatentShape shape_of(const bpdq_latent_shape* c)
{
    LatentShape p = {};
    p.heads = c->heads; p.dim_pad = c->dim_pad; p.value_pad = c->value_pad;
    p.rank = c->rank; p.rank_pad = c->rank_pad;
    p.rot_dims = c->rot_dims; p.rot_pad = c->rot_pad;
    p.q_rank = c->q_rank; p.q_rank_pad = c->q_rank_pad;
    p.rot_freq = c->rot_freq;
    p.scale = c->scale; p.eps = c->eps;
    return p;
}
static bool shape_ok(const bpdq_latent_shape* c)
{
    return c && c->heads > 0 && c->dim_pad > 0 && c->value_pad > 0 && c->rank > 0 && c->rank_pad >= c->rank && c->rot_pad >= c->rot_dims &&
           c->rot_dims >= 0 && !((c->dim_pad | c->value_pad | c->rank_pad | c->rot_pad) % 16) && c->rot_freq;
}

int bpd_latent_prepare_cuda(const bpdq_latent_shape* shape, const void* u, int ld_u, const float* q_norm, const float* kv_norm, void* cq, void* cache,
                            const int32_t* pos, int n_tokens, int act_bf16, void* stream)
{
    if (!shape_ok(shape) || n_tokens < 0 || shape->q_rank < 1 || shape->q_rank_pad < shape->q_rank) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!u || !q_norm || !cq || !pos || (cache && !kv_norm)) return latch(BPDQ_ERR_ARG);
    return latent_prepare(shape_of(shape), u, ld_u, q_norm, kv_norm, cq, cache, pos, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

int bpd_latent_attention_cuda(const bpdq_latent_shape* shape, void* q, const uint16_t* w_ukv, const void* cache, void* o, const int32_t* pos,
                              int n_tokens, int context, int act_bf16, void* stream)
{
    if (!shape_ok(shape) || n_tokens < 0 || context < n_tokens) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!q || !w_ukv || !cache || !o || !pos) return latch(BPDQ_ERR_ARG);
    const LatentShape p = shape_of(shape);
    const bool b16 = act_bf16 != 0;
    const size_t a = b16 ? 2 : 4;
    auto up = [](size_t v) { return (v + 255) / 256 * 256; };
    const size_t ql = up((size_t)n_tokens * p.heads * p.row() * a), part = up(latent_partial_floats(p, n_tokens, b16) * 4);
    const size_t exp = latent_expands(p, n_tokens, b16) ? (size_t)context * p.heads * (p.dim_pad + p.value_pad) * a : 0;
    int rc = 0;
    uint8_t* base = scratch_take(nullptr, kScratchLatent, ql + part + exp, (cudaStream_t)stream, &rc);
    if (!base) return rc;
    const LatentBuffers b = {base, (float*)(base + ql), base + ql + part};
    return latent_attention(p, q, reinterpret_cast<const bf16*>(w_ukv), cache, o, b, pos, n_tokens, context, b16, (cudaStream_t)stream);
}

}  // extern "C"
