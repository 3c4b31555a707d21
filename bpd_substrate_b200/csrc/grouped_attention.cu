// Grouped-query attention with chunks, capped scores and a sink.  Rows of a tile are (token, query head) pairs of one key head, so
// keys and values are read once for all heads that share them.
//
//   k_grouped_prepare    norms of queries and keys, cache rows
//   k_grouped_split_mma  bf16, few queries (decoding): 16 rows per CTA, keys dealt to the warps of a cluster of CTAs; keys and
//                        values go from HBM straight into mma.sync fragments (dimensions and columns are taken in the order in
//                        which 16-byte loads bring them), the cluster joins its parts through distributed shared memory
//   k_grouped_tile_mma   bf16, a prompt's portion: 64 rows per CTA, keys in double-buffered blocks of 64
//   k_grouped_rows       fp32 (and bf16 sizes beyond the others): a warp per row
//
// Scores and softmax are fp32; weights enter the product with the values as the sum of two bf16 numbers.
#include "grouped_attention.cuh"
#include "cluster_device.cuh"
#include "launch.cuh"
#include "mma_device.cuh"
#include "../../include/bpdq.h"

namespace bpdq {

constexpr float kLog2e = 1.44269504088896340736f;

// ------------------------------------------------------------------ norms and cache rows

// A warp per (token, head of the queries, keys or values).
template <typename A>
__global__ void __launch_bounds__(256) k_grouped_prepare(GroupedShape p, A* u, int ld_u, A* cache, const int* pos_p, int T)
{
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, units = p.heads + (cache ? 2 * p.groups : 0);
    const long unit = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int t = (int)(unit / units), i = (int)(unit - (long)t * units);
    if (t >= T) return;
    const int pos = *pos_p + t;
    A* dst = cache + (size_t)(pos % p.rows) * p.row();
    A* row = u + (size_t)t * ld_u;
    const bool value = i >= p.heads + p.groups;
    const int n = (value ? p.value_pad : p.dim_pad) / 4;
    const A* src;
    if (i < p.heads) { src = row + i * p.dim_pad; dst = row + i * p.dim_pad; }
    else if (!value) { src = row + i * p.dim_pad; dst += (i - p.heads) * p.dim_pad; }
    else { const int g = i - p.heads - p.groups; src = row + (p.heads + p.groups) * p.dim_pad + g * p.value_pad; dst += p.groups * p.dim_pad + g * p.value_pad; }
    float f = 1.0f;
    if (!value) {       // pad entries are zero
        float sum = 0.0f;
        for (int c = lane; c < n; c += 32) {
            const float4 v = act_load4(src + 4 * c);
            sum = fmaf(v.x, v.x, sum); sum = fmaf(v.y, v.y, sum); sum = fmaf(v.z, v.z, sum); sum = fmaf(v.w, v.w, sum);
        }
        f = 1.0f / sqrtf(warp_sum(sum) / (float)p.dim + p.eps);
    }
    for (int c = lane; c < n; c += 32) {
        const float4 v = act_load4(src + 4 * c);
        act_store4(dst + 4 * c, make_float4(v.x * f, v.y * f, v.z * f, v.w * f));
    }
}

int grouped_prepare(const GroupedShape& p, void* u, int ld_u, void* cache, const int* pos, int T, bool act_bf16, cudaStream_t s)
{
    const long units = (long)T * (p.heads + (cache ? 2 * p.groups : 0));
    const unsigned grid = (unsigned)((units + 7) / 8);
    if (act_bf16) return launch_ordered(k_grouped_prepare<bf16>, grid, 256, 0, s, p, (bf16*)u, ld_u, (bf16*)cache, pos, T);
    return launch_ordered(k_grouped_prepare<float>, grid, 256, 0, s, p, (float*)u, ld_u, (float*)cache, pos, T);
}

// ------------------------------------------------------------------ scores

// Score in units of log2: tanh(z) = 1 - 2 / (1 + e^(2 z)), whose absolute error of an fp32 unit is all a capped score needs.
struct ScoreMap {
    float plain, in, out;       // cap == 0: s plain;  else out tanh(s in / (2 log2 e))
    __device__ __forceinline__ ScoreMap(const GroupedShape& p)
    {
        plain = p.scale * kLog2e;
        in = p.cap > 0.0f ? p.scale / p.cap * 2.0f * kLog2e : 0.0f;
        out = p.cap * kLog2e;
    }
    __device__ __forceinline__ float operator()(float s) const
    {
        if (in == 0.0f) return s * plain;
        return fmaf(-2.0f * out, below(s), out);
    }
    // (1 - tanh) / 2 of a capped score
    __device__ __forceinline__ float below(float s) const { return __fdividef(1.0f, 1.0f + ex2(s * in)); }
};

// ------------------------------------------------------------------ few queries, bf16

constexpr int kSplitRows = 16, kSplitKeys = 16;
constexpr int kMaxSplits = 8;       // CTAs of a cluster

// ND groups of 32 dimensions, NV groups of 64 value columns.  grid (groups, splits, row tiles), cluster (1, splits, 1), eight warps.
template <int ND, int NV>
__global__ void __launch_bounds__(256, 1) k_grouped_split_mma(GroupedShape p, const bf16* u, int ld_u, const bf16* cache, bf16* o, const int* pos_p, int T)
{
    constexpr int kCols = 64 * NV, LD = kCols + 4;
    extern __shared__ __align__(16) float sm[];      // [8][rows][LD] sums of the warps; the CTA's end up in the first
    __shared__ float2 s_stat[8][kSplitRows];
    __shared__ float s_max[kSplitRows], s_sum[kSplitRows];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
    const int g = blockIdx.x, share = p.share(), r0 = blockIdx.z * kSplitRows, rows = T * share;
    const int n_rows = rows - r0 < kSplitRows ? rows - r0 : kSplitRows;
    const uint32_t splits = cluster_size(), split = cluster_rank();
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *pos_p;
    // this lane's rows g4 and g4 + 8: first and last position they see
    int lo[2], last[2];
    uint4 qx[2][ND];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = r0 + g4 + 8 * e, t = r / share;
        const bool in = r < rows;
        last[e] = in ? pos + t : -1;
        lo[e] = in ? p.first_seen(pos + t) : 0;
        const bf16* q = u + (size_t)t * ld_u + (g * share + r - t * share) * p.dim_pad;
#pragma unroll
        for (int d = 0; d < ND; d++)
            qx[e][d] = (in && 32 * d + 8 * t4 < p.dim_pad) ? *reinterpret_cast<const uint4*>(q + 32 * d + 8 * t4) : make_uint4(0, 0, 0, 0);
    }
    const int k_begin = p.first_seen(pos + r0 / share), k_end = pos + (r0 + n_rows - 1) / share + 1;
    const bf16* keys = cache + g * p.dim_pad;
    const bf16* values = cache + p.groups * p.dim_pad + g * p.value_pad;
    const int row = p.row();
    const ScoreMap score(p);
    float acc[NV][8][4];
#pragma unroll
    for (int v = 0; v < NV; v++)
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[v][j][e] = 0.0f;
    float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
    const int step = (int)splits * 8 * kSplitKeys;
    for (int k0 = k_begin + ((int)split * 8 + warp) * kSplitKeys; k0 < k_end; k0 += step) {
        const int slot0 = k0 % p.rows;
        auto place = [&](int i) -> size_t {
            const int sl = slot0 + i;
            return (size_t)(sl >= p.rows ? sl - p.rows : sl) * row;
        };
        uint4 kx[2][ND], vx[4][NV];
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int i = 8 * e + g4;
            const bf16* src = keys + (k0 + i < k_end ? place(i) : 0);
#pragma unroll
            for (int d = 0; d < ND; d++)
                kx[e][d] = (k0 + i < k_end && 32 * d + 8 * t4 < p.dim_pad) ? *reinterpret_cast<const uint4*>(src + 32 * d + 8 * t4) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int i = 2 * t4 + (e & 1) + 8 * (e >> 1);
            const bf16* src = values + (k0 + i < k_end ? place(i) : 0);
#pragma unroll
            for (int v = 0; v < NV; v++)
                vx[e][v] = (k0 + i < k_end && 64 * v + 8 * g4 < p.value_pad) ? *reinterpret_cast<const uint4*>(src + 64 * v + 8 * g4) : make_uint4(0, 0, 0, 0);
        }
        float s[2][4] = {};
#pragma unroll
        for (int d = 0; d < ND; d++) {
            const uint32_t a0[4] = {qx[0][d].x, qx[1][d].x, qx[0][d].y, qx[1][d].y}, a1[4] = {qx[0][d].z, qx[1][d].z, qx[0][d].w, qx[1][d].w};
#pragma unroll
            for (int e = 0; e < 2; e++) {
                mma_bf16(s[e], a0, kx[e][d].x, kx[e][d].y);
                mma_bf16(s[e], a1, kx[e][d].z, kx[e][d].w);
            }
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int r = 0; r < 2; r++) {
            float m = mx[r];
#pragma unroll
            for (int e = 0; e < 2; e++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    const int k = k0 + 8 * e + 2 * t4 + c;
                    const float v = (k <= last[r] && k >= lo[r]) ? score(s[e][2 * r + c]) : -INFINITY;
                    s[e][2 * r + c] = v;
                    m = fmaxf(m, v);
                }
            m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, 1));
            m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, 2));
            const float base = m == -INFINITY ? 0.0f : m, alpha = ex2(mx[r] - base);
            mx[r] = m;
            float w = 0.0f;
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const float e0 = ex2(s[e][2 * r] - base), e1 = ex2(s[e][2 * r + 1] - base);
                split_bf16(e0, e1, ph[2 * e + r], pl[2 * e + r]);
                w += e0 + e1;
            }
            sum[r] = sum[r] * alpha + w;
#pragma unroll
            for (int v = 0; v < NV; v++)
#pragma unroll
                for (int j = 0; j < 8; j++) {
                    acc[v][j][2 * r] *= alpha;
                    acc[v][j][2 * r + 1] *= alpha;
                }
        }
#pragma unroll
        for (int v = 0; v < NV; v++)
#pragma unroll
            for (int j = 0; j < 8; j++) {
                const uint32_t pick = (j & 1) ? 0x7632u : 0x5410u;
                const auto word = [&](const uint4& x) -> uint32_t { return j < 2 ? x.x : j < 4 ? x.y : j < 6 ? x.z : x.w; };
                const uint32_t b0 = __byte_perm(word(vx[0][v]), word(vx[1][v]), pick), b1 = __byte_perm(word(vx[2][v]), word(vx[3][v]), pick);
                mma_bf16(acc[v][j], ph, b0, b1);
                mma_bf16(acc[v][j], pl, b0, b1);
            }
    }
    // ---- the eight warps
#pragma unroll
    for (int r = 0; r < 2; r++) {
        sum[r] += __shfl_xor_sync(0xFFFFFFFFu, sum[r], 1);
        sum[r] += __shfl_xor_sync(0xFFFFFFFFu, sum[r], 2);
        if (t4 == 0) s_stat[warp][g4 + 8 * r] = make_float2(mx[r], sum[r]);
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int at = g4 + 8 * r;
        float m = -INFINITY;
#pragma unroll
        for (int i = 0; i < 8; i++) m = fmaxf(m, s_stat[i][at].x);
        const float base = m == -INFINITY ? 0.0f : m, f = ex2(mx[r] - base);
        if (warp == 0 && t4 == 0) {
            float w = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; i++) w = fmaf(ex2(s_stat[i][at].x - base), s_stat[i][at].y, w);
            s_max[at] = m;
            s_sum[at] = w;
        }
        if (at < n_rows) {
            float* dst = sm + (size_t)(warp * n_rows + at) * LD + 16 * t4;
#pragma unroll
            for (int v = 0; v < NV; v++)
#pragma unroll
                for (int c = 0; c < 2; c++)
#pragma unroll
                    for (int j = 0; j < 8; j += 4)
                        *reinterpret_cast<float4*>(dst + 64 * v + 8 * c + j) =
                            make_float4(acc[v][j][2 * r + c] * f, acc[v][j + 1][2 * r + c] * f, acc[v][j + 2][2 * r + c] * f, acc[v][j + 3][2 * r + c] * f);
        }
    }
    __syncthreads();
    for (int i = tid; i < n_rows * (kCols / 4); i += 256) {
        float* a = sm + (size_t)(i / (kCols / 4)) * LD + 4 * (i % (kCols / 4));
        float4 x = *reinterpret_cast<float4*>(a);
#pragma unroll
        for (int w = 1; w < 8; w++) {
            const float4 y = *reinterpret_cast<const float4*>(a + (size_t)w * n_rows * LD);
            x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
        }
        *reinterpret_cast<float4*>(a) = x;
    }
    // ---- the cluster: every CTA finishes a share of the columns
    if (splits > 1) { cluster_arrive(); cluster_wait(); }
    else __syncthreads();
    const int units = p.value_pad / 4;
    for (int i = (int)split * 256 + tid; i < n_rows * units; i += (int)splits * 256) {
        const int r = i / units, c = 4 * (i - r * units);
        float m = p.sink ? 0.0f : -INFINITY;
        for (uint32_t k = 0; k < splits; k++) m = fmaxf(m, splits > 1 ? load_peer(&s_max[r], k) : s_max[r]);
        float w = p.sink ? ex2(-m) : 0.0f;
        float4 x = make_float4(0, 0, 0, 0);
        for (uint32_t k = 0; k < splits; k++) {
            const float f = ex2((splits > 1 ? load_peer(&s_max[r], k) : s_max[r]) - m);
            const float4 y = splits > 1 ? load_peer4(sm + (size_t)r * LD + c, k) : *reinterpret_cast<const float4*>(sm + (size_t)r * LD + c);
            w = fmaf(f, splits > 1 ? load_peer(&s_sum[r], k) : s_sum[r], w);
            x.x = fmaf(f, y.x, x.x); x.y = fmaf(f, y.y, x.y); x.z = fmaf(f, y.z, x.z); x.w = fmaf(f, y.w, x.w);
        }
        const float inv = 1.0f / w;
        const int t = (r0 + r) / share, h = g * share + (r0 + r) - t * share;
        act_store4(o + ((size_t)t * p.heads + h) * p.value_pad + c, make_float4(x.x * inv, x.y * inv, x.z * inv, x.w * inv));
    }
    if (splits > 1) { cluster_arrive(); cluster_wait(); }     // nobody leaves while its sums are read
}

// ------------------------------------------------------------------ a prompt's portion, bf16

constexpr int kTileRows = 64, kKeyBlock = 64;

static size_t tile_smem(int dim_pad, int dv)
{
    return (size_t)(kTileRows + 2 * kKeyBlock) * (dim_pad + 8) * 2 + 2 * (size_t)kKeyBlock * (dv + 8) * 2;
}

// A capped score cannot exceed the cap, so weights can be taken relative to it and no maximum is tracked.  With a sink the sum is
// at least e^-cap; up to this cap whatever underflows beside that is below fp32's resolution.
constexpr float kBoundedCap = 64.0f;

// grid (row tiles, groups, value slices of DV); four warps of 16 rows.
template <int DV, bool kBounded>
__global__ void __launch_bounds__(128) k_grouped_tile_mma(GroupedShape p, const bf16* u, int ld_u, const bf16* cache, bf16* o, const int* pos_p, int T)
{
    constexpr int LDV = DV + 8;
    extern __shared__ __align__(128) uint8_t smem[];
    const int dq = p.dim_pad, LDQ = dq + 8;
    bf16* sQ = reinterpret_cast<bf16*>(smem);
    bf16* sK[2] = {sQ + kTileRows * LDQ, sQ + (kTileRows + kKeyBlock) * LDQ};
    bf16* sV[2] = {sQ + (kTileRows + 2 * kKeyBlock) * LDQ, sQ + (kTileRows + 2 * kKeyBlock) * LDQ + kKeyBlock * LDV};
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
    const int share = p.share(), rows = T * share, r0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kTileRows;      // late rows first
    const int n_rows = rows - r0 < kTileRows ? rows - r0 : kTileRows;
    const int g = blockIdx.y, v0 = blockIdx.z * DV;
    const int v_n = p.value_pad - v0 < DV ? p.value_pad - v0 : DV;
    const int row = p.row();
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *pos_p;
    const int k_begin = p.first_seen(pos + r0 / share), k_end = pos + (r0 + n_rows - 1) / share + 1;
    const bf16* gk = cache + g * dq;
    const bf16* gv = cache + p.groups * dq + g * p.value_pad + v0;
    const int uq = dq / 8;
    constexpr int uv = DV / 8;
    auto load_keys = [&](int k0, int b) {
        const int slot0 = k0 % p.rows;
        auto place = [&](int r) -> size_t {
            const int sl = slot0 + (k0 + r < k_end ? r : 0);
            return (size_t)(sl >= p.rows ? sl - p.rows : sl) * row;
        };
        for (int i = tid; i < kKeyBlock * uq; i += 128) {
            const int r = i / uq, c = i - r * uq;
            cp_async16(sK[b] + r * LDQ + 8 * c, gk + place(r) + 8 * c, k0 + r < k_end);
        }
        for (int i = tid; i < kKeyBlock * uv; i += 128) {
            const int r = i / uv, c = i - r * uv;
            const bool ok = k0 + r < k_end && 8 * c < v_n;
            cp_async16(sV[b] + r * LDV + 8 * c, gv + place(r) + (8 * c < v_n ? 8 * c : 0), ok);
        }
        cp_async_commit();
    };
    for (int i = tid; i < kTileRows * uq; i += 128) {
        const int r = i / uq, c = i - r * uq, rr = r0 + (r < n_rows ? r : 0), t = rr / share;
        cp_async16(sQ + r * LDQ + 8 * c, u + (size_t)t * ld_u + (g * share + rr - t * share) * dq + 8 * c, r < n_rows);
    }
    load_keys(k_begin, 0);
    float acc[DV / 8][4] = {};
    int lo[2], last[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = 16 * warp + g4 + 8 * e, i = pos + (r0 + r) / share;
        last[e] = r < n_rows ? i : -1;
        lo[e] = r < n_rows ? p.first_seen(i) : 0;
    }
    // the warp's rows need no mask between these positions
    const int w_last = pos + (r0 + 16 * warp) / share, w_lo = p.first_seen(pos + (r0 + (16 * warp + 15 < n_rows ? 16 * warp + 15 : n_rows - 1)) / share);
    const ScoreMap score(p);
    float mx[2], sum[2];
    mx[0] = mx[1] = p.sink ? 0.0f : -INFINITY;
    sum[0] = sum[1] = (p.sink && t4 == 0) ? (kBounded ? ex2(-score.out) : 1.0f) : 0.0f;        // (a row's four lanes are added up at the end)
    int b = 0;
    for (int k0 = k_begin; k0 < k_end; k0 += kKeyBlock, b ^= 1) {
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
        const bool edge = k0 + kKeyBlock - 1 > w_last || k0 < w_lo;
#pragma unroll
        for (int e = 0; e < 2; e++) {
            if (kBounded) {
                const float f = -2.0f * score.out;
                float w = 0.0f;
#pragma unroll
                for (int n = 0; n < 8; n++)
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        float v = ex2(f * score.below(s[n][2 * e + c]));
                        if (edge) {
                            const int k = k0 + 8 * n + 2 * t4 + c;
                            if (k > last[e] || k < lo[e]) v = 0.0f;
                        }
                        s[n][2 * e + c] = v;
                        w += v;
                    }
                sum[e] += w;
                continue;
            }
            float m = mx[e];
#pragma unroll
            for (int n = 0; n < 8; n++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    float v = score(s[n][2 * e + c]);
                    if (edge) {
                        const int k = k0 + 8 * n + 2 * t4 + c;
                        if (k > last[e] || k < lo[e]) v = -INFINITY;
                    }
                    s[n][2 * e + c] = v;
                    m = fmaxf(m, v);
                }
            m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, 1));
            m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, 2));
            const float base = m == -INFINITY ? 0.0f : m, alpha = ex2(mx[e] - base);
            mx[e] = m;
            float w = 0.0f;
#pragma unroll
            for (int n = 0; n < 8; n++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    s[n][2 * e + c] = ex2(s[n][2 * e + c] - base);
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
        if (r >= n_rows) continue;
        const int t = (r0 + r) / share, h = g * share + (r0 + r) - t * share;
        bf16* dst = o + ((size_t)t * p.heads + h) * p.value_pad + v0;
#pragma unroll
        for (int n = 0; n < DV / 8; n++) {
            const int c = 8 * n + 2 * t4;
            if (c < v_n) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(acc[n][2 * e] * inv, acc[n][2 * e + 1] * inv);
        }
    }
}

// ------------------------------------------------------------------ plain form

constexpr int kRowKeys = 32, kRowCols = 16;     // up to 16 * 32 value columns

// grid (row tiles of eight, groups): a warp per row; lane = key for the scores, lane = column for the sums.
template <typename A>
__global__ void __launch_bounds__(256) k_grouped_rows(GroupedShape p, const A* u, int ld_u, const A* cache, A* o, const int* pos_p, int T)
{
    extern __shared__ float sf[];               // keys [32][dim_pad + 1], values [32][value_pad], queries [8][dim_pad]
    const int D = p.dim_pad, V = p.value_pad, LD = D + 1;
    float* sk = sf;
    float* sv = sk + kRowKeys * LD;
    float* sq = sv + kRowKeys * V;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = blockIdx.y, share = p.share(), rows = T * share, r0 = blockIdx.x * 8, r = r0 + warp;
    const int n_rows = rows - r0 < 8 ? rows - r0 : 8;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *pos_p;
    const int k_begin = p.first_seen(pos + r0 / share), k_end = pos + (r0 + n_rows - 1) / share + 1;
    const int t = r / share, h = g * share + r - t * share;
    const int last = warp < n_rows ? pos + t : -1, lo = warp < n_rows ? p.first_seen(pos + t) : 0;
    for (int i = tid; i < n_rows * D; i += 256) {
        const int rr = r0 + i / D, tt = rr / share;
        sq[i] = act_load(u + (size_t)tt * ld_u + (g * share + rr - tt * share) * D + i % D);
    }
    float acc[kRowCols];
#pragma unroll
    for (int i = 0; i < kRowCols; i++) acc[i] = 0.0f;
    float mx = p.sink ? 0.0f : -INFINITY, sum = p.sink ? 1.0f : 0.0f;
    for (int k0 = k_begin; k0 < k_end; k0 += kRowKeys) {
        __syncthreads();
        const int n = k_end - k0 < kRowKeys ? k_end - k0 : kRowKeys, slot0 = k0 % p.rows;
        for (int i = tid; i < n * (D + V); i += 256) {
            const int j = i / (D + V), c = i - j * (D + V);
            const int sl = slot0 + j;
            const A* src = cache + (size_t)(sl >= p.rows ? sl - p.rows : sl) * p.row();
            if (c < D) sk[j * LD + c] = act_load(src + g * D + c);
            else sv[j * V + c - D] = act_load(src + p.groups * D + g * V + c - D);
        }
        __syncthreads();
        float v = -INFINITY;
        if (lane < n && k0 + lane <= last && k0 + lane >= lo) {
            float s0 = 0.0f, s1 = 0.0f, s2 = 0.0f, s3 = 0.0f;
            const float *a = sk + lane * LD, *b = sq + warp * D;
            for (int c = 0; c < D; c += 4) {
                s0 = fmaf(a[c], b[c], s0);
                s1 = fmaf(a[c + 1], b[c + 1], s1);
                s2 = fmaf(a[c + 2], b[c + 2], s2);
                s3 = fmaf(a[c + 3], b[c + 3], s3);
            }
            v = ((s0 + s1) + (s2 + s3)) * p.scale;
            if (p.cap > 0.0f) v = p.cap * tanhf(v / p.cap);
        }
        const float now = fmaxf(mx, warp_max(v)), base = now == -INFINITY ? 0.0f : now;
        const float w = expf(v - base), alpha = expf(mx - base);
        sum = sum * alpha + warp_sum(w);
        mx = now;
#pragma unroll
        for (int i = 0; i < kRowCols; i++) acc[i] *= alpha;
        for (int j = 0; j < n; j++) {
            const float wj = __shfl_sync(0xFFFFFFFFu, w, j);
#pragma unroll
            for (int i = 0; i < kRowCols; i++)
                if (lane + 32 * i < V) acc[i] = fmaf(wj, sv[j * V + lane + 32 * i], acc[i]);
        }
    }
    if (warp >= n_rows) return;
    const float inv = 1.0f / sum;
#pragma unroll
    for (int i = 0; i < kRowCols; i++)
        if (lane + 32 * i < V) o[((size_t)t * p.heads + h) * V + lane + 32 * i] = act_from<A>(acc[i] * inv);
}

template <typename A>
static int launch_rows(const GroupedShape& p, const void* u, int ld_u, const void* cache, void* o, const int* pos, int T, cudaStream_t s)
{
    const size_t smem = ((size_t)kRowKeys * (p.dim_pad + 1 + p.value_pad) + 8 * (size_t)p.dim_pad) * 4;
    if (smem > 220 * 1024 || p.value_pad > 32 * kRowCols) return latch(BPDQ_ERR_RANGE);
    int rc = allow_smem<k_grouped_rows<A>>(220 * 1024);
    if (rc) return rc;
    return launch_ordered(k_grouped_rows<A>, dim3((unsigned)(((long)T * p.share() + 7) / 8), p.groups), 256, smem, s, p, (const A*)u, ld_u, (const A*)cache,
                          (A*)o, pos, T);
}

// ------------------------------------------------------------------ host side

// Up to this many rows of a group the keys are split over CTAs instead of the rows.
constexpr int kSplitMaxRows = 64;

template <int ND, int NV>
static int launch_split(const GroupedShape& p, const bf16* u, int ld_u, const bf16* cache, bf16* o, const int* pos, int T, cudaStream_t s)
{
    const int rows = T * p.share(), tiles = (rows + kSplitRows - 1) / kSplitRows;
    const int span = p.chunk > 0 && p.chunk < p.rows ? p.chunk : p.rows;      // the most keys a query can see
    int splits = 1;
    while (splits < kMaxSplits && 2 * splits * tiles * p.groups <= sm_count() && splits * 8 * kSplitKeys < span) splits *= 2;
    int rc = allow_smem<k_grouped_split_mma<ND, NV>>(8 * kSplitRows * (64 * NV + 4) * 4);
    if (rc) return rc;
    const int n_rows = rows < kSplitRows ? rows : kSplitRows;
    return launch_cluster(k_grouped_split_mma<ND, NV>, dim3(p.groups, splits, tiles), dim3(1, splits, 1), 256, (size_t)8 * n_rows * (64 * NV + 4) * 4, s, p, u,
                          ld_u, cache, o, pos, T);
}

template <int DV, bool kBounded>
static int launch_tile(const GroupedShape& p, const bf16* u, int ld_u, const bf16* cache, bf16* o, const int* pos, int T, cudaStream_t s)
{
    int rc = allow_smem<k_grouped_tile_mma<DV, kBounded>>(220 * 1024);
    if (rc) return rc;
    const dim3 grid((unsigned)(((long)T * p.share() + kTileRows - 1) / kTileRows), p.groups, (p.value_pad + DV - 1) / DV);
    return launch_ordered(k_grouped_tile_mma<DV, kBounded>, grid, 128, tile_smem(p.dim_pad, DV), s, p, u, ld_u, cache, o, pos, T);
}

int grouped_attention(const GroupedShape& p, const void* u, int ld_u, const void* cache, void* o, const int* pos, int T, bool act_bf16,
                      cudaStream_t s)
{
    if (!act_bf16) return launch_rows<float>(p, u, ld_u, cache, o, pos, T, s);
    const bf16 *q = (const bf16*)u, *c = (const bf16*)cache;
    bf16* out = (bf16*)o;
    const int most = p.dim_pad > p.value_pad ? p.dim_pad : p.value_pad;
    if ((long)T * p.share() <= kSplitMaxRows && most <= 256) {
        if (most <= 64) return launch_split<2, 1>(p, q, ld_u, c, out, pos, T, s);
        if (most <= 128) return launch_split<4, 2>(p, q, ld_u, c, out, pos, T, s);
        return launch_split<8, 4>(p, q, ld_u, c, out, pos, T, s);
    }
    if (tile_smem(p.dim_pad, p.value_pad <= 64 ? 64 : 128) <= 220 * 1024) {
        const bool bounded = p.sink && p.cap > 0.0f && p.cap <= kBoundedCap;
        if (p.value_pad <= 64) return bounded ? launch_tile<64, true>(p, q, ld_u, c, out, pos, T, s) : launch_tile<64, false>(p, q, ld_u, c, out, pos, T, s);
        return bounded ? launch_tile<128, true>(p, q, ld_u, c, out, pos, T, s) : launch_tile<128, false>(p, q, ld_u, c, out, pos, T, s);
    }
    return launch_rows<bf16>(p, u, ld_u, cache, o, pos, T, s);
}

}  // namespace bpdq

using namespace bpdq;

extern "C" {

int bpd_grouped_attention_cuda(const bpdq_grouped_shape* c, void* u, int ld_u, void* cache, int append, void* o, const int32_t* pos, int n_tokens,
                               int act_bf16, void* stream)
{
    if (!c || n_tokens < 0 || c->heads < 1 || c->groups < 1 || c->heads % c->groups || c->dim < 1 || c->dim_pad < c->dim || c->value_pad < 1 ||
        (c->dim_pad | c->value_pad) % 16 || c->chunk < 0 || c->rows < 1 || c->cap < 0.0f)
        return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!u || !cache || !o || !pos) return latch(BPDQ_ERR_ARG);
    if (ld_u % 8) return latch(BPDQ_ERR_ALIGN);
    GroupedShape p = {};
    p.heads = c->heads; p.groups = c->groups; p.dim = c->dim; p.dim_pad = c->dim_pad; p.value_pad = c->value_pad;
    p.chunk = c->chunk; p.rows = c->rows; p.sink = c->sink;
    p.scale = c->scale; p.cap = c->cap; p.eps = c->eps;
    const int rc = grouped_prepare(p, u, ld_u, append ? cache : nullptr, pos, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
    return rc ? rc : grouped_attention(p, u, ld_u, cache, o, pos, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

}  // extern "C"
