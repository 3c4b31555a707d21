// Gated delta rule.
//
//   k_delta_token       one token: a cluster of CTAs per head, each with 32 value columns; the state goes through HBM once.
//                       Unit lengths, prediction and read-out come from one pass over the state (the read-out of the written
//                       state is the read-out of the decayed one plus (k.q) u); the output's norm joins its CTAs through
//                       distributed shared memory.
//   k_delta_recurrence  token by token: a warp holds four value columns of a head, eight lanes over the keys, so that a token
//                       costs three shuffles and no barrier.  Short portions, fp32 runs.
//   k_delta_prepare, k_delta_chunks
//                       a prompt's portion in chunks of 16 tokens.  Inside a chunk with decays g, c_i = g_0 .. g_i and
//                         A_ij = beta_i k_i . (g_{j+1} .. g_i k_j)  (j < i),   P_ij = q_i . (g_{j+1} .. g_i k_j)  (j <= i)
//                       the writes solve (1 + A) u = beta (v - (c k) S), so that
//                         u = U - W S,  o = O + Q S,  S <- c_15 S + sum_j (g_{j+1} .. g_15 k_j) u_j^T
//                       with (1 + A) W = beta c k,  (1 + A) U = beta v,  Q = c q - P W,  O = P U.  The first kernel works these out for
//                       all chunks at once (fp32, a thread per key or value column; only products of decays, which cannot
//                       overflow); the second walks the chunks with the transposed state in fp32 accumulators: a warp for
//                       the state of 16 value columns and one for its read-out, fed by bulk copies of ready-made fragments.
//                       What is fp32 enters mma.sync as the sum of two bf16 numbers, three products.
#include "delta_rule.cuh"
#include "cluster_device.cuh"
#include "launch.cuh"
#include "mma_device.cuh"
#include "../../include/bpdq.h"

namespace bpdq {

// An fp32 exponential that leans one way by a unit in the last place adds up over thousands of tokens.
template <typename A> __device__ __forceinline__ float decay_of(float log_decay) { return sizeof(A) == 4 ? (float)exp((double)log_decay) : expf(log_decay); }

// ------------------------------------------------------------------ one token

constexpr int kTokenCols = 32;

// grid (heads, value columns / 32), 256 threads: eight groups of four columns x 32 key phases.
template <typename A, int NI>
__global__ void __launch_bounds__(256) k_delta_token(DeltaRule a)
{
    __shared__ float4 red[8][8][2], red_s[8];
    __shared__ float s_part[8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, cg = tid & 7, phase = tid >> 3;
    const int h = blockIdx.x, g = h / (a.heads / a.groups), p = blockIdx.y * kTokenCols + 4 * cg;
    const bool live = p < a.value_pad;
    pdl_launch_dependents();
    const uint32_t parts = cluster_size();
    if (parts > 1) cluster_arrive();        // (everybody is there before anybody's shared memory is written)
    const float4 zero = make_float4(0, 0, 0, 0);
    const float4 nw = (a.norm_w && live) ? *reinterpret_cast<const float4*>(a.norm_w + (size_t)h * a.value_pad + p) : zero;
    pdl_wait();
    float* st = a.state + (size_t)h * a.key_pad * a.value_pad + p;
    const A* q = reinterpret_cast<const A*>(a.q) + g * a.key_pad;
    const A* k = reinterpret_cast<const A*>(a.k) + g * a.key_pad;
    const float* lg = a.log_decay + (size_t)h * a.key_pad;
    float4 s[NI];
    float kn[NI], qn[NI], dn[NI];
#pragma unroll
    for (int i = 0; i < NI; i++) {
        const int n = phase + 32 * i;
        const bool in = n < a.key_pad;
        s[i] = (in && live) ? *reinterpret_cast<const float4*>(st + (size_t)n * a.value_pad) : zero;
        kn[i] = in ? act_load(k + n) : 0.0f;
        qn[i] = in ? act_load(q + n) : 0.0f;
        dn[i] = in ? lg[n] : 0.0f;
    }
    const size_t at = (size_t)h * a.value_pad + p;
    const float4 v = live ? act_load4(reinterpret_cast<const A*>(a.v) + at) : zero;
    const float4 gate = (a.norm_w && live) ? act_load4(reinterpret_cast<const A*>(a.gate) + at) : zero;
    const float beta = a.beta[h];
    float4 sk = zero, sq = zero;
    float kk = 0.0f, qq = 0.0f, kq = 0.0f;
#pragma unroll
    for (int i = 0; i < NI; i++) {
        const float d = decay_of<A>(dn[i]);
        s[i] = make_float4(s[i].x * d, s[i].y * d, s[i].z * d, s[i].w * d);
        sk.x = fmaf(s[i].x, kn[i], sk.x); sk.y = fmaf(s[i].y, kn[i], sk.y); sk.z = fmaf(s[i].z, kn[i], sk.z); sk.w = fmaf(s[i].w, kn[i], sk.w);
        sq.x = fmaf(s[i].x, qn[i], sq.x); sq.y = fmaf(s[i].y, qn[i], sq.y); sq.z = fmaf(s[i].z, qn[i], sq.z); sq.w = fmaf(s[i].w, qn[i], sq.w);
        kk = fmaf(kn[i], kn[i], kk);
        qq = fmaf(qn[i], qn[i], qq);
        kq = fmaf(kn[i], qn[i], kq);
    }
#pragma unroll
    for (int o = 8; o < 32; o <<= 1) {
        sk.x += __shfl_xor_sync(0xFFFFFFFFu, sk.x, o); sk.y += __shfl_xor_sync(0xFFFFFFFFu, sk.y, o);
        sk.z += __shfl_xor_sync(0xFFFFFFFFu, sk.z, o); sk.w += __shfl_xor_sync(0xFFFFFFFFu, sk.w, o);
        sq.x += __shfl_xor_sync(0xFFFFFFFFu, sq.x, o); sq.y += __shfl_xor_sync(0xFFFFFFFFu, sq.y, o);
        sq.z += __shfl_xor_sync(0xFFFFFFFFu, sq.z, o); sq.w += __shfl_xor_sync(0xFFFFFFFFu, sq.w, o);
        kk += __shfl_xor_sync(0xFFFFFFFFu, kk, o);
        qq += __shfl_xor_sync(0xFFFFFFFFu, qq, o);
        kq += __shfl_xor_sync(0xFFFFFFFFu, kq, o);
    }
    if (lane < 8) {
        red[warp][lane][0] = sk;
        red[warp][lane][1] = sq;
        if (lane == 0) red_s[warp] = make_float4(kk, qq, kq, 0.0f);
    }
    __syncthreads();
    sk = sq = zero;
    kk = qq = kq = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const float4 x = red[i][cg][0], y = red[i][cg][1], z = red_s[i];
        sk.x += x.x; sk.y += x.y; sk.z += x.z; sk.w += x.w;
        sq.x += y.x; sq.y += y.y; sq.z += y.z; sq.w += y.w;
        kk += z.x; qq += z.y; kq += z.z;
    }
    const float rk = 1.0f / sqrtf(kk + a.unit_eps), rq = a.q_scale / sqrtf(qq + a.unit_eps);
    const float4 u = make_float4(beta * (v.x - sk.x * rk), beta * (v.y - sk.y * rk), beta * (v.z - sk.z * rk), beta * (v.w - sk.w * rk));
    const float c = kq * rk * rq;
    float4 o = make_float4(fmaf(c, u.x, sq.x * rq), fmaf(c, u.y, sq.y * rq), fmaf(c, u.z, sq.z * rq), fmaf(c, u.w, sq.w * rq));
    if (live) {
#pragma unroll
        for (int i = 0; i < NI; i++) {
            const int n = phase + 32 * i;
            if (n >= a.key_pad) break;
            const float f = kn[i] * rk;
            *reinterpret_cast<float4*>(st + (size_t)n * a.value_pad) =
                make_float4(fmaf(f, u.x, s[i].x), fmaf(f, u.y, s[i].y), fmaf(f, u.z, s[i].z), fmaf(f, u.w, s[i].w));
        }
    }
    if (a.norm_w) {
        float ss = o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;      // columns beyond the head are zero
        ss += __shfl_xor_sync(0xFFFFFFFFu, ss, 1);
        ss += __shfl_xor_sync(0xFFFFFFFFu, ss, 2);
        ss += __shfl_xor_sync(0xFFFFFFFFu, ss, 4);
        if (parts > 1) {
            cluster_wait();
            if (tid < (int)parts) store_peer(&s_part[cluster_rank()], tid, ss);
            cluster_arrive();
            cluster_wait();
            ss = 0.0f;
            for (uint32_t i = 0; i < parts; i++) ss += s_part[i];
        }
        const float f = 1.0f / sqrtf(ss / (float)a.value_dim + a.eps);
        o = make_float4(o.x * f * nw.x * sigmoid_act<A>(gate.x), o.y * f * nw.y * sigmoid_act<A>(gate.y), o.z * f * nw.z * sigmoid_act<A>(gate.z),
                        o.w * f * nw.w * sigmoid_act<A>(gate.w));
    }
    if (phase == 0 && live) act_store4(reinterpret_cast<A*>(a.o) + at, o);
}

template <typename A, int NI>
static int launch_token(const DeltaRule& a, cudaStream_t s)
{
    int parts = 1;
    while (parts * kTokenCols < a.value_pad) parts *= 2;
    return launch_cluster(k_delta_token<A, NI>, dim3(a.heads, parts), dim3(1, a.norm_w ? parts : 1), 256, 0, s, a);
}

template <typename A>
static int delta_token(const DeltaRule& a, cudaStream_t s)
{
    if (a.key_pad <= 32) return launch_token<A, 1>(a, s);
    if (a.key_pad <= 64) return launch_token<A, 2>(a, s);
    if (a.key_pad <= 128) return launch_token<A, 4>(a, s);
    if (a.key_pad <= 256) return launch_token<A, 8>(a, s);
    return launch_token<A, 16>(a, s);
}

bool delta_token_norms(int key_pad, int value_pad) { return key_pad <= 512 && value_pad <= 8 * kTokenCols; }

// ------------------------------------------------------------------ recurrence

// grid (heads, value columns / 32), eight warps of four columns; lane: keys 4 (lane & 7) + 32 i + j of column lane >> 3.  Tokens
// pass through shared memory in blocks of TB with unit lengths, decays and k.q worked out.
template <int NI, int TB>
struct DeltaStage {
    static constexpr int kKeys = 32 * NI, kToken = 3 * kKeys + kTokenCols + 4;
    static constexpr size_t kSmem = 2 * (size_t)TB * kToken * 4;
};

template <typename A, int NI, int TB>
__global__ void __launch_bounds__(256) k_delta_recurrence(DeltaRule a, int T)
{
    using S = DeltaStage<NI, TB>;
    extern __shared__ __align__(16) float sm[];      // [2][TB] of k, q, decay [kKeys] each, v [32], beta, k.q
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, kl = 4 * (lane & 7);
    const int h = blockIdx.x, g = h / (a.heads / a.groups), c0 = blockIdx.y * kTokenCols;
    const int col = 4 * warp + (lane >> 3);
    const bool live = c0 + col < a.value_pad;
    pdl_launch_dependents();
    pdl_wait();
    float* st = a.state + (size_t)h * a.key_pad * a.value_pad + c0 + col;
    float s[4 * NI];
#pragma unroll
    for (int i = 0; i < 4 * NI; i++) {
        const int n = kl + 32 * (i >> 2) + (i & 3);
        s[i] = (live && n < a.key_pad) ? st[(size_t)n * a.value_pad] : 0.0f;
    }
    auto stage = [&](int t0, int b) {
        for (int r = warp; r < TB && t0 + r < T; r += 8) {
            const size_t t = t0 + r;
            float* dst = sm + (size_t)(b * TB + r) * S::kToken;
            const A* k = reinterpret_cast<const A*>(a.k) + t * a.ld + g * a.key_pad;
            const A* q = reinterpret_cast<const A*>(a.q) + t * a.ld + g * a.key_pad;
            const float* lg = a.log_decay + (t * a.heads + h) * a.key_pad;
            float kv[NI], qv[NI], dv[NI], kk = 0.0f, qq = 0.0f, kq = 0.0f;
#pragma unroll
            for (int i = 0; i < NI; i++) {
                const int n = lane + 32 * i;
                const bool in = n < a.key_pad;
                kv[i] = in ? act_load(k + n) : 0.0f;
                qv[i] = in ? act_load(q + n) : 0.0f;
                dv[i] = in ? lg[n] : 0.0f;
            }
#pragma unroll
            for (int i = 0; i < NI; i++) { kk = fmaf(kv[i], kv[i], kk); qq = fmaf(qv[i], qv[i], qq); kq = fmaf(kv[i], qv[i], kq); }
            kk = warp_sum(kk);
            qq = warp_sum(qq);
            kq = warp_sum(kq);
            const float rk = 1.0f / sqrtf(kk + a.unit_eps), rq = a.q_scale / sqrtf(qq + a.unit_eps);
#pragma unroll
            for (int i = 0; i < NI; i++) {
                dst[lane + 32 * i] = kv[i] * rk;
                dst[S::kKeys + lane + 32 * i] = qv[i] * rq;
                dst[2 * S::kKeys + lane + 32 * i] = decay_of<A>(dv[i]);
            }
            dst[3 * S::kKeys + lane] = c0 + lane < a.value_pad ? act_load(reinterpret_cast<const A*>(a.v) + t * a.ld + (size_t)h * a.value_pad + c0 + lane) : 0.0f;
            if (lane == 0) {
                dst[3 * S::kKeys + kTokenCols] = a.beta[t * a.heads + h];
                dst[3 * S::kKeys + kTokenCols + 1] = kq * rk * rq;
            }
        }
    };
    stage(0, 0);
    for (int t0 = 0, b = 0; t0 < T; t0 += TB, b ^= 1) {
        __syncthreads();                    // this block is here, everybody has left the other buffer
        if (t0 + TB < T) stage(t0 + TB, b ^ 1);
        const int n_t = T - t0 < TB ? T - t0 : TB;
        for (int r = 0; r < n_t; r++) {
            const float* src = sm + (size_t)(b * TB + r) * S::kToken;
            float4 k4[NI];
            float sk = 0.0f, sq = 0.0f;
#pragma unroll
            for (int i = 0; i < NI; i++) {
                k4[i] = *reinterpret_cast<const float4*>(src + kl + 32 * i);
                const float4 q4 = *reinterpret_cast<const float4*>(src + S::kKeys + kl + 32 * i);
                const float4 d4 = *reinterpret_cast<const float4*>(src + 2 * S::kKeys + kl + 32 * i);
                s[4 * i] *= d4.x; s[4 * i + 1] *= d4.y; s[4 * i + 2] *= d4.z; s[4 * i + 3] *= d4.w;
                sk = fmaf(s[4 * i], k4[i].x, sk); sk = fmaf(s[4 * i + 1], k4[i].y, sk); sk = fmaf(s[4 * i + 2], k4[i].z, sk); sk = fmaf(s[4 * i + 3], k4[i].w, sk);
                sq = fmaf(s[4 * i], q4.x, sq); sq = fmaf(s[4 * i + 1], q4.y, sq); sq = fmaf(s[4 * i + 2], q4.z, sq); sq = fmaf(s[4 * i + 3], q4.w, sq);
            }
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) {
                sk += __shfl_xor_sync(0xFFFFFFFFu, sk, o);
                sq += __shfl_xor_sync(0xFFFFFFFFu, sq, o);
            }
            const float u = src[3 * S::kKeys + kTokenCols] * (src[3 * S::kKeys + col] - sk);
#pragma unroll
            for (int i = 0; i < NI; i++) {
                s[4 * i] = fmaf(k4[i].x, u, s[4 * i]); s[4 * i + 1] = fmaf(k4[i].y, u, s[4 * i + 1]);
                s[4 * i + 2] = fmaf(k4[i].z, u, s[4 * i + 2]); s[4 * i + 3] = fmaf(k4[i].w, u, s[4 * i + 3]);
            }
            if ((lane & 7) == 0 && live)
                reinterpret_cast<A*>(a.o)[((size_t)(t0 + r) * a.heads + h) * a.value_pad + c0 + col] =
                    act_from<A>(fmaf(src[3 * S::kKeys + kTokenCols + 1], u, sq));
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < 4 * NI; i++) {
            const int n = kl + 32 * (i >> 2) + (i & 3);
            if (n < a.key_pad) st[(size_t)n * a.value_pad] = s[i];
        }
    }
}

template <typename A, int NI, int TB>
static int launch_delta_recurrence(const DeltaRule& a, int T, cudaStream_t s)
{
    constexpr size_t smem = DeltaStage<NI, TB>::kSmem;
    int rc = allow_smem<k_delta_recurrence<A, NI, TB>>((int)smem);
    if (rc) return rc;
    return launch_ordered(k_delta_recurrence<A, NI, TB>, dim3(a.heads, (a.value_pad + kTokenCols - 1) / kTokenCols), 256, smem, s, a, T);
}

template <typename A>
static int delta_recurrence(const DeltaRule& a, int T, cudaStream_t s)
{
    if (a.key_pad <= 32) return launch_delta_recurrence<A, 1, 16>(a, T, s);
    if (a.key_pad <= 64) return launch_delta_recurrence<A, 2, 16>(a, T, s);
    if (a.key_pad <= 128) return launch_delta_recurrence<A, 4, 16>(a, T, s);
    if (a.key_pad <= 256) return launch_delta_recurrence<A, 8, 8>(a, T, s);
    return launch_delta_recurrence<A, 16, 8>(a, T, s);
}

// ------------------------------------------------------------------ chunks of 16 tokens

constexpr int kChunk = 16;
constexpr int kSegmentChunks = 64;          // chunks worked out at a time: what they need stays in L2

// Of a chunk and head, in the order in which k_delta_chunks' lanes read them: fragments of -W, Q and of the keys with the decays
// that follow them (64 bytes per key each: two bf16 numbers per value), then c_15 in fp32.
__host__ __device__ constexpr size_t fragment_bytes(int key_pad) { return (size_t)key_pad * (3 * 64 + 4); }
// U and O: [value column block of 16][U, O][lane][8]
__host__ __device__ constexpr size_t update_floats(int value_pad) { return (size_t)value_pad * 2 * kChunk; }

// v[j] of all lanes added up: lane j gets the sum of v[j].
__device__ __forceinline__ float transposed_sum(float (&v)[32], int lane)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < o; i++) {
            const float keep = up ? v[i + o] : v[i], send = up ? v[i] : v[i + o];
            v[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, o);
        }
    }
    return v[0];
}

// grid (heads, chunks), a thread per key (rounded up to whole warps); tokens t0 .. t1 - 1, those beyond count as zeros that
// neither decay nor write.
template <int kThreads, int kBlocks>
__global__ void __launch_bounds__(kThreads, kBlocks) k_delta_prepare(DeltaRule a, uint8_t* frags, float* updates, int t0, int t1)
{
    extern __shared__ __align__(16) uint8_t sf[];     // the chunk's fragments
    __shared__ float s_part[8][256], s_norm[8][32];
    __shared__ float4 sA[kChunk][4], sP[kChunk][4];
    __shared__ float s_beta[kChunk];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
    const int h = blockIdx.x, gr = h / (a.heads / a.groups), first = t0 + blockIdx.y * kChunk;
    const int D = a.key_pad, V = a.value_pad, n = tid;
    const bool key = n < D;
    pdl_launch_dependents();
    pdl_wait();
    float k[kChunk], q[kChunk], g[kChunk];
    {
        const bf16* pk = reinterpret_cast<const bf16*>(a.k) + (size_t)first * a.ld + gr * D + n;
        const bf16* pq = reinterpret_cast<const bf16*>(a.q) + (size_t)first * a.ld + gr * D + n;
        const float* pd = a.log_decay + ((size_t)first * a.heads + h) * D + n;
        const int left = key ? t1 - first : 0, step = a.heads * D;
#pragma unroll
        for (int i = 0; i < kChunk; i++) {
            k[i] = i < left ? act_load(pk + i * a.ld) : 0.0f;
            q[i] = i < left ? act_load(pq + i * a.ld) : 0.0f;
            g[i] = i < left ? pd[i * step] : 0.0f;
        }
    }
    if (tid < kChunk) s_beta[tid] = first + tid < t1 ? a.beta[(size_t)(first + tid) * a.heads + h] : 0.0f;
    float v[32];
#pragma unroll
    for (int i = 0; i < kChunk; i++) {
        v[i] = k[i] * k[i];
        v[kChunk + i] = q[i] * q[i];
        g[i] = expf(g[i]);
    }
    s_norm[warp][lane] = transposed_sum(v, lane);
    __syncthreads();
    {
        float sum = 0.0f;
        for (int w = 0; w < warps; w++) sum += s_norm[w][lane];
        const float f = (lane < kChunk ? 1.0f : a.q_scale) / sqrtf(sum + a.unit_eps);
#pragma unroll
        for (int i = 0; i < kChunk; i++) {
            k[i] *= __shfl_sync(0xFFFFFFFFu, f, i);
            q[i] *= __shfl_sync(0xFFFFFFFFu, f, kChunk + i);
        }
    }
    // columns m and 15 - m of P and A together are 32 sums
#pragma unroll
    for (int m = 0; m < 8; m++) {
        float r = k[m];
#pragma unroll
        for (int i = m; i < kChunk; i++) {
            if (i > m) {
                r *= g[i];
                v[16 - m + i - m - 1] = k[i] * r;
            }
            v[i - m] = q[i] * r;
        }
        r = k[15 - m];
#pragma unroll
        for (int i = 15 - m; i < kChunk; i++) {
            if (i > 15 - m) {
                r *= g[i];
                v[32 - m + i - (16 - m)] = k[i] * r;
            }
            v[31 - 2 * m + i - (15 - m)] = q[i] * r;
        }
        s_part[warp][32 * m + lane] = transposed_sum(v, lane);
    }
    __syncthreads();
    for (int x = tid; x < 256; x += blockDim.x) {
        float sum = 0.0f;
        for (int w = 0; w < warps; w++) sum += s_part[w][x];
        const int m = x >> 5, l = x & 31;
        float *A = reinterpret_cast<float*>(sA), *P = reinterpret_cast<float*>(sP);
        if (l < 16 - m) P[(m + l) * kChunk + m] = sum;
        else if (l < 31 - 2 * m) { const int i = 2 * m + 1 + l - 16; A[i * kChunk + m] = sum * s_beta[i]; }
        else if (l < 32 - m) P[(15 - m + l - (31 - 2 * m)) * kChunk + 15 - m] = sum;
        else { const int i = 16 - m + l - (32 - m); A[i * kChunk + 15 - m] = sum * s_beta[i]; }
    }
    __syncthreads();
    // the first n entries of a row
    auto load_row = [](const float4 (&m)[kChunk][4], int i, int n, float (&r)[kChunk]) {
#pragma unroll
        for (int j = 0; j < 4; j++)
            if (4 * j < n) *reinterpret_cast<float4*>(r + 4 * j) = m[i][j];
    };
    const size_t unit = (size_t)blockIdx.y * a.heads + h;
    if (key) {
        uint32_t* fw = reinterpret_cast<uint32_t*>(sf);
        uint32_t* fq = fw + 16 * D;
        uint32_t* fk = fq + 16 * D;
        // the keys with the decays that follow them: a lane's 16 bytes are tokens 2 t, 2 t + 1 and 2 t + 8, 2 t + 9 of one key
        float z[kChunk], r = 1.0f;
#pragma unroll
        for (int i = kChunk - 1; i >= 0; i--) {
            z[i] = k[i] * r;
            r *= g[i];
        }
        reinterpret_cast<float*>(fk + 16 * D)[n] = r;
#pragma unroll
        for (int t = 0; t < 4; t++) {
            uint4 w;
            split_bf16(z[2 * t], z[2 * t + 1], w.x, w.z);
            split_bf16(z[2 * t + 8], z[2 * t + 9], w.y, w.w);
            *reinterpret_cast<uint4*>(fk + ((n >> 3) * 32 + (n & 7) * 4 + t) * 4) = w;
        }
        // W by forward substitution, Q from it
        float w[kChunk], c = 1.0f;
#pragma unroll
        for (int i = 0; i < kChunk; i++) {
            c *= g[i];
            float x = s_beta[i] * k[i] * c, y = q[i] * c;
            alignas(16) float ar[kChunk], pr[kChunk];
            load_row(sA, i, i, ar);
            load_row(sP, i, i + 1, pr);
#pragma unroll
            for (int j = 0; j < i; j++) {
                x = fmaf(-ar[j], w[j], x);
                y = fmaf(-pr[j], w[j], y);
            }
            w[i] = x;
            z[i] = fmaf(-pr[i], x, y);
        }
        // keys n and n + 1 share a register: the even thread writes tokens 0 .. 7, the odd one 8 .. 15
        const unsigned live = D - (n & ~31) >= 32 ? 0xFFFFFFFFu : 0xFFFFu;
        const bool odd = n & 1;
        const int nn = (n & 15) >> 1;
        const size_t at = (((size_t)(n >> 4) * 2 + odd) * 32 + (nn & 3)) * 4 + (nn >> 2);
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const float pw = __shfl_xor_sync(live, odd ? w[i] : w[i + 8], 1), pz = __shfl_xor_sync(live, odd ? z[i] : z[i + 8], 1);
            const float w0 = odd ? pw : w[i], w1 = odd ? w[i + 8] : pw, z0 = odd ? pz : z[i], z1 = odd ? z[i + 8] : pz;
            uint32_t hi, lo;
            split_bf16(-w0, -w1, hi, lo);
            fw[at + 16 * i] = hi;
            fw[at + 16 * i + 2] = lo;
            split_bf16(z0, z1, hi, lo);
            fq[at + 16 * i] = hi;
            fq[at + 16 * i + 2] = lo;
        }
    }
    float* up = updates + unit * update_floats(V);
    for (int p = tid; p < V; p += blockDim.x) {
        const bf16* pv = reinterpret_cast<const bf16*>(a.v) + (size_t)first * a.ld + (size_t)h * V + p;
        const int left = t1 - first;
        float x[kChunk], u[kChunk], o[kChunk];
#pragma unroll
        for (int i = 0; i < kChunk; i++) x[i] = i < left ? act_load(pv + i * a.ld) : 0.0f;
#pragma unroll
        for (int i = 0; i < kChunk; i++) {
            float y = s_beta[i] * x[i], z = 0.0f;
            alignas(16) float ar[kChunk], pr[kChunk];
            load_row(sA, i, i, ar);
            load_row(sP, i, i + 1, pr);
#pragma unroll
            for (int j = 0; j < i; j++) {
                y = fmaf(-ar[j], u[j], y);
                z = fmaf(pr[j], u[j], z);
            }
            u[i] = y;
            o[i] = fmaf(pr[i], y, z);
        }
        float* dst = up + (size_t)(p >> 4) * 512 + (p & 7) * 32 + ((p >> 3) & 1) * 2;
#pragma unroll
        for (int t = 0; t < 4; t++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                *reinterpret_cast<float2*>(dst + t * 8 + e * 4) = make_float2(u[8 * e + 2 * t], u[8 * e + 2 * t + 1]);
                *reinterpret_cast<float2*>(dst + 256 + t * 8 + e * 4) = make_float2(o[8 * e + 2 * t], o[8 * e + 2 * t + 1]);
            }
    }
    __syncthreads();
    uint4* dst = reinterpret_cast<uint4*>(frags + unit * fragment_bytes(D));
    for (int i = tid; i < (int)(fragment_bytes(D) / 16); i += blockDim.x) dst[i] = reinterpret_cast<const uint4*>(sf)[i];
}

// (Not a barrier for the compiler: loads of other shared memory may pass it; an arrival on a barrier publishes it.)
__device__ __forceinline__ void store_shared(uint32_t at, const uint32_t (&v)[4])
{
    asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(at), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]));
}

template <int NMAX>
struct DeltaChunks {
    static constexpr int kStages = NMAX == 256 ? 3 : 4;
    static constexpr size_t kState = (size_t)NMAX / 16 * 1024;      // fragments of 16 columns of the state, high and low parts
    static size_t smem(int key_pad) { return kStages * fragment_bytes(key_pad) + 4 * kState; }
};

// grid (heads, value columns / 32): warps 0, 1 hold the state of 16 value columns each, warps 2, 3 read it out, warp 4 feeds.  kExact: the keys
// are NMAX, so that no step of the products hangs on a branch.
template <int NMAX, bool kExact>
__global__ void __launch_bounds__(160, 1) k_delta_chunks(DeltaRule a, const uint8_t* frags, const float* updates, int t0, int t1, int chunks, int* err)
{
    using S = DeltaChunks<NMAX>;
    constexpr int NT = NMAX / 8, KS = NMAX / 16;
    extern __shared__ __align__(128) uint8_t smem[];
    __shared__ uint64_t full[S::kStages], empty[S::kStages], state_full[2][2], state_empty[2][2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
    const int h = blockIdx.x, D = kExact ? NMAX : a.key_pad, V = a.value_pad, ks_n = D / 16;
    const int blocks = V / 16 - 2 * (int)blockIdx.y < 2 ? V / 16 - 2 * (int)blockIdx.y : 2;
    const uint32_t bytes = (uint32_t)fragment_bytes(D);
    uint8_t* s_state = smem + S::kStages * (size_t)bytes;
    if (tid == 0) {
        for (int i = 0; i < S::kStages; i++) { mbar_init(&full[i], 1); mbar_init(&empty[i], 2 * blocks); }
        for (int i = 0; i < 4; i++) { mbar_init(&state_full[i >> 1][i & 1], 1); mbar_init(&state_empty[i >> 1][i & 1], 1); }
        mbar_init_fence();
    }
    __syncthreads();
    pdl_launch_dependents();
    pdl_wait();
    if (warp == 4) {
        if (lane == 0) {
            int c = 0;
            for (; c < chunks; c++) {
                const int s = c % S::kStages;
                if (c >= S::kStages && !mbar_wait_bounded(&empty[s], (uint32_t)(c / S::kStages - 1) & 1u, err, 61)) break;
                mbar_expect_tx(&full[s], bytes);
                bulk_g2s(smem + s * (size_t)bytes, frags + ((size_t)c * a.heads + h) * bytes, bytes, &full[s]);
            }
            for (int i = c > S::kStages ? c - S::kStages : 0; i < c; i++)      // no copy is left in flight
                if (!mbar_wait_bounded(&full[i % S::kStages], (uint32_t)(i / S::kStages) & 1u, err, 66)) break;
        }
        return;
    }
    const int pair = warp & 1, block = 2 * blockIdx.y + pair;
    if (pair >= blocks) return;
    uint8_t* mine = s_state + (size_t)pair * 2 * S::kState + lane * 16;
    const float* up = updates + (size_t)h * update_floats(V) + (size_t)block * 512 + (warp >> 1) * 256 + lane * 8;
    const size_t next_up = (size_t)a.heads * update_floats(V);
    float4 u0 = *reinterpret_cast<const float4*>(up), u1 = *reinterpret_cast<const float4*>(up + 4);
    if (warp < 2) {
        // ---------------- the state, transposed: rows are value columns, columns are keys
        float st[NT][4];
        float* gs = a.state + (size_t)h * D * V + 16 * block + g4;
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int n = 8 * j + 2 * t4 + (e & 1);
                st[j][e] = n < D ? gs[(size_t)n * V + 8 * (e >> 1)] : 0.0f;
            }
        for (int c = 0; c < chunks; c++) {
            const int s = c % S::kStages, b = c & 1;
            if (!mbar_wait_bounded(&full[s], (uint32_t)(c / S::kStages) & 1u, err, 62)) break;
            if (c >= 2 && !mbar_wait_bounded(&state_empty[pair][b], (uint32_t)(c / 2 - 1) & 1u, err, 63)) break;
            const uint8_t* f = smem + s * (size_t)bytes;
            const uint32_t to = smem_addr(mine + b * S::kState);
            float x[2][4] = {{u0.x, u0.y, u0.z, u0.w}, {u1.x, u1.y, u1.z, u1.w}}, y[2][4] = {}, z[2][4] = {};
            if (c + 1 < chunks) {
                up += next_up;
                u0 = *reinterpret_cast<const float4*>(up);
                u1 = *reinterpret_cast<const float4*>(up + 4);
            }
            const uint4* fw = reinterpret_cast<const uint4*>(f) + lane;
            uint4 w0 = fw[0], w1 = fw[32];
#pragma unroll
            for (int ks = 0; ks < KS; ks++) {
                if (ks >= ks_n) break;
                uint4 n0 = w0, n1 = w1;
                if (ks + 1 < KS && ks + 1 < ks_n) { n0 = fw[(2 * ks + 2) * 32]; n1 = fw[(2 * ks + 3) * 32]; }
                uint32_t ah[4], al[4];
                split_bf16(st[2 * ks][0], st[2 * ks][1], ah[0], al[0]);
                split_bf16(st[2 * ks][2], st[2 * ks][3], ah[1], al[1]);
                split_bf16(st[2 * ks + 1][0], st[2 * ks + 1][1], ah[2], al[2]);
                split_bf16(st[2 * ks + 1][2], st[2 * ks + 1][3], ah[3], al[3]);
                store_shared(to + ks * 1024, ah);
                store_shared(to + ks * 1024 + 512, al);
                mma_bf16(x[0], ah, w0.x, w0.y);
                mma_bf16(x[1], ah, w1.x, w1.y);
                mma_bf16(y[0], ah, w0.z, w0.w);
                mma_bf16(y[1], ah, w1.z, w1.w);
                mma_bf16(z[0], al, w0.x, w0.y);
                mma_bf16(z[1], al, w1.x, w1.y);
                w0 = n0;
                w1 = n1;
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&state_full[pair][b]);
            const uint8_t* fk = f + (size_t)128 * D;
            const float* decay = reinterpret_cast<const float*>(f + (size_t)192 * D);
#pragma unroll
            for (int j = 0; j < NT; j++) {
                if (8 * j >= D) break;
                const float2 d = *reinterpret_cast<const float2*>(decay + 8 * j + 2 * t4);
                st[j][0] *= d.x; st[j][1] *= d.y; st[j][2] *= d.x; st[j][3] *= d.y;
            }
            uint32_t uh[4], ul[4];
#pragma unroll
            for (int e = 0; e < 2; e++) {
                split_bf16(x[e][0] + (y[e][0] + z[e][0]), x[e][1] + (y[e][1] + z[e][1]), uh[2 * e], ul[2 * e]);
                split_bf16(x[e][2] + (y[e][2] + z[e][2]), x[e][3] + (y[e][3] + z[e][3]), uh[2 * e + 1], ul[2 * e + 1]);
            }
#pragma unroll
            for (int j = 0; j < NT; j += 8) {
                if (8 * j >= D) break;
                uint4 kf[8];
#pragma unroll
                for (int i = 0; i < 8; i++) kf[i] = 8 * (j + i) < D ? *reinterpret_cast<const uint4*>(fk + ((j + i) * 32 + lane) * 16) : make_uint4(0, 0, 0, 0);
#pragma unroll
                for (int i = 0; i < 8; i++) mma_bf16(st[j + i], uh, kf[i].x, kf[i].y);
#pragma unroll
                for (int i = 0; i < 8; i++) mma_bf16(st[j + i], uh, kf[i].z, kf[i].w);
#pragma unroll
                for (int i = 0; i < 8; i++) mma_bf16(st[j + i], ul, kf[i].x, kf[i].y);
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[s]);
        }
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int n = 8 * j + 2 * t4 + (e & 1);
                if (n < D) gs[(size_t)n * V + 8 * (e >> 1)] = st[j][e];
            }
    } else {
        // ---------------- the read-out
        bf16* out = reinterpret_cast<bf16*>(a.o) + (size_t)h * V + 16 * block + (g4 & ~1);
        for (int c = 0; c < chunks; c++) {
            const int s = c % S::kStages, b = c & 1;
            if (!mbar_wait_bounded(&full[s], (uint32_t)(c / S::kStages) & 1u, err, 64)) break;
            if (!mbar_wait_bounded(&state_full[pair][b], (uint32_t)(c / 2) & 1u, err, 65)) break;
            const uint8_t* f = smem + s * (size_t)bytes + (size_t)64 * D;
            float x[2][4] = {{u0.x, u0.y, u0.z, u0.w}, {u1.x, u1.y, u1.z, u1.w}}, y[2][4] = {}, z[2][4] = {};
            if (c + 1 < chunks) {
                up += next_up;
                u0 = *reinterpret_cast<const float4*>(up);
                u1 = *reinterpret_cast<const float4*>(up + 4);
            }
            const uint4* fq = reinterpret_cast<const uint4*>(f) + lane;
            const uint4* from = reinterpret_cast<const uint4*>(mine + b * S::kState);
            uint4 hi = from[0], lo = from[32], w0 = fq[0], w1 = fq[32];
#pragma unroll
            for (int ks = 0; ks < KS; ks++) {
                if (ks >= ks_n) break;
                const uint32_t ah[4] = {hi.x, hi.y, hi.z, hi.w}, al[4] = {lo.x, lo.y, lo.z, lo.w};
                uint4 n0 = w0, n1 = w1;
                if (ks + 1 < KS && ks + 1 < ks_n) {
                    n0 = fq[(2 * ks + 2) * 32];
                    n1 = fq[(2 * ks + 3) * 32];
                    hi = from[(2 * ks + 2) * 32];
                    lo = from[(2 * ks + 3) * 32];
                }
                mma_bf16(x[0], ah, w0.x, w0.y);
                mma_bf16(x[1], ah, w1.x, w1.y);
                mma_bf16(y[0], ah, w0.z, w0.w);
                mma_bf16(y[1], ah, w1.z, w1.w);
                mma_bf16(z[0], al, w0.x, w0.y);
                mma_bf16(z[1], al, w1.x, w1.y);
                w0 = n0;
                w1 = n1;
            }
            __syncwarp();
            if (lane == 0) { mbar_arrive(&state_empty[pair][b]); mbar_arrive(&empty[s]); }
            // two neighbouring columns per store: lanes of even columns finish even tokens, those of odd ones odd tokens
            const bool odd = g4 & 1;
#pragma unroll
            for (int e = 0; e < 2; e++)
#pragma unroll
                for (int r = 0; r < 4; r += 2) {
                    const float v0 = x[e][r] + (y[e][r] + z[e][r]), v1 = x[e][r + 1] + (y[e][r + 1] + z[e][r + 1]);
                    const float other = __shfl_xor_sync(0xFFFFFFFFu, odd ? v0 : v1, 4);
                    const int t = t0 + kChunk * c + 8 * e + 2 * t4 + odd;
                    if (t < t1)
                        *reinterpret_cast<uint32_t*>(out + (size_t)t * a.heads * V + 4 * r) = odd ? pack_bf16(other, v1) : pack_bf16(v0, other);
                }
        }
    }
}

template <int NMAX, bool kExact>
static int launch_chunks(const DeltaRule& a, int T, cudaStream_t s)
{
    int rc = allow_smem<k_delta_chunks<NMAX, kExact>>((int)DeltaChunks<NMAX>::smem(NMAX));
    if (rc) return rc;
    constexpr auto prepare = k_delta_prepare<NMAX == 256 ? 256 : 128, NMAX == 256 ? 1 : 3>;
    if ((rc = allow_smem<prepare>((int)fragment_bytes(256)))) return rc;
    for (int t0 = 0; t0 < T; t0 += kSegmentChunks * kChunk) {
        const int t1 = T - t0 < kSegmentChunks * kChunk ? T : t0 + kSegmentChunks * kChunk, chunks = (t1 - t0 + kChunk - 1) / kChunk;
        uint8_t* frags = (uint8_t*)a.scratch;
        float* updates = (float*)(frags + (size_t)chunks * a.heads * fragment_bytes(a.key_pad));
        if ((rc = launch_ordered(prepare, dim3(a.heads, chunks), (a.key_pad + 31) / 32 * 32, fragment_bytes(a.key_pad), s, a, frags, updates, t0, t1)))
            return rc;
        if ((rc = launch_ordered(k_delta_chunks<NMAX, kExact>, dim3(a.heads, (a.value_pad + 31) / 32), 160, DeltaChunks<NMAX>::smem(a.key_pad), s, a,
                                 (const uint8_t*)frags, (const float*)updates, t0, t1, chunks, device_error_flag())))
            return rc;
    }
    return 0;
}

// ------------------------------------------------------------------ host side

// From this many tokens on a bf16 prompt goes through the chunked kernels.
constexpr int kChunkedMinTokens = 32;
static bool takes_chunks(int key_pad, int T, bool act_bf16) { return act_bf16 && T >= kChunkedMinTokens && key_pad <= 256; }

size_t delta_scratch_bytes(int heads, int key_pad, int value_pad, int T, bool act_bf16)
{
    if (!takes_chunks(key_pad, T, act_bf16)) return 0;
    const int chunks = (T + kChunk - 1) / kChunk;
    return (size_t)(chunks < kSegmentChunks ? chunks : kSegmentChunks) * heads * (fragment_bytes(key_pad) + 4 * update_floats(value_pad));
}

int delta_rule(const DeltaRule& a, int T, bool act_bf16, cudaStream_t s)
{
    if (a.heads < 1 || a.groups < 1 || a.heads % a.groups || a.key_pad % 16 || a.value_pad % 16 || a.ld % 8 || T < 1) return latch(BPDQ_ERR_ARG);
    if (a.key_pad > 512) return latch(BPDQ_ERR_RANGE);
    if (a.norm_w && (T > 1 || !a.gate || !delta_token_norms(a.key_pad, a.value_pad))) return latch(BPDQ_ERR_ARG);
    if (T == 1) return act_bf16 ? delta_token<bf16>(a, s) : delta_token<float>(a, s);
    if (a.scratch && takes_chunks(a.key_pad, T, act_bf16)) {
        if (a.key_pad == 64) return launch_chunks<64, true>(a, T, s);
        if (a.key_pad == 128) return launch_chunks<128, true>(a, T, s);
        if (a.key_pad < 64) return launch_chunks<64, false>(a, T, s);
        if (a.key_pad < 128) return launch_chunks<128, false>(a, T, s);
        return launch_chunks<256, false>(a, T, s);
    }
    return act_bf16 ? delta_recurrence<bf16>(a, T, s) : delta_recurrence<float>(a, T, s);
}

}  // namespace bpdq

using namespace bpdq;

extern "C" {

int bpd_delta_rule_cuda(const void* q, const void* k, const void* v, int ld, const float* log_decay, const float* beta, float q_scale, float unit_eps,
                        float* state, void* o, const float* norm_w, const void* gate, float eps, int n_tokens, int heads, int groups, int key_pad,
                        int value_dim, int value_pad, int act_bf16, void* stream)
{
    if (n_tokens < 0 || heads < 1 || groups < 1 || key_pad < 16 || value_pad < 16 || value_dim < 1 || value_dim > value_pad) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!q || !k || !v || !log_decay || !beta || !state || !o) return latch(BPDQ_ERR_ARG);
    DeltaRule a = {};
    a.q = q; a.k = k; a.v = v;
    a.ld = ld;
    a.heads = heads; a.groups = groups; a.key_pad = key_pad; a.value_dim = value_dim; a.value_pad = value_pad;
    a.log_decay = log_decay;
    a.beta = beta;
    a.q_scale = q_scale; a.unit_eps = unit_eps;
    a.state = state;
    a.o = o;
    a.norm_w = norm_w; a.gate = gate; a.eps = eps;
    const size_t scratch = delta_scratch_bytes(heads, key_pad, value_pad, n_tokens, act_bf16 != 0);
    if (scratch) {
        int rc = 0;
        if (!(a.scratch = scratch_take(nullptr, kScratchDelta, scratch, (cudaStream_t)stream, &rc))) return rc;
    }
    return delta_rule(a, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

}  // extern "C"
