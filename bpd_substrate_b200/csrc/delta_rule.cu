// Gated delta rule.
//
//   k_delta_token       one token: a cluster of CTAs per head, each with 32 value columns; the state goes through HBM once.
//                       Unit lengths, prediction and read-out come from one pass over the state (the read-out of the written
//                       state is the read-out of the decayed one plus (k.q) u); the output's norm joins its CTAs through
//                       distributed shared memory.
//   k_delta_recurrence  token by token: a warp holds four value columns of a head, eight lanes over the keys, so that a token
//                       costs three shuffles and no barrier.  Short portions, fp32 runs.
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
        o = make_float4(o.x * f * nw.x * sigmoid_f32(gate.x), o.y * f * nw.y * sigmoid_f32(gate.y), o.z * f * nw.z * sigmoid_f32(gate.z),
                        o.w * f * nw.w * sigmoid_f32(gate.w));
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

// ------------------------------------------------------------------ host side

int delta_rule(const DeltaRule& a, int T, bool act_bf16, cudaStream_t s)
{
    if (a.heads < 1 || a.groups < 1 || a.heads % a.groups || a.key_pad % 16 || a.value_pad % 16 || a.ld % 8 || T < 1) return latch(BPDQ_ERR_ARG);
    if (a.key_pad > 512) return latch(BPDQ_ERR_RANGE);
    if (a.norm_w && (T > 1 || !a.gate || !delta_token_norms(a.key_pad, a.value_pad))) return latch(BPDQ_ERR_ARG);
    if (T == 1) return act_bf16 ? delta_token<bf16>(a, s) : delta_token<float>(a, s);
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
    return delta_rule(a, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

}  // extern "C"
