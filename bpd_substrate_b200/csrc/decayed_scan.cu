// Linear attention with a decaying state and the small steps around it.
//
//   k_decayed_recurrence  token by token: a CTA holds the state of one head and 64 value columns in registers.  Decoding
//                         (the state goes through HBM once per token, all its loads in flight at once), short portions
//                         of a prompt, and every fp32 run.
//   k_decayed_chunks      a prompt's portion in chunks of 64 tokens on the tensor cores (mma.sync bf16, fp32
//                         accumulation): scores of a chunk against itself, decayed and masked in fp32; the state stays
//                         in fp32 accumulators from chunk to chunk.  Whatever is fp32 by nature (decayed scores, the
//                         state, weighted values) enters a product as the sum of two bf16 numbers, so nothing of the
//                         recurrence is rounded to bf16.
#include "decayed_scan.cuh"
#include "launch.cuh"
#include "mma_device.cuh"
#include "../../include/bpdq.h"

namespace bpdq {

// ------------------------------------------------------------------ recurrence

// 256 threads: 16 groups of four value columns x 16 key phases; a thread keeps keys n = phase + 16 i, i < NI.
template <typename A, int NI>
__global__ void __launch_bounds__(256) k_decayed_recurrence(DecayedScan a, int T)
{
    __shared__ float sq[2][16 * NI], sk[2][16 * NI];
    __shared__ float red[16][64];
    const int tid = threadIdx.x, cg = tid & 15, ng = tid >> 4;
    const int h = blockIdx.x, g = h / (a.heads / a.groups), p = blockIdx.y * 64 + 4 * cg;
    const bool live = p < a.value_pad;
    pdl_launch_dependents();
    pdl_wait();
    float4 s[NI];
    float* st = a.state + (size_t)h * a.key_pad * a.value_pad + p;
#pragma unroll
    for (int i = 0; i < NI; i++) {
        const int n = ng + 16 * i;
        s[i] = (live && n < a.key_pad) ? *reinterpret_cast<const float4*>(st + (size_t)n * a.value_pad) : make_float4(0, 0, 0, 0);
    }
    const A* q = reinterpret_cast<const A*>(a.q) + g * a.key_pad;
    const A* k = reinterpret_cast<const A*>(a.k) + g * a.key_pad;
    const A* v = reinterpret_cast<const A*>(a.v) + h * a.value_pad;
    A* o = reinterpret_cast<A*>(a.o) + h * a.value_pad;
    const float skip = a.d_skip ? a.d_skip[h] : 0.0f;
    const float fixed = a.decay ? a.decay[h] : 0.0f, rate = a.neg_exp_a ? a.neg_exp_a[h] : 0.0f;
    for (int t = 0; t < T; t++) {
        float* cq = sq[t & 1];
        float* ck = sk[t & 1];
        const A *qt = q + (size_t)t * a.ld_q, *kt = k + (size_t)t * a.ld_k;
        if (a.rot_freq) {
            const int half = a.rot_dims / 2, pos = *a.pos + t;
            for (int n = tid; n < 16 * NI; n += 256) {
                float qv = 0, kv = 0;
                if (n < a.key_pad) {
                    qv = act_load(qt + n);
                    kv = act_load(kt + n);
                    if (n < a.rot_dims) {
                        const int i = n < half ? n : n - half, m = n < half ? n + half : n - half;
                        float sn, cs;
                        sincosf((float)pos * a.rot_freq[i], &sn, &cs);
                        const float qo = act_load(qt + m), ko = act_load(kt + m);
                        qv = n < half ? qv * cs - qo * sn : qv * cs + qo * sn;
                        kv = n < half ? kv * cs - ko * sn : kv * cs + ko * sn;
                    }
                }
                cq[n] = qv;
                ck[n] = kv * a.k_scale;
            }
        } else {
            for (int n = tid; n < 16 * NI; n += 256) {
                cq[n] = n < a.key_pad ? act_load(qt + n) : 0.0f;
                ck[n] = n < a.key_pad ? act_load(kt + n) : 0.0f;
            }
        }
        const float4 vv = live ? act_load4(v + (size_t)t * a.ld_v + p) : make_float4(0, 0, 0, 0);
        float4 wv = vv;
        float decay = fixed;
        if (a.dt) {
            const float dt = a.dt[(size_t)t * a.ld_dt + h];
            // an fp32 exponential that leans one way by a unit in the last place adds up over thousands of tokens
            decay = sizeof(A) == 4 ? (float)exp((double)rate * (double)dt) : expf(rate * dt);
            wv = make_float4(vv.x * dt, vv.y * dt, vv.z * dt, vv.w * dt);
        }
        __syncthreads();
        float4 acc = make_float4(0, 0, 0, 0);
#pragma unroll
        for (int i = 0; i < NI; i++) {
            const float kn = ck[ng + 16 * i], qn = cq[ng + 16 * i];
            s[i].x = fmaf(s[i].x, decay, kn * wv.x); acc.x = fmaf(qn, s[i].x, acc.x);
            s[i].y = fmaf(s[i].y, decay, kn * wv.y); acc.y = fmaf(qn, s[i].y, acc.y);
            s[i].z = fmaf(s[i].z, decay, kn * wv.z); acc.z = fmaf(qn, s[i].z, acc.z);
            s[i].w = fmaf(s[i].w, decay, kn * wv.w); acc.w = fmaf(qn, s[i].w, acc.w);
        }
        *reinterpret_cast<float4*>(&red[ng][4 * cg]) = acc;
        __syncthreads();
        if (tid < 64 && blockIdx.y * 64 + tid < a.value_pad) {
            const int c = blockIdx.y * 64 + tid;
            float r = 0.0f;
#pragma unroll
            for (int i = 0; i < 16; i++) r += red[i][tid];
            if (a.d_skip) r = fmaf(skip, act_load(v + (size_t)t * a.ld_v + c), r);
            o[(size_t)t * a.ld_o + c] = act_from<A>(r);
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < NI; i++) {
            const int n = ng + 16 * i;
            if (n < a.key_pad) *reinterpret_cast<float4*>(st + (size_t)n * a.value_pad) = s[i];
        }
    }
}

// ------------------------------------------------------------------ chunks of 64 tokens on the tensor cores

constexpr int kChunk = 64;

template <int NMAX>
struct ChunkShape {
    static constexpr int kLdN = NMAX + 8, kLdV = 72, kLdO = 68;
    static constexpr size_t kQK = (size_t)kChunk * kLdN * 2, kV = (size_t)kChunk * kLdV * 2;
    static constexpr size_t kSmem = 2 * (2 * kQK + kV) + 2 * kV + (size_t)kChunk * kLdO * 4 + 5 * kChunk * 4;
};

// One CTA: one head, 64 value columns, all tokens.  Eight warps: value rows 16 (w & 3) .. + 15 of the transposed state
// and half (w >> 2) of its keys.
template <int NMAX>
__global__ void __launch_bounds__(256, 1) k_decayed_chunks(DecayedScan a, int T)
{
    using S = ChunkShape<NMAX>;
    constexpr int LDN = S::kLdN, LDV = S::kLdV, LDO = S::kLdO;
    constexpr int NH = NMAX / 2, NTILES = NH / 8;
    extern __shared__ __align__(128) uint8_t smem[];
    bf16* sQ[2] = {reinterpret_cast<bf16*>(smem), reinterpret_cast<bf16*>(smem + S::kQK)};
    bf16* sK[2] = {reinterpret_cast<bf16*>(smem + 2 * S::kQK), reinterpret_cast<bf16*>(smem + 3 * S::kQK)};
    bf16* sV[2] = {reinterpret_cast<bf16*>(smem + 4 * S::kQK), reinterpret_cast<bf16*>(smem + 4 * S::kQK + S::kV)};
    bf16* sPh = reinterpret_cast<bf16*>(smem + 4 * S::kQK + 2 * S::kV);
    bf16* sPl = sPh + kChunk * LDV;
    float* sO = reinterpret_cast<float*>(smem + 4 * S::kQK + 4 * S::kV);
    float* sL = sO + kChunk * LDO;                 // [2][64] cumulative log decay of a chunk, inclusive
    float* sDt = sL + 2 * kChunk;                  // [2][64]
    float* sW = sDt + 2 * kChunk;                  // [64] weight of a token in the chunk's final state

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
    const int pw = warp & 3, half = warp >> 2;
    const int h = blockIdx.x, grp = h / (a.heads / a.groups), p0 = blockIdx.y * 64;
    const int p_n = a.value_pad - p0 < 64 ? a.value_pad - p0 : 64;
    const int Np = a.key_pad;
    const bf16* gq = reinterpret_cast<const bf16*>(a.q) + grp * Np;
    const bf16* gk = reinterpret_cast<const bf16*>(a.k) + grp * Np;
    const bf16* gv = reinterpret_cast<const bf16*>(a.v) + h * a.value_pad + p0;
    pdl_launch_dependents();
    // columns beyond the head's own sizes are never loaded: zero in both buffers
    for (size_t i = tid; i < (4 * S::kQK + 2 * S::kV) / 16; i += 256) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
    const float fixed = a.log_decay ? a.log_decay[h] : 0.0f;
    const float rate = a.neg_exp_a ? a.neg_exp_a[h] : 0.0f;
    const float skip = a.d_skip ? a.d_skip[h] : 0.0f;
    __syncthreads();
    pdl_wait();

    auto load_chunk = [&](int c, int b) {
        const int t0 = c * kChunk;
        const int un = Np / 8, uv = p_n / 8;
        for (int i = tid; i < kChunk * un; i += 256) {
            const int r = i / un, u = i - r * un, t = t0 + r;
            const int tc = t < T ? t : T - 1;
            cp_async16(sQ[b] + r * LDN + 8 * u, gq + (size_t)tc * a.ld_q + 8 * u, t < T);
            cp_async16(sK[b] + r * LDN + 8 * u, gk + (size_t)tc * a.ld_k + 8 * u, t < T);
        }
        for (int i = tid; i < kChunk * uv; i += 256) {
            const int r = i / uv, u = i - r * uv, t = t0 + r;
            const int tc = t < T ? t : T - 1;
            cp_async16(sV[b] + r * LDV + 8 * u, gv + (size_t)tc * a.ld_v + 8 * u, t < T);
        }
        cp_async_commit();
    };
    // lane i of warp 0 holds tokens 2 i and 2 i + 1 of a chunk
    auto dt_of = [&](int c, float& d0, float& d1) {
        const int t = c * kChunk + 2 * lane;
        d0 = t < T ? (a.dt ? a.dt[(size_t)t * a.ld_dt + h] : 1.0f) : 0.0f;
        d1 = t + 1 < T ? (a.dt ? a.dt[(size_t)(t + 1) * a.ld_dt + h] : 1.0f) : 0.0f;
    };
    auto scan_decays = [&](float d0, float d1, int b) {
        const float l0 = a.dt ? rate * d0 : fixed * d0, l1 = a.dt ? rate * d1 : fixed * d1;    // no decay beyond the last token
        float sum = l0 + l1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xFFFFFFFFu, sum, o);
            if (lane >= o) sum += u;
        }
        sL[b * kChunk + 2 * lane] = sum - l1;
        sL[b * kChunk + 2 * lane + 1] = sum;
        sDt[b * kChunk + 2 * lane] = d0;
        sDt[b * kChunk + 2 * lane + 1] = d1;
    };

    // the state, transposed: rows p = 16 pw + .., columns n = NH half + ..
    float st[NTILES][4];
    float* gs = a.state + (size_t)h * Np * a.value_pad + p0;
#pragma unroll
    for (int j = 0; j < NTILES; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int n = half * NH + 8 * j + 2 * t4 + (e & 1), p = 16 * pw + g4 + 8 * (e >> 1);
            st[j][e] = (n < Np && p < p_n) ? gs[(size_t)n * a.value_pad + p] : 0.0f;
        }

    const int chunks = (T + kChunk - 1) / kChunk;
    load_chunk(0, 0);
    if (warp == 0) {
        float d0, d1;
        dt_of(0, d0, d1);
        scan_decays(d0, d1, 0);
    }
    for (int c = 0; c < chunks; c++) {
        const int b = c & 1;
        cp_async_wait_all();
        __syncthreads();                            // this chunk is here; everybody has left the other buffer
        float d0 = 0, d1 = 0;
        if (c + 1 < chunks) {
            load_chunk(c + 1, b ^ 1);
            if (warp == 0) dt_of(c + 1, d0, d1);
        }
        const float* L = sL + b * kChunk;
        const float* Dt = sDt + b * kChunk;
        const float total = L[kChunk - 1];
        if (tid < kChunk) sW[tid] = expf(total - L[tid]) * Dt[tid];

        // ---- scores of the chunk: rows i = 16 pw .., columns j = 32 half ..; decay and mask in fp32
        {
            float acc[4][4] = {};
#pragma unroll
            for (int kk = 0; kk < NMAX / 16; kk++) {
                if (16 * kk >= Np) break;
                uint32_t af[4], b0[4], b1[4];
                ldsm4(af, sQ[b] + (16 * pw + (lane & 15)) * LDN + 16 * kk + 8 * (lane >> 4));
                const int jr = 32 * half + (lane & 7) + 8 * (lane >> 4), jc = 16 * kk + 8 * ((lane >> 3) & 1);
                ldsm4(b0, sK[b] + jr * LDN + jc);
                ldsm4(b1, sK[b] + (jr + 16) * LDN + jc);
                mma_bf16(acc[0], af, b0[0], b0[1]);
                mma_bf16(acc[1], af, b0[2], b0[3]);
                mma_bf16(acc[2], af, b1[0], b1[1]);
                mma_bf16(acc[3], af, b1[2], b1[3]);
            }
#pragma unroll
            for (int j = 0; j < 4; j++)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int i = 16 * pw + g4 + 4 * e, col = 32 * half + 8 * j + 2 * t4;
                    const float v0 = col <= i ? acc[j][e] * expf(L[i] - L[col]) * Dt[col] : 0.0f;
                    const float v1 = col + 1 <= i ? acc[j][e + 1] * expf(L[i] - L[col + 1]) * Dt[col + 1] : 0.0f;
                    uint32_t hi, lo;
                    split_bf16(v0, v1, hi, lo);
                    *reinterpret_cast<uint32_t*>(sPh + i * LDV + col) = hi;
                    *reinterpret_cast<uint32_t*>(sPl + i * LDV + col) = lo;
                }
        }
        // ---- what the state before the chunk gives: o^T[p][i] += S^T[p][n] q[i][n], then the decay up to token i
        float o[8][4] = {};
#pragma unroll
        for (int kk = 0; kk < NH / 16; kk++) {
            if (half * NH + 16 * kk >= Np) break;
            uint32_t ah[4], al[4];
            split_bf16(st[2 * kk][0], st[2 * kk][1], ah[0], al[0]);
            split_bf16(st[2 * kk][2], st[2 * kk][3], ah[1], al[1]);
            split_bf16(st[2 * kk + 1][0], st[2 * kk + 1][1], ah[2], al[2]);
            split_bf16(st[2 * kk + 1][2], st[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
            for (int ct = 0; ct < 8; ct += 2) {
                uint32_t bq[4];
                ldsm4(bq, sQ[b] + (8 * ct + (lane & 7) + 8 * (lane >> 4)) * LDN + half * NH + 16 * kk + 8 * ((lane >> 3) & 1));
                mma_bf16(o[ct], ah, bq[0], bq[1]);
                mma_bf16(o[ct], al, bq[0], bq[1]);
                mma_bf16(o[ct + 1], ah, bq[2], bq[3]);
                mma_bf16(o[ct + 1], al, bq[2], bq[3]);
            }
        }
#pragma unroll
        for (int ct = 0; ct < 8; ct++) {
            const float e0 = expf(L[8 * ct + 2 * t4]), e1 = expf(L[8 * ct + 2 * t4 + 1]);
            o[ct][0] *= e0; o[ct][1] *= e1; o[ct][2] *= e0; o[ct][3] *= e1;
        }
        __syncthreads();                            // scores and sW are complete
        // ---- the chunk's own tokens: o^T[p][i] += v[j][p] P[i][j], j in this warp's half
#pragma unroll
        for (int kk = 0; kk < 2; kk++) {
            const int j0 = 32 * half + 16 * kk;
            uint32_t av[4];
            ldsm4_t(av, sV[b] + (j0 + (lane & 7) + 8 * (lane >> 4)) * LDV + 16 * pw + 8 * ((lane >> 3) & 1));
#pragma unroll
            for (int ct = 0; ct < 8; ct += 2) {
                if (j0 > 8 * ct + 15) continue;     // later tokens only
                const int off = (8 * ct + (lane & 7) + 8 * (lane >> 4)) * LDV + j0 + 8 * ((lane >> 3) & 1);
                uint32_t bh[4], bl[4];
                ldsm4(bh, sPh + off);
                ldsm4(bl, sPl + off);
                mma_bf16(o[ct], av, bh[0], bh[1]);
                mma_bf16(o[ct], av, bl[0], bl[1]);
                mma_bf16(o[ct + 1], av, bh[2], bh[3]);
                mma_bf16(o[ct + 1], av, bl[2], bl[3]);
            }
        }
        // ---- the two halves' parts are joined: tokens 0..31 by half 0, 32..63 by half 1
#pragma unroll
        for (int ct = 0; ct < 8; ct++)
            if ((ct >> 2) != half)
#pragma unroll
                for (int e = 0; e < 4; e++) sO[(8 * ct + 2 * t4 + (e & 1)) * LDO + 16 * pw + g4 + 8 * (e >> 1)] = o[ct][e];
        // ---- the state after the chunk
        const float carry = expf(total);
#pragma unroll
        for (int j = 0; j < NTILES; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) st[j][e] *= carry;
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            const int j0 = 16 * kk;
            uint32_t av[4], ah[4], al[4];
            ldsm4_t(av, sV[b] + (j0 + (lane & 7) + 8 * (lane >> 4)) * LDV + 16 * pw + 8 * ((lane >> 3) & 1));
            const float w0 = sW[j0 + 2 * t4], w1 = sW[j0 + 2 * t4 + 1], w2 = sW[j0 + 2 * t4 + 8], w3 = sW[j0 + 2 * t4 + 9];
            split_bf16(bf_lo(av[0]) * w0, bf_hi(av[0]) * w1, ah[0], al[0]);
            split_bf16(bf_lo(av[1]) * w0, bf_hi(av[1]) * w1, ah[1], al[1]);
            split_bf16(bf_lo(av[2]) * w2, bf_hi(av[2]) * w3, ah[2], al[2]);
            split_bf16(bf_lo(av[3]) * w2, bf_hi(av[3]) * w3, ah[3], al[3]);
#pragma unroll
            for (int j = 0; j < NTILES; j += 2) {
                if (half * NH + 8 * j >= Np) break;
                uint32_t bk[4];
                ldsm4_t(bk, sK[b] + (j0 + (lane & 7) + 8 * ((lane >> 3) & 1)) * LDN + half * NH + 8 * j + 8 * (lane >> 4));
                mma_bf16(st[j], ah, bk[0], bk[1]);
                mma_bf16(st[j], al, bk[0], bk[1]);
                mma_bf16(st[j + 1], ah, bk[2], bk[3]);
                mma_bf16(st[j + 1], al, bk[2], bk[3]);
            }
        }
        if (warp == 0 && c + 1 < chunks) scan_decays(d0, d1, b ^ 1);
        __syncthreads();                            // the other half's part is in sO
#pragma unroll
        for (int ct = 0; ct < 8; ct++)
            if ((ct >> 2) == half)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int i = 8 * ct + 2 * t4 + (e & 1), p = 16 * pw + g4 + 8 * (e >> 1);
                    sO[i * LDO + p] += o[ct][e];
                }
        __syncthreads();
        for (int i = tid; i < kChunk * 16; i += 256) {
            const int r = i >> 4, u = 4 * (i & 15), t = c * kChunk + r;
            if (t < T && u < p_n) {
                float4 v = *reinterpret_cast<const float4*>(sO + r * LDO + u);
                if (a.d_skip) {
                    const float4 x = act_load4(sV[b] + r * LDV + u);
                    v.x = fmaf(skip, x.x, v.x); v.y = fmaf(skip, x.y, v.y); v.z = fmaf(skip, x.z, v.z); v.w = fmaf(skip, x.w, v.w);
                }
                uint2 w;
                w.x = pack_bf16(v.x, v.y);
                w.y = pack_bf16(v.z, v.w);
                *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(a.o) + (size_t)t * a.ld_o + h * a.value_pad + p0 + u) = w;
            }
        }
    }
#pragma unroll
    for (int j = 0; j < NTILES; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int n = half * NH + 8 * j + 2 * t4 + (e & 1), p = 16 * pw + g4 + 8 * (e >> 1);
            if (n < Np && p < p_n) gs[(size_t)n * a.value_pad + p] = st[j][e];
        }
}

template <typename A>
static int launch_recurrence(const DecayedScan& a, int T, cudaStream_t s)
{
    const dim3 grid(a.heads, (a.value_pad + 63) / 64);
    if (a.key_pad <= 64) return launch_ordered(k_decayed_recurrence<A, 4>, grid, 256, 0, s, a, T);
    if (a.key_pad <= 128) return launch_ordered(k_decayed_recurrence<A, 8>, grid, 256, 0, s, a, T);
    if (a.key_pad <= 256) return launch_ordered(k_decayed_recurrence<A, 16>, grid, 256, 0, s, a, T);
    if (a.key_pad <= 512) return launch_ordered(k_decayed_recurrence<A, 32>, grid, 256, 0, s, a, T);
    return latch(BPDQ_ERR_RANGE);
}

template <int NMAX>
static int launch_chunks(const DecayedScan& a, int T, cudaStream_t s)
{
    int rc = allow_smem<k_decayed_chunks<NMAX>>((int)ChunkShape<NMAX>::kSmem);
    if (rc) return rc;
    return launch_ordered(k_decayed_chunks<NMAX>, dim3(a.heads, (a.value_pad + 63) / 64), 256, ChunkShape<NMAX>::kSmem, s, a, T);
}

// From this many tokens on a bf16 prompt goes through the chunked kernel.
constexpr int kChunkedMinTokens = 24;

int decayed_scan(const DecayedScan& a, int T, bool act_bf16, cudaStream_t s)
{
    if (a.heads < 1 || a.groups < 1 || a.heads % a.groups || a.key_pad % 16 || a.value_pad % 16 || T < 1) return latch(BPDQ_ERR_ARG);
    if (act_bf16 && T >= kChunkedMinTokens && !a.rot_freq && a.key_pad <= 256) {
        if (a.key_pad <= 64) return launch_chunks<64>(a, T, s);
        if (a.key_pad <= 128) return launch_chunks<128>(a, T, s);
        return launch_chunks<256>(a, T, s);
    }
    return act_bf16 ? launch_recurrence<bf16>(a, T, s) : launch_recurrence<float>(a, T, s);
}

// ------------------------------------------------------------------ rotary positions, rotate-half pairs

// Thread = (token, pair or unrotated entry of a head), all heads: one sine and cosine for all of them.
template <typename A>
__global__ void __launch_bounds__(128) k_rotate_half_qk(A* q, A* k, int ld, int heads, int dim_pad, int rot_dims,
                                                        const float* __restrict__ freq, float k_scale, const int* pos)
{
    pdl_launch_dependents();
    pdl_wait();
    const int half = rot_dims / 2, per = dim_pad - half, t = blockIdx.y;
    const int i = blockIdx.x * 128 + threadIdx.x;
    if (i >= per) return;
    A* pq = q + (size_t)t * ld;
    A* pk = k + (size_t)t * ld;
    if (i < half) {
        float sn, cs;
        sincosf((float)(*pos + t) * freq[i], &sn, &cs);
#pragma unroll 4
        for (int h = 0; h < heads; h++, pq += dim_pad, pk += dim_pad) {
            const float q0 = act_load(pq + i), q1 = act_load(pq + i + half), k0 = act_load(pk + i), k1 = act_load(pk + i + half);
            pq[i] = act_from<A>(q0 * cs - q1 * sn);
            pq[i + half] = act_from<A>(q1 * cs + q0 * sn);
            pk[i] = act_from<A>((k0 * cs - k1 * sn) * k_scale);
            pk[i + half] = act_from<A>((k1 * cs + k0 * sn) * k_scale);
        }
    } else {
        const int n = half + i;         // k's unrotated entries are scaled too
        for (int h = 0; h < heads; h++, pk += dim_pad) pk[n] = act_from<A>(act_load(pk + n) * k_scale);
    }
}

int rotate_half_qk(void* q, void* k, int ld, int heads, int dim_pad, int rot_dims, const float* rot_freq, float k_scale,
                   const int* pos, int T, bool act_bf16, cudaStream_t s)
{
    const dim3 grid((dim_pad - rot_dims / 2 + 127) / 128, T);
    if (act_bf16)
        return launch_ordered(k_rotate_half_qk<bf16>, grid, 128, 0, s, (bf16*)q, (bf16*)k, ld, heads, dim_pad, rot_dims, rot_freq, k_scale, pos);
    return launch_ordered(k_rotate_half_qk<float>, grid, 128, 0, s, (float*)q, (float*)k, ld, heads, dim_pad, rot_dims, rot_freq, k_scale, pos);
}

// ------------------------------------------------------------------ causal convolution

constexpr int kConvTile = 32;      // tokens per thread

// Thread = (NC neighbouring channels, tile of tokens), the window in registers (up to four taps) or read again per token.
template <typename A, int NC>
__global__ void __launch_bounds__(128) k_causal_conv(const A* in, int ld_in, A* out, int channels, int taps,
                                                     const float* __restrict__ w, const float* __restrict__ b, const float* tail, int T)
{
    struct alignas(NC * sizeof(A)) Group { A v[NC]; };
    struct alignas(NC * 4) Floats { float v[NC]; };
    pdl_launch_dependents();
    const int c = NC * (blockIdx.x * 128 + threadIdx.x);
    if (c >= channels) return;
    const int t0 = blockIdx.y * kConvTile, t1 = t0 + kConvTile < T ? t0 + kConvTile : T;
    auto floats = [&](const float* p) -> Floats { return *reinterpret_cast<const Floats*>(p + c); };
    Floats bias = {};
    if (b) bias = floats(b);
    auto input = [&](int t) -> Floats {      // t >= -(taps - 1)
        if (t < 0) return floats(tail + (size_t)(t + taps - 1) * channels);
        const Group g = *reinterpret_cast<const Group*>(in + (size_t)t * ld_in + c);
        Floats f;
#pragma unroll
        for (int i = 0; i < NC; i++) f.v[i] = act_load(&g.v[i]);
        return f;
    };
    auto store = [&](int t, const Floats& f) {
        Group g;
#pragma unroll
        for (int i = 0; i < NC; i++) g.v[i] = act_from<A>(silu_act<A>(f.v[i]));
        *reinterpret_cast<Group*>(out + (size_t)t * channels + c) = g;
    };
    if (taps <= 4) {
        Floats wv[4], win[3];
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int jj = j - (4 - taps);      // the last tap is always slot 3
            wv[j] = Floats{};
            if (jj >= 0) wv[j] = floats(w + (size_t)jj * channels);
        }
        pdl_wait();
#pragma unroll
        for (int j = 0; j < 3; j++) {
            win[j] = Floats{};
            if (j - (4 - taps) >= 0) win[j] = input(t0 - 3 + j);
        }
        for (int tb = t0; tb < t1; tb += 8) {
            Floats x[8];
#pragma unroll
            for (int i = 0; i < 8; i++) {
                x[i] = Floats{};
                if (tb + i < t1) x[i] = input(tb + i);
            }
#pragma unroll
            for (int i = 0; i < 8; i++) {
                Floats acc = bias;
#pragma unroll
                for (int k = 0; k < NC; k++) {
                    acc.v[k] = fmaf(wv[0].v[k], win[0].v[k], acc.v[k]);
                    acc.v[k] = fmaf(wv[1].v[k], win[1].v[k], acc.v[k]);
                    acc.v[k] = fmaf(wv[2].v[k], win[2].v[k], acc.v[k]);
                    acc.v[k] = fmaf(wv[3].v[k], x[i].v[k], acc.v[k]);
                }
                if (tb + i < t1) store(tb + i, acc);
                win[0] = win[1]; win[1] = win[2]; win[2] = x[i];
            }
        }
    } else {
        pdl_wait();
        for (int t = t0; t < t1; t++) {
            Floats acc = bias;
            for (int j = 0; j < taps; j++) {
                const Floats x = input(t - taps + 1 + j), wj = floats(w + (size_t)j * channels);
#pragma unroll
                for (int k = 0; k < NC; k++) acc.v[k] = fmaf(wj.v[k], x.v[k], acc.v[k]);
            }
            store(t, acc);
        }
    }
}

// The window after T tokens.  A thread owns a channel and moves its entries in order, so the old ones are read first.
template <typename A>
__global__ void __launch_bounds__(128) k_conv_tail(const A* in, int ld_in, int channels, int taps, float* tail, int T)
{
    pdl_launch_dependents();
    pdl_wait();
    const int c = blockIdx.x * 128 + threadIdx.x;
    if (c >= channels) return;
    for (int j = 0; j < taps - 1; j++) {
        const int t = T - (taps - 1) + j;
        tail[(size_t)j * channels + c] = t >= 0 ? act_load(in + (size_t)t * ld_in + c) : tail[(size_t)(j + T) * channels + c];
    }
}

template <typename A>
static int launch_conv(const void* in, int ld_in, void* out, int channels, int taps, const float* w, const float* b, float* tail,
                       int T, cudaStream_t s)
{
    const bool pairs = channels % 2 == 0 && ld_in % 2 == 0 && !(((uintptr_t)in | (uintptr_t)out) % (2 * sizeof(A)));
    const dim3 grid((channels / (pairs ? 2 : 1) + 127) / 128, (T + kConvTile - 1) / kConvTile);
    int rc = pairs ? launch_ordered(k_causal_conv<A, 2>, grid, 128, 0, s, (const A*)in, ld_in, (A*)out, channels, taps, w, b, (const float*)tail, T)
                   : launch_ordered(k_causal_conv<A, 1>, grid, 128, 0, s, (const A*)in, ld_in, (A*)out, channels, taps, w, b, (const float*)tail, T);
    if (rc || taps < 2) return rc;
    return launch_ordered(k_conv_tail<A>, (channels + 127) / 128, 128, 0, s, (const A*)in, ld_in, channels, taps, tail, T);
}

int causal_conv(const void* in, int ld_in, void* out, int channels, int taps, const float* w, const float* b, float* tail, int T,
                bool act_bf16, cudaStream_t s)
{
    return act_bf16 ? launch_conv<bf16>(in, ld_in, out, channels, taps, w, b, tail, T, s)
                    : launch_conv<float>(in, ld_in, out, channels, taps, w, b, tail, T, s);
}

// ------------------------------------------------------------------ gate and norm

// What multiplies: silu, or (after a norm with a weight) sigmoid of the gate.
template <typename A> __device__ __forceinline__ float gate_value(int form, float g) { return form == kNormWeightGate ? sigmoid_act<A>(g) : silu_act<A>(g); }

// Any sizes: one CTA per (part, token).  Values are kept in registers up to 16 per thread, else computed again.
template <typename A>
__global__ void __launch_bounds__(256) k_gated_norm(const A* o, int ld_o, const A* g, int ld_g, const float* __restrict__ w, A* y,
                                                    int ld_y, int heads, int value_dim, int value_pad, int part, int form, float eps)
{
    __shared__ float s_part[8];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.y, first = blockIdx.x * part, n = blockDim.x;
    if (value_dim != value_pad && blockIdx.x == 0) {       // pad columns meet zero weights, but must be finite
        const int rest = value_pad - value_dim;
        for (int i = threadIdx.x; i < heads * rest; i += n)
            y[(size_t)t * ld_y + i / rest * value_pad + value_dim + i % rest] = act_from<A>(0.0f);
    }
    const A* po = o + (size_t)t * ld_o;
    const A* pg = g + (size_t)t * ld_g;
    auto where = [&](int i) -> int {       // channel of the unpadded heads -> stored place
        const int c = first + i;
        return value_dim == value_pad ? c : c / value_dim * value_pad + c % value_dim;
    };
    constexpr int kKeep = 16;
    float keep[kKeep], gate[kKeep];
    float sum = 0.0f;
    const bool fits = part <= kKeep * n;
    if (fits) {
#pragma unroll
        for (int j = 0; j < kKeep; j++) {
            const int i = threadIdx.x + j * n;
            keep[j] = gate[j] = 0.0f;
            if (i < part) {
                const int c = where(i);
                keep[j] = act_load(po + c);
                gate[j] = act_load(pg + c);
            }
        }
#pragma unroll
        for (int j = 0; j < kKeep; j++) {
            gate[j] = gate_value<A>(form, gate[j]);
            if (form == kGateThenNorm) keep[j] *= gate[j];
            sum = fmaf(keep[j], keep[j], sum);
        }
    } else {
        for (int i = threadIdx.x; i < part; i += n) {
            const int c = where(i);
            float v = act_load(po + c);
            if (form == kGateThenNorm) v *= silu_act<A>(act_load(pg + c));
            sum = fmaf(v, v, sum);
        }
    }
    sum = warp_sum(sum);
    if ((threadIdx.x & 31) == 0) s_part[threadIdx.x >> 5] = sum;
    __syncthreads();
    float tot = 0.0f;
    for (int i = 0; i < n / 32; i++) tot += s_part[i];
    const float scale = 1.0f / sqrtf(tot / (float)part + eps);
    A* py = y + (size_t)t * ld_y;
    if (fits) {
#pragma unroll
        for (int j = 0; j < kKeep; j++) {
            const int i = threadIdx.x + j * n;
            if (i < part) {
                const int c = where(i);
                py[c] = act_from<A>(keep[j] * scale * (form != kNormThenGate ? w[c] : 1.0f) * (form != kGateThenNorm ? gate[j] : 1.0f));
            }
        }
    } else {
        for (int i = threadIdx.x; i < part; i += n) {
            const int c = where(i);
            const float v = act_load(po + c), z = gate_value<A>(form, act_load(pg + c));
            py[c] = act_from<A>(v * z * scale * (form != kNormThenGate ? w[c] : 1.0f));
        }
    }
}

// Unpadded heads, parts of whole groups of four: W warps per (part, token), four channels per lane and load, at most NJ
// loads per lane.
template <typename A, int W, int NJ>
__global__ void __launch_bounds__(256) k_gated_norm_vec(const A* o, int ld_o, const A* g, int ld_g, const float* __restrict__ w, A* y, int ld_y,
                                                        int part, int parts, int T, int form, float eps)
{
    __shared__ float s_part[8];
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long unit = (long)blockIdx.x * (8 / W) + warp / W;
    const int t = (int)(unit / parts), first = (int)(unit - (long)t * parts) * part;
    const bool live = t < T;
    const int at = 4 * (lane + 32 * (warp % W)), step = 128 * W;
    pdl_wait();
    float4 v[NJ], z[NJ];
#pragma unroll
    for (int j = 0; j < NJ; j++) {
        const int i = at + step * j;
        const bool in = live && i < part;
        v[j] = in ? act_load4(o + (size_t)t * ld_o + first + i) : make_float4(0, 0, 0, 0);
        z[j] = in ? act_load4(g + (size_t)t * ld_g + first + i) : make_float4(0, 0, 0, 0);
    }
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; j++) {
        z[j] = make_float4(gate_value<A>(form, z[j].x), gate_value<A>(form, z[j].y), gate_value<A>(form, z[j].z), gate_value<A>(form, z[j].w));
        if (form == kGateThenNorm) v[j] = make_float4(v[j].x * z[j].x, v[j].y * z[j].y, v[j].z * z[j].z, v[j].w * z[j].w);
        sum = fmaf(v[j].x, v[j].x, sum); sum = fmaf(v[j].y, v[j].y, sum); sum = fmaf(v[j].z, v[j].z, sum); sum = fmaf(v[j].w, v[j].w, sum);
    }
    sum = warp_sum(sum);
    if (W > 1) {
        if (lane == 0) s_part[warp] = sum;
        __syncthreads();
        sum = 0.0f;
#pragma unroll
        for (int i = 0; i < W; i++) sum += s_part[warp / W * W + i];
    }
    const float scale = 1.0f / sqrtf(sum / (float)part + eps);
#pragma unroll
    for (int j = 0; j < NJ; j++) {
        const int i = at + step * j;
        if (live && i < part) {
            float4 f = z[j];
            if (form != kNormThenGate) {
                f = *reinterpret_cast<const float4*>(w + first + i);
                if (form == kNormWeightGate) f = make_float4(f.x * z[j].x, f.y * z[j].y, f.z * z[j].z, f.w * z[j].w);
            }
            act_store4(y + (size_t)t * ld_y + first + i, make_float4(v[j].x * scale * f.x, v[j].y * scale * f.y, v[j].z * scale * f.z, v[j].w * scale * f.w));
        }
    }
}

template <typename A>
static int launch_gated_norm(const A* o, int ld_o, const A* g, int ld_g, const float* w, A* y, int ld_y, int heads, int value_dim, int value_pad,
                             int parts, int form, float eps, int T, cudaStream_t s)
{
    const int part = heads * value_dim / parts;
    const bool vec = value_dim == value_pad && part % 4 == 0 && ld_o % 4 == 0 && ld_g % 4 == 0 && ld_y % 4 == 0;
    const long units = (long)T * parts;
    const unsigned packed = (unsigned)((units + 7) / 8), single = (unsigned)units;
    // a single token has few parts: spread one over the CTA's warps
    const bool few = units <= 64;
    if (vec && !few && part <= 256)
        return launch_ordered(k_gated_norm_vec<A, 1, 2>, packed, 256, 0, s, o, ld_o, g, ld_g, w, y, ld_y, part, parts, T, form, eps);
    if (vec && !few && part <= 1024)
        return launch_ordered(k_gated_norm_vec<A, 1, 8>, packed, 256, 0, s, o, ld_o, g, ld_g, w, y, ld_y, part, parts, T, form, eps);
    if (vec && part <= 2048)
        return launch_ordered(k_gated_norm_vec<A, 8, 2>, single, 256, 0, s, o, ld_o, g, ld_g, w, y, ld_y, part, parts, T, form, eps);
    if (vec && part <= 8192)
        return launch_ordered(k_gated_norm_vec<A, 8, 8>, single, 256, 0, s, o, ld_o, g, ld_g, w, y, ld_y, part, parts, T, form, eps);
    int threads = (part / 4 + 31) / 32 * 32;
    threads = threads < 32 ? 32 : threads > 256 ? 256 : threads;
    return launch_ordered(k_gated_norm<A>, dim3(parts, T), threads, 0, s, o, ld_o, g, ld_g, w, y, ld_y, heads, value_dim, value_pad, part, form, eps);
}

int gated_norm(const void* o, int ld_o, const void* g, int ld_g, const float* w, void* y, int ld_y, int heads, int value_dim,
               int value_pad, int parts, int form, float eps, int T, bool act_bf16, cudaStream_t s)
{
    if (parts < 1 || heads * value_dim % parts || form < 0 || form > 2 || (form != kNormThenGate && !w)) return latch(BPDQ_ERR_ARG);
    if (act_bf16)
        return launch_gated_norm((const bf16*)o, ld_o, (const bf16*)g, ld_g, w, (bf16*)y, ld_y, heads, value_dim, value_pad, parts, form, eps, T, s);
    return launch_gated_norm((const float*)o, ld_o, (const float*)g, ld_g, w, (float*)y, ld_y, heads, value_dim, value_pad, parts, form, eps, T, s);
}

}  // namespace bpdq

using namespace bpdq;

extern "C" {

int bpd_decayed_scan_cuda(const void* q, int ld_q, const void* k, int ld_k, const void* v, int ld_v, const float* decay, const float* log_decay,
                          const float* dt, const float* neg_exp_a, const float* d_skip, float* state, void* o, int ld_o, int n_tokens, int heads,
                          int groups, int key_pad, int value_pad, int act_bf16, void* stream)
{
    if (n_tokens < 0 || heads < 1 || groups < 1 || key_pad < 16 || value_pad < 16) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!q || !k || !v || !state || !o || (dt ? !neg_exp_a : (!decay || !log_decay))) return latch(BPDQ_ERR_ARG);
    if ((ld_q | ld_k | ld_v | ld_o) % 8) return latch(BPDQ_ERR_ALIGN);
    DecayedScan a = {};
    a.q = q; a.k = k; a.v = v;
    a.ld_q = ld_q; a.ld_k = ld_k; a.ld_v = ld_v;
    a.heads = heads; a.groups = groups; a.key_pad = key_pad; a.value_pad = value_pad;
    a.decay = decay; a.log_decay = log_decay;
    a.dt = dt; a.neg_exp_a = neg_exp_a; a.ld_dt = heads;
    a.d_skip = d_skip;
    a.state = state;
    a.o = o; a.ld_o = ld_o;
    return decayed_scan(a, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

int bpd_rotate_half_qk_cuda(void* q, void* k, int ld, int n_tokens, int heads, int dim_pad, int rot_dims, const float* rot_freq, float k_scale,
                            const int32_t* pos, int act_bf16, void* stream)
{
    if (n_tokens < 0 || heads < 1 || dim_pad < 1 || rot_dims < 0 || rot_dims % 2 || rot_dims > dim_pad) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!q || !k || !pos || (rot_dims && !rot_freq)) return latch(BPDQ_ERR_ARG);
    return rotate_half_qk(q, k, ld, heads, dim_pad, rot_dims, rot_freq, k_scale, pos, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

int bpd_causal_conv_silu_cuda(const void* in, int ld_in, void* out, int n_tokens, int channels, int taps, const float* w, const float* b, float* tail,
                              int act_bf16, void* stream)
{
    if (n_tokens < 0 || channels < 1 || taps < 1) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!in || !out || !w || (taps > 1 && !tail)) return latch(BPDQ_ERR_ARG);
    return causal_conv(in, ld_in, out, channels, taps, w, b, tail, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

int bpd_gated_norm_cuda(const void* o, int ld_o, const void* g, int ld_g, const float* w, void* y, int ld_y, int n_tokens, int heads, int value_dim,
                        int value_pad, int parts, int form, float eps, int act_bf16, void* stream)
{
    if (n_tokens < 0 || heads < 1 || value_dim < 1 || value_pad < value_dim) return latch(BPDQ_ERR_ARG);
    if (n_tokens == 0) return 0;
    if (!o || !g || !y) return latch(BPDQ_ERR_ARG);
    return gated_norm(o, ld_o, g, ld_g, w, y, ld_y, heads, value_dim, value_pad, parts, form, eps, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

}  // extern "C"
