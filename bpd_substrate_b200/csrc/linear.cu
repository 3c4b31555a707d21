// Matrix products of the hybrid decoders: bf16 weights [N][K], activations bf16 or fp32, fp32 accumulation, and
// everything elementwise that follows a product as its epilogue (residual add between two dynamic-tanh norms, residual
// streams, SwiGLU of paired rows, GELU, step sizes, decays and the one-token convolution of a recurrent layer).  The
// dynamic-tanh norm needs no row statistics; an RMS norm ahead of a one-token product is taken into the product, whose
// CTAs all read the whole row anyway (the row enters times the norm's weight, the root mean square divides the sums).
//
//   k_linear_vec   one token: a warp streams two weight rows at a time with 16-byte loads, the first of them before the
//                  launch ahead has finished (weights are constant); HBM bound
//   k_linear_tc5   several tokens, bf16: tcgen05.mma kind::f16, 128 weight rows (TMEM lanes) x up to 256 tokens
//                  (TMEM columns) per tile, persistent CTAs, operands by tiled TMA into a 128-byte-swizzled ring, two
//                  accumulators so that a tile's epilogue runs under the next tile's products
//   k_linear_tile  several tokens, fp32: plain fp32 multiply-adds on 64 x 64 tiles
#include "decoder_device.cuh"
#include "launch.cuh"
#include "tcgen05_device.cuh"
#include "../../include/bpdq.h"

namespace bpdq {

// ------------------------------------------------------------------ one token

template <typename A>
__global__ void __launch_bounds__(256, 2) k_linear_vec(Linear l)
{
    extern __shared__ float4 xs[];      // [2][K / 8]: first and second four of every eight activations (split: twice)
    __shared__ float s_sum[8];
    constexpr int kBatch = 8;           // 16-byte loads in flight per row and lane
    const int units = l.K / 8, pairs = (l.N + 1) / 2;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int stride = gridDim.x * 8;
    int p = blockIdx.x + gridDim.x * warp;      // row pairs are dealt over the CTAs first: every SM gets its share
    pdl_launch_dependents();
    uint4 w[2][kBatch];
    auto fetch = [&](int base) {
        const int r1 = 2 * p + 1 < l.N ? 2 * p + 1 : 2 * p;
        const uint4* a = reinterpret_cast<const uint4*>(l.W + (size_t)(2 * p) * l.K);
        const uint4* b = reinterpret_cast<const uint4*>(l.W + (size_t)r1 * l.K);
#pragma unroll
        for (int i = 0; i < kBatch; i++) {
            const int u = base + lane + 32 * i;
            w[0][i] = u < units ? __ldg(a + u) : make_uint4(0, 0, 0, 0);
            w[1][i] = u < units ? __ldg(b + u) : make_uint4(0, 0, 0, 0);
        }
    };
    if (p < pairs) fetch(0);
    pdl_wait();
    float rnorm = 1.0f;
    if (l.norm_w) {
        const float* in = reinterpret_cast<const float*>(l.in);
        float sum = 0.0f;
        for (int j = threadIdx.x; j < 2 * units; j += 256) {
            float4 v = act_load4(in + 4 * j);
            const float4 w4 = act_load4(l.norm_w + 4 * j);
            sum = fmaf(v.x, v.x, sum); sum = fmaf(v.y, v.y, sum); sum = fmaf(v.z, v.z, sum); sum = fmaf(v.w, v.w, sum);
            xs[(j & 1) * units + (j >> 1)] = make_float4(v.x * w4.x, v.y * w4.y, v.z * w4.z, v.w * w4.w);
        }
        sum = warp_sum(sum);
        if (lane == 0) s_sum[warp] = sum;
        __syncthreads();
        sum = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) sum += s_sum[i];
        rnorm = 1.0f / sqrtf(sum / (float)l.norm_n + l.norm_eps);
    } else {
        const A* in = reinterpret_cast<const A*>(l.in);
        for (int j = threadIdx.x; j < 2 * units; j += 256) xs[(j & 1) * units + (j >> 1)] = act_load4(in + 4 * j);
        if (l.split)
            for (int j = threadIdx.x; j < 2 * units; j += 256) xs[(2 + (j & 1)) * units + (j >> 1)] = act_load4(in + l.in2 + 4 * j);
        __syncthreads();
    }
    bool have = true;
    for (; p < pairs; p += stride) {
        const int row = 2 * p + lane;
        const float4* x = l.split && 2 * p >= l.split ? xs + 2 * units : xs;
        const bool residual = l.mode == kLinResidual && lane < 2 && row < l.N;
        const bool streams = l.mode == kLinStreams && lane < 2 && row < l.N;
        float xo[kMaxStreams];
        if (streams) {
#pragma unroll
            for (int i = 0; i < kMaxStreams; i++) xo[i] = i < l.streams.n ? l.x[(size_t)i * l.ld_x + row] : 0.0f;
        }
        float xr = 0, pw = 0, pb = 0, nw = 0, nb = 0;       // what the residual epilogue of row 2 p + lane needs, ahead of its use
        if (residual) {
            xr = l.x[row];
            pw = l.post.w[row];
            pb = l.post.b[row];
            if (l.next.w) { nw = l.next.w[row]; nb = l.next.b[row]; }
        }
        float acc[2] = {0.0f, 0.0f};
        for (int base = 0; base < units; base += 32 * kBatch) {
            if (!have) fetch(base);
            have = false;
#pragma unroll
            for (int i = 0; i < kBatch; i++) {
                const int u = base + lane + 32 * i;
                if (u >= units) break;
                const float4 x0 = x[u], x1 = x[units + u];
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const uint4 q = w[r][i];
                    acc[r] = fmaf(__uint_as_float(q.x << 16), x0.x, acc[r]);
                    acc[r] = fmaf(__uint_as_float(q.x & 0xFFFF0000u), x0.y, acc[r]);
                    acc[r] = fmaf(__uint_as_float(q.y << 16), x0.z, acc[r]);
                    acc[r] = fmaf(__uint_as_float(q.y & 0xFFFF0000u), x0.w, acc[r]);
                    acc[r] = fmaf(__uint_as_float(q.z << 16), x1.x, acc[r]);
                    acc[r] = fmaf(__uint_as_float(q.z & 0xFFFF0000u), x1.y, acc[r]);
                    acc[r] = fmaf(__uint_as_float(q.w << 16), x1.z, acc[r]);
                    acc[r] = fmaf(__uint_as_float(q.w & 0xFFFF0000u), x1.w, acc[r]);
                }
            }
        }
        acc[0] = warp_sum(acc[0]);
        acc[1] = warp_sum(acc[1]);
        const float v = (lane ? acc[1] : acc[0]) * rnorm;
        if (l.mode == kLinSwiglu) {
            if (lane == 0) reinterpret_cast<A*>(l.out)[p] = act_from<A>(silu_act<A>(acc[0] * rnorm) * (acc[1] * rnorm));
        } else if (streams) {
            float u = 0.0f;
#pragma unroll
            for (int i = 0; i < kMaxStreams; i++) {
                if (i >= l.streams.n) break;
                float r = l.streams.out[i] * v;
#pragma unroll
                for (int j = 0; j < kMaxStreams; j++)
                    if (j < l.streams.n) r = fmaf(l.streams.mix[j][i], xo[j], r);
                l.x[(size_t)i * l.ld_x + row] = r;
                u = fmaf(l.streams.next[i], r, u);
            }
            l.u[row] = u;
        } else if (residual) {
            const float r = xr + fmaf(tanhf(l.post.alpha * v), pw, pb);
            l.x[row] = r;
            if (l.next.w) reinterpret_cast<A*>(l.out)[row] = act_from<A>(fmaf(tanhf(l.next.alpha * r), nw, nb));
        } else if (l.mode != kLinResidual && l.mode != kLinStreams && lane < 2 && row < l.N) {
            linear_store<A>(l, 0, row, v);
        }
    }
}

// ------------------------------------------------------------------ several tokens, fp32

__global__ void __launch_bounds__(256) k_linear_tile(Linear l, int T)
{
    __shared__ float sw[16][68], sx[16][68];
    const int tid = threadIdx.x, tr = tid & 15, tt = tid >> 4;      // rows 4 tr .., tokens 4 tt ..
    const int n0 = blockIdx.x * 64, t0 = blockIdx.y * 64;
    pdl_launch_dependents();
    pdl_wait();
    const float* in = reinterpret_cast<const float*>(l.in);
    float acc[4][4] = {};
    const int row = tid >> 2, kq = (tid & 3) * 4;
    for (int k0 = 0; k0 < l.K; k0 += 16) {
        float4 a = make_float4(0, 0, 0, 0), b = a;
        if (n0 + row < l.N) a = act_load4(l.W + (size_t)(n0 + row) * l.K + k0 + kq);
        if (t0 + row < T) b = act_load4(in + (size_t)(t0 + row) * l.ld_in + k0 + kq);
        sw[kq][row] = a.x; sw[kq + 1][row] = a.y; sw[kq + 2][row] = a.z; sw[kq + 3][row] = a.w;
        sx[kq][row] = b.x; sx[kq + 1][row] = b.y; sx[kq + 2][row] = b.z; sx[kq + 3][row] = b.w;
        __syncthreads();
        float part[4][4] = {};      // a block's sum on its own: long sums then lose less
#pragma unroll
        for (int k = 0; k < 16; k++) {
            const float4 wv = *reinterpret_cast<const float4*>(&sw[k][4 * tr]);
            const float4 xv = *reinterpret_cast<const float4*>(&sx[k][4 * tt]);
            const float wr[4] = {wv.x, wv.y, wv.z, wv.w}, xr[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
            for (int j = 0; j < 4; j++)
#pragma unroll
                for (int i = 0; i < 4; i++) part[j][i] = fmaf(wr[i], xr[j], part[j][i]);
        }
#pragma unroll
        for (int j = 0; j < 4; j++)
#pragma unroll
            for (int i = 0; i < 4; i++) acc[j][i] += part[j][i];
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; j++) {
        const int t = t0 + 4 * tt + j;
        if (t >= T) break;
        if (l.mode == kLinSwiglu) {
#pragma unroll
            for (int i = 0; i < 4; i += 2) {
                const int n = n0 + 4 * tr + i;
                if (n < l.N) reinterpret_cast<float*>(l.out)[(size_t)t * l.ld_out + n / 2] = silu_act<float>(acc[j][i]) * acc[j][i + 1];
            }
        } else {
#pragma unroll
            for (int i = 0; i < 4; i++)
                if (n0 + 4 * tr + i < l.N) linear_store<float>(l, t, n0 + 4 * tr + i, acc[j][i]);
        }
    }
}

// ------------------------------------------------------------------ several tokens, bf16, tensor cores

template <int BN>
struct Tc5Linear {
    static constexpr int kRows = 128, kDepth = 64;                     // weight rows per tile, K elements per ring stage
    static constexpr int kABytes = kRows * kDepth * 2, kBBytes = BN * kDepth * 2;
    static constexpr int kStageBytes = kABytes + kBBytes;              // a multiple of 1024: the swizzle's atom
    static constexpr int kStages = BN == 256 ? 4 : BN == 128 ? 6 : 8;
    static constexpr int kEpiWarps = 8;                                // two per TMEM lane quarter, each half of the columns
    static constexpr int kThreads = 32 * (2 + kEpiWarps);
    static constexpr int kTmemCols = 2 * BN;
    static constexpr size_t kSmem = 1024 + (size_t)kStages * kStageBytes + 8 * (2 * kStages + 4) + 16;
};

// K-major operand in the 128-byte swizzle: 8-row groups 1024 bytes apart.
__device__ __forceinline__ uint64_t swizzled_desc(uint32_t saddr)
{
    return (uint64_t)((saddr >> 4) & 0x3FFFu) | (1ull << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void umma_bf16_ss(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accum)
{
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accum)
        : "memory");
}

template <int BN>
__global__ void __launch_bounds__(Tc5Linear<BN>::kThreads, 1)
k_linear_tc5(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap, Linear l, int T, int* err)
{
    using S = Tc5Linear<BN>;
    constexpr int kStages = S::kStages;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* ring = reinterpret_cast<uint8_t*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(ring + (size_t)kStages * S::kStageBytes);
    uint64_t* empty = full + kStages;
    uint64_t* acc_full = empty + kStages;      // [2]
    uint64_t* acc_empty = acc_full + 2;        // [2]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (tid == 0) {
        for (int s = 0; s < kStages; s++) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int s = 0; s < 2; s++) { mbar_init(&acc_full[s], 1); mbar_init(&acc_empty[s], S::kEpiWarps); }
        mbar_init_fence();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(tmem_slot)), "r"(S::kTmemCols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;
    pdl_launch_dependents();

    const int n_tiles = (l.N + S::kRows - 1) / S::kRows, t_tiles = (T + BN - 1) / BN;
    // tokens vary fastest: the CTAs at work share few rows of weights, which go through HBM once
    const int tiles = n_tiles * t_tiles, kb_n = (l.K + S::kDepth - 1) / S::kDepth;

    if (warp == 0) {
        // ---------------- producer: the weights of the first ring round are requested before the launch ahead has finished
        if (lane == 0) {
            const int mine = blockIdx.x < tiles ? (tiles - blockIdx.x + gridDim.x - 1) / gridDim.x : 0;
            const long steps = (long)mine * kb_n;
            auto weights = [&](long i, int s) {
                const int tile = blockIdx.x + (int)(i / kb_n) * gridDim.x, kb = (int)(i % kb_n);
                mbar_expect_tx(&full[s], S::kStageBytes);
                tma_rows_2d(ring + (size_t)s * S::kStageBytes, &wmap, kb * S::kDepth, (tile / t_tiles) * S::kRows, &full[s]);
            };
            auto tokens = [&](long i, int s) {
                const int tile = blockIdx.x + (int)(i / kb_n) * gridDim.x, kb = (int)(i % kb_n);
                tma_rows_2d(ring + (size_t)s * S::kStageBytes + S::kABytes, &xmap, kb * S::kDepth, (tile % t_tiles) * BN, &full[s]);
            };
            const long ahead = steps < kStages ? steps : kStages;
            for (long i = 0; i < ahead; i++) weights(i, (int)i);
            pdl_wait();
            for (long i = 0; i < ahead; i++) tokens(i, (int)i);
            int s = 0;
            uint32_t par = 0;
            for (long i = ahead; i < steps; i++) {
                if (!mbar_wait_bounded(&empty[s], par, err, 41)) break;
                weights(i, s);
                tokens(i, s);
                if (++s == kStages) { s = 0; par ^= 1u; }
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer
        constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(S::kRows >> 4) << 24);
        int s = 0, local = 0;
        uint32_t full_par = 0;
        bool ok = true;
        for (int tile = blockIdx.x; ok && tile < tiles; tile += gridDim.x, local++) {
            const int a = local & 1;
            if (local >= 2 && !mbar_wait_bounded(&acc_empty[a], (uint32_t)((local >> 1) - 1) & 1u, err, 42)) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int kb = 0; kb < kb_n; kb++) {
                if (!mbar_wait_bounded(&full[s], full_par, err, 43)) { ok = false; break; }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t stage = smem_addr(ring + (size_t)s * S::kStageBytes);
                const uint64_t ad = swizzled_desc(stage), bd = swizzled_desc(stage + S::kABytes);
                const int left = (l.K - kb * S::kDepth) / 16, k_n = left < 4 ? left : 4;
                if (elect_one()) {
                    for (int k = 0; k < k_n; k++)
                        umma_bf16_ss(tmem_base + (uint32_t)(a * BN), ad + 2 * k, bd + 2 * k, idesc, (kb | k) ? 1u : 0u);
                    umma_commit(&empty[s]);
                    if (kb + 1 == kb_n) umma_commit(&acc_full[a]);
                }
                __syncwarp();
                if (++s == kStages) { s = 0; full_par ^= 1u; }
            }
        }
    } else {
        // ---------------- epilogue: a thread owns one weight row of the tile and walks over its tokens
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        constexpr int kCols = BN / 2;
        const int r = 32 * quarter + lane;
        int local = 0;
        pdl_wait();
        for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, local++) {
            const int a = local & 1;
            if (!mbar_wait_bounded(&acc_full[a], (uint32_t)(local >> 1) & 1u, err, 44)) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int n = (tile / t_tiles) * S::kRows + r;
            const int tb = (tile % t_tiles) * BN + half * kCols;
            const bool live = n < l.N;
            const uint32_t ta = tmem_base + ((uint32_t)(32 * quarter) << 16) + (uint32_t)(a * BN + half * kCols);
            DynTanh post = l.post, next = l.next;
            float pw = 0, pb = 0, nw = 0, nb = 0;
            if (l.mode == kLinResidual && live) {
                pw = post.w[n]; pb = post.b[n];
                if (next.w) { nw = next.w[n]; nb = next.b[n]; }
            } else if (l.mode == kLinLogDecay && live) {
                pw = l.neg_exp_a[n]; pb = l.dt_bias[n];
            }
            const bool is_step = l.mode == kLinMixerIn && live && n >= l.dt_row;      // (lanes of one warp may differ)
            if (is_step && l.dt_bias) pb = l.dt_bias[n - l.dt_row];
            const bool plain_f32 = l.mode == kLinF32 && l.cap == 0.0f;
            // rows of this warp that are only rounded and stored (after a GELU)
            const int n_end = (n - lane) + 32;
            const bool plain_warp = !((l.N | l.ld_out) & 1) &&
                                    (l.mode == kLinAct || l.mode == kLinGelu || (l.mode == kLinMixerIn && n_end <= l.dt_row && !l.conv.w));
            for (int c0 = 0; c0 < kCols; c0 += 16) {
                int v[16];
                tmem_ld(ta + c0, v);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                const int t0 = tb + c0;
                if (t0 >= T) continue;
                if (l.mode == kLinResidual) {
                    float xv[16];
#pragma unroll
                    for (int j = 0; j < 16; j++) xv[j] = (live && t0 + j < T) ? l.x[(size_t)(t0 + j) * l.ld_x + n] : 0.0f;
#pragma unroll
                    for (int j = 0; j < 16; j++) {
                        const float q = xv[j] + fmaf(tanhf(post.alpha * __int_as_float(v[j])), pw, pb);
                        if (live && t0 + j < T) {
                            l.x[(size_t)(t0 + j) * l.ld_x + n] = q;
                            if (next.w)
                                reinterpret_cast<bf16*>(l.out)[(size_t)(t0 + j) * l.ld_out + n] =
                                    act_from<bf16>(fmaf(tanhf(next.alpha * q), nw, nb));
                        }
                    }
                } else if (l.mode == kLinSwiglu) {
                    // lane pairs hold gate (even) and up (odd): the even lane finishes even tokens, the odd lane odd ones
#pragma unroll
                    for (int j = 0; j < 16; j += 2) {
                        const float keep = __int_as_float((lane & 1) ? v[j + 1] : v[j]);
                        const float other = __shfl_xor_sync(0xFFFFFFFFu, __int_as_float((lane & 1) ? v[j] : v[j + 1]), 1);
                        const float g = (lane & 1) ? other : keep, u = (lane & 1) ? keep : other;
                        const int t = t0 + j + (lane & 1);
                        if (live && t < T) reinterpret_cast<bf16*>(l.out)[(size_t)t * l.ld_out + n / 2] = act_from<bf16>(silu_act<bf16>(g) * u);
                    }
                } else if (plain_warp) {
                    if (l.mode == kLinGelu)
#pragma unroll
                        for (int j = 0; j < 16; j++) v[j] = __float_as_int(gelu_act<bf16>(__int_as_float(v[j])));
                    // two neighbouring rows per store: the even lane finishes even tokens, the odd lane odd ones
#pragma unroll
                    for (int j = 0; j < 16; j += 2) {
                        const float keep = __int_as_float((lane & 1) ? v[j + 1] : v[j]);
                        const float other = __shfl_xor_sync(0xFFFFFFFFu, __int_as_float((lane & 1) ? v[j] : v[j + 1]), 1);
                        const __nv_bfloat162 two = __floats2bfloat162_rn((lane & 1) ? other : keep, (lane & 1) ? keep : other);
                        const int t = t0 + j + (lane & 1);
                        if (live && t < T) *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(l.out) + (size_t)t * l.ld_out + (n & ~1)) = two;
                    }
                } else if (plain_f32) {
#pragma unroll
                    for (int j = 0; j < 16; j++)
                        if (live && t0 + j < T) reinterpret_cast<float*>(l.out)[(size_t)(t0 + j) * l.ld_out + n] = __int_as_float(v[j]);
                } else if (l.mode == kLinLogDecay) {
#pragma unroll
                    for (int j = 0; j < 16; j++)
                        if (live && t0 + j < T) l.dt[(size_t)(t0 + j) * l.ld_dt + n] = pw * softplus_act<bf16>(__int_as_float(v[j]) + pb);
                } else if (is_step) {
                    float q[16];
#pragma unroll
                    for (int j = 0; j < 16; j++) q[j] = l.dt_bias ? softplus_act<bf16>(__int_as_float(v[j]) + pb) : sigmoid_act<bf16>(__int_as_float(v[j]));
#pragma unroll
                    for (int j = 0; j < 16; j++)
                        if (t0 + j < T) l.dt[(size_t)(t0 + j) * l.ld_dt + n - l.dt_row] = q[j];
                } else if (live) {
#pragma unroll
                    for (int j = 0; j < 16; j++)
                        if (t0 + j < T) linear_store<bf16>(l, t0 + j, n, __int_as_float(v[j]));
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[a]);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(S::kTmemCols) : "memory");
    }
}

// ------------------------------------------------------------------ host side

typedef CUresult (*TensorMapEncode)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                    const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                    CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// bf16 matrix [rows][cols] with `ld` elements between rows, read in boxes of box_rows x 64 columns.
static int bf16_map(CUtensorMap* map, const void* p, int rows, int cols, int ld, int box_rows)
{
    static TensorMapEncode encode = nullptr;
    if (!encode) {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult q;
        cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q);
        if (e != cudaSuccess || q != cudaDriverEntryPointSuccess || !fn) return latch(BPDQ_ERR_CUDA);
        encode = (TensorMapEncode)fn;
    }
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {64, (cuuint32_t)box_rows}, estr[2] = {1, 1};
    CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(p), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : latch(BPDQ_ERR_CUDA - 900 - (int)r);
}

template <int BN>
static int launch_tc5(const Linear& l, int T, cudaStream_t s)
{
    using S = Tc5Linear<BN>;
    CUtensorMap wmap, xmap;
    int rc;
    if ((rc = bf16_map(&wmap, l.W, l.N, l.K, l.K, S::kRows))) return rc;
    if ((rc = bf16_map(&xmap, l.in, T, l.K, l.ld_in, BN))) return rc;
    if ((rc = allow_smem<k_linear_tc5<BN>>((int)S::kSmem))) return rc;
    const long tiles = (long)((l.N + S::kRows - 1) / S::kRows) * ((T + BN - 1) / BN);
    const int grid = (int)(tiles < sm_count() ? tiles : sm_count());
    return launch_ordered(k_linear_tc5<BN>, grid, S::kThreads, S::kSmem, s, wmap, xmap, l, T, device_error_flag());
}

int linear_forward(const Linear& l, int T, bool act_bf16, cudaStream_t s)
{
    if (l.K % 16 || l.K < 16 || l.N < 1 || T < 1 || l.ld_in % 8) return latch(BPDQ_ERR_ARG);
    if (T > 1 && (l.norm_w || l.split || l.mode == kLinStreams)) return latch(BPDQ_ERR_ARG);
    if (l.mode == kLinStreams && (l.streams.n < 1 || l.streams.n > kMaxStreams)) return latch(BPDQ_ERR_ARG);
    if (T == 1) {
        const size_t smem = (size_t)l.K * (l.split ? 8 : 4);
        if (smem > 200 * 1024) return latch(BPDQ_ERR_RANGE);
        int rc = act_bf16 ? allow_smem<k_linear_vec<bf16>>(200 * 1024) : allow_smem<k_linear_vec<float>>(200 * 1024);
        if (rc) return rc;
        const int want = (l.N + 1) / 2, cap = 2 * sm_count();
        const int grid = want < cap ? want : cap;
        return act_bf16 ? launch_ordered(k_linear_vec<bf16>, grid, 256, smem, s, l) : launch_ordered(k_linear_vec<float>, grid, 256, smem, s, l);
    }
    if (!act_bf16) return launch_ordered(k_linear_tile, dim3((l.N + 63) / 64, (T + 63) / 64), 256, 0, s, l, T);
    const long n_tiles = (l.N + 127) / 128;
    if (T > 128 && n_tiles * ((T + 255) / 256) >= sm_count()) return launch_tc5<256>(l, T, s);
    if (T > 64) return launch_tc5<128>(l, T, s);
    if (T > 32) return launch_tc5<64>(l, T, s);
    return launch_tc5<32>(l, T, s);
}

}  // namespace bpdq

using namespace bpdq;

extern "C" {

// out[t][n] = sum_k W[n][k] x[t][k]: bf16 weights, bf16 or fp32 activations, fp32 results.  K a multiple of 16.
int bpd_linear_bf16_cuda(const uint16_t* W, const void* x, float* out, int n_tokens, int N, int K, int act_bf16, void* stream)
{
    if (n_tokens < 0 || N < 1 || K < 16 || (n_tokens > 0 && (!W || !x || !out))) return latch(BPDQ_ERR_ARG);
    if (((uintptr_t)W | (uintptr_t)x) & 15) return latch(BPDQ_ERR_ALIGN);
    if (n_tokens == 0) return 0;
    Linear l = {};
    l.W = reinterpret_cast<const bf16*>(W);
    l.in = x;
    l.N = N; l.K = K; l.ld_in = K;
    l.mode = kLinF32;
    l.out = out;
    l.ld_out = N;
    return linear_forward(l, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

// The same product followed by what a decoder's epilogues do to its sums (BPDQ_MAP_*).
int bpd_linear_map_cuda(const uint16_t* W, const void* x, void* out, int n_tokens, int N, int K, int map, const float* bias, const float* rate, float cap,
                        int act_bf16, void* stream)
{
    if (n_tokens < 0 || N < 1 || K < 16 || (n_tokens > 0 && (!W || !x || !out))) return latch(BPDQ_ERR_ARG);
    if (((uintptr_t)W | (uintptr_t)x) & 15) return latch(BPDQ_ERR_ALIGN);
    if (n_tokens == 0) return 0;
    Linear l = {};
    l.W = reinterpret_cast<const bf16*>(W);
    l.in = x;
    l.N = N; l.K = K; l.ld_in = K;
    l.out = out;
    l.ld_out = N;
    l.dt = reinterpret_cast<float*>(out);
    l.ld_dt = N;
    l.dt_bias = bias;
    l.neg_exp_a = rate;
    switch (map) {
    case BPDQ_MAP_GELU: l.mode = kLinGelu; break;
    case BPDQ_MAP_CAP:
        if (!(cap > 0.0f)) return latch(BPDQ_ERR_ARG);
        l.mode = kLinF32;
        l.cap = cap;
        break;
    case BPDQ_MAP_LOG_DECAY:
        if (!bias || !rate) return latch(BPDQ_ERR_ARG);
        l.mode = kLinLogDecay;
        break;
    case BPDQ_MAP_SIGMOID: l.mode = kLinMixerIn; l.dt_bias = nullptr; break;      // (rows from 0 on are write shares)
    default: return latch(BPDQ_ERR_ARG);
    }
    return linear_forward(l, n_tokens, act_bf16 != 0, (cudaStream_t)stream);
}

}  // extern "C"
