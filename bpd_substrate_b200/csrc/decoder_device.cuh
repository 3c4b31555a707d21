// Building blocks shared by the kernels of the hybrid decoders (recurrent and attention layers on bf16 weights):
// activation types, the dynamic-tanh norm, the epilogues of their matrix products, bf16 tensor-core fragments.
//
// Weights are bf16.  Activations are bf16 or fp32 (the template parameter A); the residual stream, norms, scores,
// softmax, decays and recurrent states are fp32 in both cases.  Every inner size is padded to a multiple of 16 with
// zero weights when a model is loaded, so rows are 16-byte aligned and kernels need no ragged inner loops; pad
// columns of activations hold finite values that meet zero weights.
#pragma once
#include "bpdq_common.cuh"

#include <cuda_bf16.h>

namespace bpdq {

typedef __nv_bfloat16 bf16;

// tanh(alpha x) * w + b, element by element (no statistics).  w == null: no norm.
struct DynTanh {
    const float *w, *b;
    float alpha;
};

enum LinearMode {
    kLinAct = 0,        // out[t][n] = A(v)
    kLinF32 = 1,        // out[t][n] = v
    kLinResidual = 2,   // x[t][n] += post(v); out[t][n] = A(next(x[t][n])) when `next` is given
    kLinSwiglu = 3,     // rows come in pairs (2i: gate, 2i + 1: up); out[t][i] = A(silu(gate) * up)
    kLinMixerIn = 4,    // rows >= dt_row are step sizes in fp32: dt[t][n - dt_row] = softplus(v + dt_bias), or sigmoid(v)
                        // without a dt_bias; with conv.w also conv.channels rows from conv_row on pass the causal
                        // convolution (one token only)
    kLinLogDecay = 5,   // dt[t][n] = neg_exp_a[n] softplus(v + dt_bias[n]) in fp32; with split (one token only) the rows
                        // from there on read the input from in + in2 on: out[t][n - split] = A(v)
    kLinGelu = 6,       // out[t][n] = A(gelu(v)), tanh form
    kLinStreams = 7     // one token only: the residual streams of column n take v in, and their sum with the next
                        // sublayer's weights goes to u[n]
};

// Residual streams joined by hyper-connections: x_t <- sum_s mix[s][t] x_s + out[t] y; the next sublayer reads
// sum_t next[t] x_t.
constexpr int kMaxStreams = 8;
struct StreamMix {
    int n;
    float mix[kMaxStreams][kMaxStreams];
    float out[kMaxStreams], next[kMaxStreams];
};

// Depthwise causal convolution of one token: tail [taps - 1][channels] holds the inputs before it, oldest first.
struct ConvStep {
    const float *w, *b;     // w [taps][channels]; w == null: no convolution here; b == null: no bias
    float* tail;
    void* out;              // [channels], activation type
    int taps, channels;
};

struct Linear {
    const bf16* W;          // [N][K]
    const void* in;         // [T][ld_in], activation type
    int N, K, ld_in;
    int mode;
    void* out;
    int ld_out;
    float* x;               // residual stream [T][ld_x]
    int ld_x;
    DynTanh post, next;
    int conv_row, dt_row;
    const float *dt_bias, *neg_exp_a;
    float* dt;              // [T][ld_dt]
    int ld_dt;
    ConvStep conv;
    int split, in2;
    float cap;              // kLinF32: v becomes cap tanh(v / cap); 0: as it is
    const float* norm_w;    // one token only: `in` is fp32 and passes an RMS norm with this weight over norm_n entries
    int norm_n;
    float norm_eps;
    StreamMix streams;      // kLinStreams: of x [streams.n][ld_x]
    float* u;
};

// Runs one product over T tokens (linear.cu); act_bf16: A is bf16, else fp32.
int linear_forward(const Linear& l, int T, bool act_bf16, cudaStream_t s);

#ifdef __CUDACC__

template <typename A> __device__ __forceinline__ float act_load(const A* p);
template <> __device__ __forceinline__ float act_load<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float act_load<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename A> __device__ __forceinline__ A act_from(float v);
template <> __device__ __forceinline__ float act_from<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 act_from<bf16>(float v) { return __float2bfloat16_rn(v); }

template <typename A> __device__ __forceinline__ float act_round(float v);
template <> __device__ __forceinline__ float act_round<float>(float v) { return v; }
template <> __device__ __forceinline__ float act_round<bf16>(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }

// Four consecutive activations (16-byte or 8-byte aligned).
__device__ __forceinline__ float4 act_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 act_load4(const bf16* p)
{
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16),
                       __uint_as_float(u.y & 0xFFFF0000u));
}

__device__ __forceinline__ void act_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void act_store4(bf16* p, float4 v)
{
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

__device__ __forceinline__ float ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f32(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

// Of results that are rounded to A: with bf16 activations a few units in the last place of fp32 do not matter.
template <typename A> __device__ __forceinline__ float sigmoid_act(float z)
{
    if (sizeof(A) == 4) return sigmoid_f32(z);
    return __fdividef(1.0f, 1.0f + ex2(-1.44269504088896341f * z));
}
template <typename A> __device__ __forceinline__ float silu_act(float z)
{
    if (sizeof(A) == 4) return z / (1.0f + expf(-z));
    return z * sigmoid_act<A>(z);
}
template <typename A> __device__ __forceinline__ float gelu_act(float z)
{
    // 0.5 (1 + tanh(a)) = sigmoid(2 a)
    return z * sigmoid_act<A>(1.59576912160573071f * fmaf(0.044715f * z * z, z, z));
}
// log(1 + e^z) = max(z, 0) + log(1 + e), e = e^-|z| <= 1; with fp32 activations by CUDA's functions, else by
// log(1 + e) = 2 artanh(t), t = e / (2 + e) <= 1/3, whose Taylor series keeps the relative accuracy of small values.
template <typename A> __device__ __forceinline__ float softplus_act(float z)
{
    if (sizeof(A) == 4) return softplus_f32(z);
    const float e = ex2(-1.44269504088896341f * fabsf(z)), t = __fdividef(e, 2.0f + e), s = t * t;
    float p = fmaf(s, 1.0f / 15, 1.0f / 13);
    p = fmaf(s, p, 1.0f / 11);
    p = fmaf(s, p, 1.0f / 9);
    p = fmaf(s, p, 1.0f / 7);
    p = fmaf(s, p, 1.0f / 5);
    p = fmaf(s, p, 1.0f / 3);
    return fmaxf(z, 0.0f) + 2.0f * fmaf(t * s, p, t);
}
__device__ __forceinline__ float dyn_tanh(const DynTanh& p, int n, float v) { return fmaf(tanhf(p.alpha * v), p.w[n], p.b[n]); }

// Everything but the pairwise mode: row n, token t.
template <typename A>
__device__ __forceinline__ void linear_store(const Linear& l, int t, int n, float v)
{
    switch (l.mode) {
    case kLinF32: reinterpret_cast<float*>(l.out)[(size_t)t * l.ld_out + n] = l.cap > 0.0f ? l.cap * tanhf(v / l.cap) : v; break;
    case kLinGelu: reinterpret_cast<A*>(l.out)[(size_t)t * l.ld_out + n] = act_from<A>(gelu_act<A>(v)); break;
    case kLinLogDecay:
        if (l.split && n >= l.split) reinterpret_cast<A*>(l.out)[(size_t)t * l.ld_out + n - l.split] = act_from<A>(v);
        else l.dt[(size_t)t * l.ld_dt + n] = l.neg_exp_a[n] * softplus_act<A>(v + l.dt_bias[n]);
        break;
    case kLinResidual: {
        float* px = l.x + (size_t)t * l.ld_x + n;
        const float r = *px + dyn_tanh(l.post, n, v);
        *px = r;
        if (l.next.w) reinterpret_cast<A*>(l.out)[(size_t)t * l.ld_out + n] = act_from<A>(dyn_tanh(l.next, n, r));
        break;
    }
    case kLinMixerIn:
        if (n >= l.dt_row) {
            l.dt[(size_t)t * l.ld_dt + n - l.dt_row] = l.dt_bias ? softplus_f32(v + l.dt_bias[n - l.dt_row]) : sigmoid_f32(v);
            break;
        }
        if (l.conv.w && n >= l.conv_row && n - l.conv_row < l.conv.channels) {
            const int c = n - l.conv_row, C = l.conv.channels;
            float acc = l.conv.b ? l.conv.b[c] : 0.0f;
            for (int j = 0; j + 1 < l.conv.taps; j++) {
                const float u = l.conv.tail[(size_t)j * C + c];
                acc = fmaf(l.conv.w[(size_t)j * C + c], u, acc);
                if (j > 0) l.conv.tail[(size_t)(j - 1) * C + c] = u;
            }
            // the window holds activations: in bf16 runs the newest input is rounded as a prompt's projection is
            const float u = act_round<A>(v);
            const int last = l.conv.taps - 1;
            acc = fmaf(l.conv.w[(size_t)last * C + c], u, acc);
            if (last > 0) l.conv.tail[(size_t)(last - 1) * C + c] = u;
            reinterpret_cast<A*>(l.conv.out)[c] = act_from<A>(silu_act<A>(acc));
            break;
        }
        reinterpret_cast<A*>(l.out)[(size_t)t * l.ld_out + n] = act_from<A>(v);
        break;
    default: reinterpret_cast<A*>(l.out)[(size_t)t * l.ld_out + n] = act_from<A>(v);
    }
}

#endif
}  // namespace bpdq
