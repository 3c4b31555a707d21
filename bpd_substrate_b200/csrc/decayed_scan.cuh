// Linear attention with a decaying state (retention, state-space duality): one interface for both.
#pragma once
#include "decoder_device.cuh"

namespace bpdq {

// Per head h and token t:  S <- decay S + (dt k) v^T,  o = S^T q + d_skip v.
// S is [key_pad][value_pad] fp32 per head, one state for the sequence; q and k are shared by heads / groups heads.
// decay = decay_h (constant per head) or exp(neg_exp_a_h dt) with a step size dt per token and head.
struct DecayedScan {
    const void *q, *k, *v;              // activation type, [T][ld]
    int ld_q, ld_k, ld_v;
    int heads, groups, key_pad, value_pad;
    const float *decay, *log_decay;     // [heads], or null
    const float *dt, *neg_exp_a;        // [T][ld_dt] and [heads], or null
    int ld_dt;
    const float* d_skip;                // [heads] or null
    // one-token calls can rotate q and k here: rotate-half pairs, then k times k_scale (rot_freq null: as they are)
    const float* rot_freq;
    const int* pos;                     // device: position of token 0
    int rot_dims;
    float k_scale;
    float* state;
    void* o;                            // activation type, [T][ld_o]
    int ld_o;
};
int decayed_scan(const DecayedScan& a, int T, bool act_bf16, cudaStream_t s);

// Rotate-half rotary positions on q and k in place (`heads` heads of `dim_pad`, token t at *pos + t), k then times
// k_scale.
int rotate_half_qk(void* q, void* k, int ld, int heads, int dim_pad, int rot_dims, const float* rot_freq, float k_scale,
                   const int* pos, int T, bool act_bf16, cudaStream_t s);

// Causal depthwise convolution with bias (b null: none) and silu over T tokens: in [T][ld_in] -> out [T][channels]; tail
// [taps - 1][channels] (oldest first) is the window before the first token and is moved on to the last one.
int causal_conv(const void* in, int ld_in, void* out, int channels, int taps, const float* w, const float* b, float* tail, int T,
                bool act_bf16, cudaStream_t s);

// Gate and RMS norm over `parts` equal parts of the heads' outputs (heads of value_dim stored value_pad apart):
// in one of three forms; w has an entry per stored channel.
enum GatedNormForm {
    kNormThenGate = 0,      // y = o / rms(o) * silu(g)
    kGateThenNorm = 1,      // u = o * silu(g), y = u / rms(u) * w
    kNormWeightGate = 2     // y = o / rms(o) * w * sigmoid(g)
};
int gated_norm(const void* o, int ld_o, const void* g, int ld_g, const float* w, void* y, int ld_y, int heads, int value_dim,
               int value_pad, int parts, int form, float eps, int T, bool act_bf16, cudaStream_t s);

}  // namespace bpdq
