// Gated delta rule with a decay per key channel: linear attention whose write is the error of what the state predicts.
#pragma once
#include "decoder_device.cuh"

namespace bpdq {

// Per head h and token t, with S [key_pad][value_pad] fp32:
//   S <- diag(exp(log_decay)) S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q
// k and q are taken to unit length (x / sqrt(x.x + unit_eps)), q then times q_scale; heads / groups heads share them.
struct DeltaRule {
    const void *q, *k, *v;              // activation type, [T][ld]: [groups][key_pad], [groups][key_pad], [heads][value_pad]
    int ld;
    int heads, groups, key_pad, value_dim, value_pad;
    const float* log_decay;             // [T][heads * key_pad]
    const float* beta;                  // [T][heads]
    float q_scale, unit_eps;
    float* state;
    void* o;                            // activation type, [T][heads * value_pad]
    // one-token calls can norm and gate the output here: o / rms(o) * norm_w * sigmoid(gate) over value_dim (norm_w null: o
    // as it is); norm_w [heads * value_pad], gate activation type like o
    const float* norm_w;
    const void* gate;
    float eps;
    void* scratch;                      // delta_scratch_bytes() for long bf16 portions, else null
};
int delta_rule(const DeltaRule& a, int T, bool act_bf16, cudaStream_t s);
size_t delta_scratch_bytes(int heads, int key_pad, int value_pad, int T, bool act_bf16);
// Whether a one-token call takes norm and gate in.
bool delta_token_norms(int key_pad, int value_pad);

}  // namespace bpdq
