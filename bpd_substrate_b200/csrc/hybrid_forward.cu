// Forward pass of the hybrid decoders: a list of layers, each with one of five mixers (retention, state-space duality, gated delta
// rule, latent or grouped-query attention) and an optional feed-forward (SwiGLU or GELU), around one of two residuals.
//
// One stream, dynamic-tanh norms before and after every sublayer:
//   x = embed[token];   x += norm1b(mixer(norm1(x)));  x += norm2b(ff(norm2(x)))  per layer;   logits = head norm(x)
// Several streams joined by hyper-connections, RMS norms before every sublayer:
//   x_s = scale embed[token];   y = sublayer(norm(sum_s in_s x_s)),  x_t <- sum_s mix_st x_s + out_t y;   logits = head norm(sum_s x_s)
//
// Dynamic-tanh norms have no launch of their own: the product that ends a sublayer adds to the residual through its post norm
// and writes the next sublayer's normed input (linear.cu).  With streams, a one-token step does the same with the streams in the
// epilogue and the RMS norm in the product that follows; a prompt has one launch per sublayer for both (residual_streams.cu).
// Launches per layer for one token: 4 (retention: in, recurrence, gate + norm, out), 4 (state space: in with convolution and step
// sizes, recurrence, gate + norm, out), 4 (delta rule: in with convolutions and write shares, decays + gates, recurrence with gate
// and norm, out), 7 (latent attention), 4 (grouped attention: in, norms + cache, attention, out), 2 (feed-forward).  One-token steps
// are recorded as a CUDA graph per sequence slot and replayed; token and position are read from device memory.
#include "decayed_scan.cuh"
#include "delta_rule.cuh"
#include "grouped_attention.cuh"
#include "latent_attention.cuh"
#include "launch.cuh"
#include "residual_streams.cuh"
#include "../../include/bpdq.h"

#include <map>
#include <new>
#include <vector>

namespace bpdq {

// grid (columns / 1024, tokens), four columns per thread: the residual stream and the first sublayer's normed input.
template <typename A>
__global__ void __launch_bounds__(256) k_embed_norm(const bf16* __restrict__ table, const int32_t* tokens, float* x, A* h, DynTanh norm, int width,
                                                    int vocab, int* err)
{
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.y, c = 4 * (blockIdx.x * 256 + threadIdx.x);
    if (c >= width) return;
    const int tok = tokens[t];
    float4 v = make_float4(0, 0, 0, 0);
    if (tok >= 0 && tok < vocab) v = act_load4(table + (size_t)tok * width + c);
    else if (c == 0 && err) atomicCAS(err, 0, 21);      // no such row: nothing is read, code 21 is recorded
    *reinterpret_cast<float4*>(x + (size_t)t * width + c) = v;
    act_store4(h + (size_t)t * width + c, make_float4(dyn_tanh(norm, c, v.x), dyn_tanh(norm, c + 1, v.y), dyn_tanh(norm, c + 2, v.z), dyn_tanh(norm, c + 3, v.w)));
}

template <typename A>
__global__ void __launch_bounds__(256) k_gather_rows(const A* h, const int32_t* rows, A* out, int width, int n)
{
    pdl_launch_dependents();
    pdl_wait();
    const long total = (long)n * width;
    for (long u = (long)blockIdx.x * blockDim.x + threadIdx.x; u < total; u += (long)gridDim.x * blockDim.x) {
        const int r = (int)(u / width);
        out[u] = h[(size_t)rows[r] * width + (u - (long)r * width)];
    }
}

namespace {

struct Buffers {
    uint8_t* base = nullptr;
    size_t bytes = 0;
    int tokens = 0, context = 0, wanted = 0;
    float *x, *dt, *partial, *logits, *sum, *ys, *decays;
    void *h, *u, *o, *y, *xbc, *act, *cq, *q, *q_latent, *expanded, *rows, *gates, *chunks;
    int32_t *ids, *want;
    int* pos;
    long long* picked;
};

struct Plan {
    bpdq_hybrid_config cfg;
    std::vector<bpdq_hybrid_layer> layers;
    bool bf16_acts;
    Buffers one, many;                              // one-token steps (fixed, recorded in graphs), everything else
    Buffers* last = nullptr;                        // holds the results of the last call
    std::map<void*, cudaGraphExec_t> graphs;        // by state base
};

DynTanh norm_of(const bpdq_dyn_tanh& n) { return DynTanh{n.w, n.b, n.alpha}; }

LatentShape latent_shape(const Plan& p, const bpdq_hybrid_layer& l)
{
    LatentShape s = {};
    s.heads = l.heads;
    s.dim_pad = l.key_pad;
    s.value_pad = l.value_pad;
    s.rank = l.kv_rank; s.rank_pad = l.kv_rank_pad;
    s.rot_dims = l.rot_dims; s.rot_pad = l.rot_pad;
    s.q_rank = l.q_rank; s.q_rank_pad = l.q_rank_pad;
    s.rot_freq = l.rot_freq;
    s.scale = l.scale;
    s.eps = p.cfg.eps;
    return s;
}

GroupedShape grouped_shape(const Plan& p, const bpdq_hybrid_layer& l)
{
    GroupedShape s = {};
    s.heads = l.heads; s.groups = l.groups;
    s.dim = l.key_dim; s.dim_pad = l.key_pad;
    s.value_pad = l.value_pad;
    s.chunk = l.chunk;
    s.rows = l.cache_rows;
    s.sink = 1;
    s.scale = l.scale; s.cap = l.softcap;
    s.eps = p.cfg.eps;
    return s;
}

int in_rows(const bpdq_hybrid_layer& l)
{
    if (l.mixer == BPDQ_MIX_RETENTION) return 2 * l.heads * l.key_pad + 2 * l.heads * l.value_pad;
    if (l.mixer == BPDQ_MIX_MAMBA2) return 2 * l.heads * l.value_pad + 2 * l.groups * l.key_pad + l.heads;
    if (l.mixer == BPDQ_MIX_DELTA) return l.heads * l.value_pad + 2 * l.groups * l.key_pad + 2 * l.gate_rank_pad + l.heads;
    if (l.mixer == BPDQ_MIX_GROUPED) return l.heads * l.key_pad + (l.kv_from < 0 ? l.groups * (l.key_pad + l.value_pad) : 0);
    return l.q_rank_pad + (l.kv_from < 0 ? l.kv_rank_pad + l.rot_pad : 0);
}
// (of a state-space or delta-rule layer)
int conv_channels(const bpdq_hybrid_layer& l) { return l.heads * l.value_pad + 2 * l.groups * l.key_pad; }

// Lays the buffers out (base == null: counts bytes).  A buffer is as large as the largest layer needs it.
size_t lay_out(const Plan& p, Buffers& b, uint8_t* base, int T, int context, int wanted)
{
    const size_t a = p.bf16_acts ? 2 : 4, t = (size_t)T;
    const int W = p.cfg.width_pad;
    const bool streams = p.cfg.streams > 0;
    size_t u = 0, o = 0, xbc = 0, dt = 0, act = 0, cq = 0, q = 0, ql = 0, part = 0, exp = 0, gates = 0, decays = 0, chunks = 0;
    auto grow = [](size_t& m, size_t v) { if (v > m) m = v; };
    for (const auto& l : p.layers) {
        grow(u, t * ((in_rows(l) + 15) / 16 * 16));
        grow(o, t * l.heads * l.value_pad);
        grow(act, t * l.ff_pad);
        if (l.mixer == BPDQ_MIX_MAMBA2) {
            grow(xbc, t * conv_channels(l));
            grow(dt, t * l.heads);
        } else if (l.mixer == BPDQ_MIX_DELTA) {
            grow(xbc, t * conv_channels(l));
            grow(dt, t * l.heads);
            grow(gates, t * l.heads * l.value_pad);
            grow(decays, t * l.heads * l.key_pad);
            grow(chunks, delta_scratch_bytes(l.heads, l.key_pad, l.value_pad, T, p.bf16_acts));
        } else if (l.mixer == BPDQ_MIX_LATENT) {
            const LatentShape s = latent_shape(p, l);
            grow(cq, t * s.q_rank_pad);
            grow(q, t * s.heads * s.q_head());
            if (latent_expands(s, T, p.bf16_acts)) grow(exp, (size_t)context * s.heads * (s.dim_pad + s.value_pad));
            else grow(ql, t * s.heads * s.row());
            grow(part, latent_partial_floats(s, T, p.bf16_acts));
        }
    }
    size_t at = 0;
    auto take = [&](size_t bytes) -> uint8_t* {
        uint8_t* r = base ? base + at : nullptr;
        at += (bytes + 255) / 256 * 256;
        return r;
    };
    b.x = (float*)take(t * W * 4 * (streams ? p.cfg.streams : 1));
    b.sum = (float*)take(streams && T == 1 ? t * W * 4 : 0);
    b.ys = (float*)take(streams && T > 1 ? t * W * 4 : 0);
    b.h = take(t * W * a);
    b.u = take(u * a);
    b.o = take(o * a);
    b.y = take(o * a);
    b.xbc = take(xbc * a);
    b.act = take(act * a);
    b.cq = take(cq * a);
    b.q = take(q * a);
    b.q_latent = take(ql * a);
    b.expanded = take(exp * a);
    b.rows = take((size_t)wanted * W * a);
    b.gates = take(gates * a);
    b.chunks = take(chunks);
    b.decays = (float*)take(decays * 4);
    b.dt = (float*)take(dt * 4);
    b.partial = (float*)take(part * 4);
    b.logits = (float*)take((size_t)wanted * p.cfg.vocab * 4);
    b.ids = (int32_t*)take(t * 4);
    b.want = (int32_t*)take((size_t)wanted * 4);
    b.pos = (int*)take(4);
    b.picked = (long long*)take((size_t)wanted * 8);
    b.tokens = T;
    b.context = context;
    b.wanted = wanted;
    return at;
}

// Makes room for a call.  Buffers are laid out anew for every call's sizes (what depends on the number of tokens, like
// the number of key splits, is then as that call needs it) and the memory only grows.
int make_room(Plan& p, Buffers& b, int T, int context, int wanted, cudaStream_t s)
{
    const size_t need = lay_out(p, b, nullptr, T, context, wanted);
    if (need > b.bytes) {
        int rc;
        if (b.base) {
            if ((rc = check_cuda(cudaStreamSynchronize(s)))) return rc;
            check_cuda(cudaFree(b.base));
            b.base = nullptr;
            b.bytes = 0;
        }
        const size_t want = need + need / 4;
        void* m = nullptr;
        if ((rc = check_cuda(cudaMalloc(&m, want)))) return rc;
        b.base = (uint8_t*)m;
        b.bytes = want;
    }
    lay_out(p, b, b.base, T, context, wanted);
    return 0;
}

struct Runner {
    Plan& p;
    Buffers& b;
    int T, context;
    uint8_t* state;
    cudaStream_t s;

    void* at(void* base, size_t elements) const { return (uint8_t*)base + elements * (p.bf16_acts ? 2 : 4); }

    Linear product(const uint16_t* W, int N, int K, const void* in, int ld_in, void* out, int ld_out, int mode) const
    {
        Linear l = {};
        l.W = reinterpret_cast<const bf16*>(W);
        l.N = N; l.K = K;
        l.in = in; l.ld_in = ld_in;
        l.out = out; l.ld_out = ld_out;
        l.mode = mode;
        return l;
    }
    // A sublayer's place in the residual: its norms, its connections, and what reads afterwards.
    struct Sublayer {
        const bpdq_dyn_tanh *norm, *post, *next;
        const bpdq_stream_mix* mix;
        const float* next_in;
    };
    // The product that begins a sublayer, on its normed input.  With streams one token's norm is part of it.
    Linear open(const Sublayer& sub, const uint16_t* W, int N, void* out, int ld_out, int mode) const
    {
        Linear l = product(W, N, p.cfg.width_pad, b.h, p.cfg.width_pad, out, ld_out, mode);
        if (p.cfg.streams && T == 1) {
            l.in = b.sum;
            l.norm_w = sub.norm->w;
            l.norm_n = p.cfg.width;
            l.norm_eps = p.cfg.eps;
        }
        return l;
    }
    // The product that ends a sublayer.  One stream: residual add through the post norm, then the next sublayer's normed
    // input.  Several: into the streams, and what the next sublayer reads (of a prompt: normed).
    int close(const Sublayer& sub, const uint16_t* W, int K, const void* in) const
    {
        const int Wp = p.cfg.width_pad;
        Linear l = product(W, Wp, K, in, K, b.h, Wp, kLinResidual);
        l.x = b.x;
        l.ld_x = Wp;
        if (!p.cfg.streams) {
            l.post = norm_of(*sub.post);
            l.next = norm_of(*sub.next);
            return linear_forward(l, T, p.bf16_acts, s);
        }
        if (T == 1) {
            l.mode = kLinStreams;
            l.streams = stream_mix(*sub.mix, p.cfg.streams, sub.next_in);
            l.u = b.sum;
            return linear_forward(l, T, p.bf16_acts, s);
        }
        l.mode = kLinF32;
        l.out = b.ys;
        const int rc = linear_forward(l, T, p.bf16_acts, s);
        if (rc) return rc;
        StreamStep st = streams_of(*sub.next);
        st.y = b.ys;
        st.m = stream_mix(*sub.mix, p.cfg.streams, sub.next_in);
        return stream_step(st, T, p.bf16_acts, s);
    }
    // The streams, with `norm` ahead of what reads them.
    StreamStep streams_of(const bpdq_dyn_tanh& norm) const
    {
        StreamStep st = {};
        st.x = b.x;
        st.norm_w = norm.w;
        st.eps = p.cfg.eps;
        st.width = p.cfg.width;
        st.width_pad = p.cfg.width_pad;
        if (T == 1) st.u = b.sum;
        else st.h = b.h;
        return st;
    }

    int retention(const bpdq_hybrid_layer& l, const Sublayer& sub) const
    {
        const int HD = l.heads * l.key_pad, HV = l.heads * l.value_pad, N = in_rows(l);
        int rc = linear_forward(open(sub, l.w_in, N, b.u, N, kLinAct), T, p.bf16_acts, s);
        if (rc) return rc;
        DecayedScan a = {};
        a.q = b.u; a.k = at(b.u, HD); a.v = at(b.u, 2 * HD);
        a.ld_q = a.ld_k = a.ld_v = N;
        a.heads = a.groups = l.heads;
        a.key_pad = l.key_pad; a.value_pad = l.value_pad;
        a.decay = l.decay; a.log_decay = l.log_decay;
        a.state = (float*)(state + l.state_offset);
        a.o = b.o; a.ld_o = HV;
        if (T == 1) {
            a.rot_freq = l.rot_freq; a.rot_dims = l.rot_dims; a.pos = b.pos; a.k_scale = l.scale;
        } else if ((rc = rotate_half_qk(b.u, at(b.u, HD), N, l.heads, l.key_pad, l.rot_dims, l.rot_freq, l.scale, b.pos, T, p.bf16_acts, s))) {
            return rc;
        }
        if ((rc = decayed_scan(a, T, p.bf16_acts, s))) return rc;
        if ((rc = gated_norm(b.o, HV, at(b.u, 2 * HD + HV), N, nullptr, b.y, HV, l.heads, l.value_dim, l.value_pad, l.heads, 0, p.cfg.eps, T,
                             p.bf16_acts, s)))
            return rc;
        return close(sub, l.w_o, HV, b.y);
    }

    int mamba2(const bpdq_hybrid_layer& l, const Sublayer& sub) const
    {
        const int HV = l.heads * l.value_pad, GN = l.groups * l.key_pad, C = conv_channels(l), N = in_rows(l), ld = (N + 15) / 16 * 16;
        Linear in = open(sub, l.w_in, N, b.u, ld, kLinMixerIn);
        in.conv_row = HV;
        in.dt_row = HV + C;
        in.dt = b.dt;
        in.ld_dt = l.heads;
        in.dt_bias = l.dt_bias;
        float* tail = (float*)(state + l.tail_offset);
        if (T == 1) in.conv = ConvStep{l.conv_w, l.conv_b, tail, b.xbc, l.conv, C};
        int rc = linear_forward(in, T, p.bf16_acts, s);
        if (rc) return rc;
        if (T > 1 && (rc = causal_conv(at(b.u, HV), ld, b.xbc, C, l.conv, l.conv_w, l.conv_b, tail, T, p.bf16_acts, s))) return rc;
        DecayedScan a = {};
        a.v = b.xbc; a.k = at(b.xbc, HV); a.q = at(b.xbc, HV + GN);
        a.ld_q = a.ld_k = a.ld_v = C;
        a.heads = l.heads; a.groups = l.groups;
        a.key_pad = l.key_pad; a.value_pad = l.value_pad;
        a.dt = b.dt; a.ld_dt = l.heads; a.neg_exp_a = l.neg_exp_a;
        a.d_skip = l.d_skip;
        a.state = (float*)(state + l.state_offset);
        a.o = b.o; a.ld_o = HV;
        if ((rc = decayed_scan(a, T, p.bf16_acts, s))) return rc;
        if ((rc = gated_norm(b.o, HV, b.u, ld, l.norm_w, b.y, HV, l.heads, l.value_dim, l.value_pad, l.norm_groups, 1, p.cfg.eps, T, p.bf16_acts, s)))
            return rc;
        return close(sub, l.w_o, HV, b.y);
    }

    int latent(const bpdq_hybrid_layer& l, const Sublayer& sub) const
    {
        const LatentShape sh = latent_shape(p, l);
        const bool own = l.kv_from < 0;
        const int N = in_rows(l);
        void* cache = state + (own ? l : p.layers[l.kv_from]).cache_offset;
        int rc = linear_forward(open(sub, l.w_in, N, b.u, N, kLinAct), T, p.bf16_acts, s);
        if (rc) return rc;
        if ((rc = latent_prepare(sh, b.u, N, l.q_norm_w, l.kv_norm_w, b.cq, own ? cache : nullptr, b.pos, T, p.bf16_acts, s))) return rc;
        const int Q = sh.heads * sh.q_head();
        if ((rc = linear_forward(product(l.w_uq, Q, sh.q_rank_pad, b.cq, sh.q_rank_pad, b.q, Q, kLinAct), T, p.bf16_acts, s))) return rc;
        const LatentBuffers lb = {b.q_latent, b.partial, b.expanded};
        if ((rc = latent_attention(sh, b.q, reinterpret_cast<const bf16*>(l.w_ukv), cache, b.o, lb, b.pos, T, context, p.bf16_acts, s))) return rc;
        return close(sub, l.w_o, sh.heads * sh.value_pad, b.o);
    }

    // in rows: queries, keys, values (convolved), then what decays and gates are made of, then the write shares
    int delta(const bpdq_hybrid_layer& l, const Sublayer& sub) const
    {
        const int HD = l.heads * l.key_pad, HV = l.heads * l.value_pad, GD = l.groups * l.key_pad, C = conv_channels(l), R = l.gate_rank_pad;
        const int N = in_rows(l), ld = (N + 15) / 16 * 16;
        Linear in = open(sub, l.w_in, N, b.u, ld, kLinMixerIn);
        in.conv_row = 0;
        in.dt_row = C + 2 * R;
        in.dt = b.dt;
        in.ld_dt = l.heads;
        float* tail = (float*)(state + l.tail_offset);
        if (T == 1) in.conv = ConvStep{l.conv_w, nullptr, tail, b.xbc, l.conv, C};
        int rc = linear_forward(in, T, p.bf16_acts, s);
        if (rc) return rc;
        if (T > 1 && (rc = causal_conv(b.u, ld, b.xbc, C, l.conv, l.conv_w, nullptr, tail, T, p.bf16_acts, s))) return rc;
        Linear d = product(l.w_gates, HD, R, at(b.u, C), ld, b.gates, HV, kLinLogDecay);
        d.dt = b.decays;
        d.ld_dt = HD;
        d.dt_bias = l.dt_bias;
        d.neg_exp_a = l.neg_exp_a;
        if (T == 1) {           // decays and gates in one launch
            d.N = HD + HV;
            d.split = HD;
            d.in2 = R;
        } else if ((rc = linear_forward(product(l.w_gates + (size_t)HD * R, HV, R, at(b.u, C + R), ld, b.gates, HV, kLinAct), T, p.bf16_acts, s))) {
            return rc;
        }
        if ((rc = linear_forward(d, T, p.bf16_acts, s))) return rc;
        DeltaRule a = {};
        a.q = b.xbc; a.k = at(b.xbc, GD); a.v = at(b.xbc, 2 * GD);
        a.ld = C;
        a.heads = l.heads; a.groups = l.groups;
        a.key_pad = l.key_pad; a.value_dim = l.value_dim; a.value_pad = l.value_pad;
        a.log_decay = b.decays;
        a.beta = b.dt;
        a.q_scale = l.scale;
        a.unit_eps = 1e-6f;
        a.state = (float*)(state + l.state_offset);
        a.o = b.o;
        a.scratch = b.chunks;
        const bool norms = T == 1 && delta_token_norms(l.key_pad, l.value_pad);
        if (norms) {
            a.norm_w = l.norm_w;
            a.gate = b.gates;
            a.eps = p.cfg.eps;
        }
        if ((rc = delta_rule(a, T, p.bf16_acts, s))) return rc;
        if (!norms && (rc = gated_norm(b.o, HV, b.gates, HV, l.norm_w, b.y, HV, l.heads, l.value_dim, l.value_pad, l.heads, kNormWeightGate, p.cfg.eps, T,
                                       p.bf16_acts, s)))
            return rc;
        return close(sub, l.w_o, HV, norms ? b.o : b.y);
    }

    int grouped(const bpdq_hybrid_layer& l, const Sublayer& sub) const
    {
        const GroupedShape sh = grouped_shape(p, l);
        const bool own = l.kv_from < 0;
        const int N = in_rows(l);
        void* cache = state + (own ? l : p.layers[l.kv_from]).cache_offset;
        int rc = linear_forward(open(sub, l.w_in, N, b.u, N, kLinAct), T, p.bf16_acts, s);
        if (rc) return rc;
        if ((rc = grouped_prepare(sh, b.u, N, own ? cache : nullptr, b.pos, T, p.bf16_acts, s))) return rc;
        if ((rc = grouped_attention(sh, b.u, N, cache, b.o, b.pos, T, p.bf16_acts, s))) return rc;
        return close(sub, l.w_o, l.heads * l.value_pad, b.o);
    }

    int mix(const bpdq_hybrid_layer& l, const Sublayer& sub) const
    {
        switch (l.mixer) {
        case BPDQ_MIX_RETENTION: return retention(l, sub);
        case BPDQ_MIX_MAMBA2: return mamba2(l, sub);
        case BPDQ_MIX_DELTA: return delta(l, sub);
        case BPDQ_MIX_GROUPED: return grouped(l, sub);
        default: return latent(l, sub);
        }
    }

    int feed_forward(const bpdq_hybrid_layer& l, const Sublayer& sub) const
    {
        const bool gelu = l.ff_kind == BPDQ_FF_GELU;
        const int rc = linear_forward(open(sub, l.w_gate_up, gelu ? l.ff_pad : 2 * l.ff_pad, b.act, l.ff_pad, gelu ? kLinGelu : kLinSwiglu), T, p.bf16_acts, s);
        return rc ? rc : close(sub, l.w_down, l.ff_pad, b.act);
    }

    int embed(const Sublayer& first) const
    {
        const int W = p.cfg.width_pad;
        const bf16* table = reinterpret_cast<const bf16*>(p.cfg.embed);
        if (p.cfg.streams) {
            StreamStep st = streams_of(*first.norm);
            st.table = table;
            st.tokens = b.ids;
            st.embed_scale = p.cfg.embed_scale;
            st.vocab = p.cfg.vocab;
            st.m.n = p.cfg.streams;
            for (int i = 0; i < p.cfg.streams; i++) st.m.next[i] = first.next_in[i];
            return stream_step(st, T, p.bf16_acts, s);
        }
        const DynTanh norm = norm_of(*first.norm);
        return p.bf16_acts ? launch_ordered(k_embed_norm<bf16>, dim3((W + 1023) / 1024, T), 256, 0, s, table, (const int32_t*)b.ids, b.x, (bf16*)b.h, norm, W, p.cfg.vocab, device_error_flag())
                           : launch_ordered(k_embed_norm<float>, dim3((W + 1023) / 1024, T), 256, 0, s, table, (const int32_t*)b.ids, b.x, (float*)b.h, norm, W, p.cfg.vocab, device_error_flag());
    }

    int copy_residual(float* out) const
    {
        if (p.cfg.streams) return stream_sum(b.x, p.cfg.streams, p.cfg.width, p.cfg.width_pad, out, T, s);
        return check_cuda(cudaMemcpy2DAsync(out, (size_t)p.cfg.width * 4, b.x, (size_t)p.cfg.width_pad * 4, (size_t)p.cfg.width * 4, T,
                                            cudaMemcpyDeviceToDevice, s));
    }

    int run(float* residuals, int n_want, bool all_wanted) const
    {
        const int W = p.cfg.width_pad, n = (int)p.layers.size();
        float ones[BPDQ_MAX_STREAMS];
        for (float& v : ones) v = 1.0f;
        Sublayer last = {&p.cfg.final_norm, nullptr, nullptr, nullptr, ones};       // the output head
        auto mixer_of = [&](int i) {
            if (i >= n) return last;
            const bpdq_hybrid_layer& l = p.layers[i];
            return Sublayer{&l.norm1, &l.norm1b, nullptr, &l.mix1, l.mix1.in};
        };
        auto follow = [](Sublayer& a, const Sublayer& next) { a.next = next.norm; a.next_in = next.next_in; };
        // (a Sublayer's own reading weights are in next_in until the one that follows it is known)
        int rc = embed(mixer_of(0));
        if (rc) return rc;
        for (int i = 0; i < n; i++) {
            const bpdq_hybrid_layer& l = p.layers[i];
            Sublayer m = mixer_of(i), ff = {&l.norm2, &l.norm2b, nullptr, &l.mix2, l.mix2.in};
            follow(m, l.ff_pad ? ff : mixer_of(i + 1));
            if ((rc = mix(l, m))) return rc;
            if (l.ff_pad) {
                follow(ff, mixer_of(i + 1));
                if ((rc = feed_forward(l, ff))) return rc;
            }
            if (residuals && (rc = copy_residual(residuals + (size_t)i * T * p.cfg.width))) return rc;
        }
        if (n_want == 0) return 0;
        const bool vec = p.cfg.streams && T == 1;       // the norm is part of the product; the same row for every place
        const void* rows = b.h;
        if (!all_wanted && !vec) {
            rc = p.bf16_acts ? launch_ordered(k_gather_rows<bf16>, grid_1d((long)n_want * W), 256, 0, s, (const bf16*)b.h, (const int32_t*)b.want, (bf16*)b.rows, W, n_want)
                             : launch_ordered(k_gather_rows<float>, grid_1d((long)n_want * W), 256, 0, s, (const float*)b.h, (const int32_t*)b.want, (float*)b.rows, W, n_want);
            if (rc) return rc;
            rows = b.rows;
        }
        for (int i = 0; i < (vec ? n_want : 1); i++) {
            Linear head = open(last, p.cfg.head, p.cfg.vocab, b.logits + (size_t)i * p.cfg.vocab, p.cfg.vocab, kLinF32);
            if (!vec) head.in = rows;
            head.cap = p.cfg.logit_cap;
            if ((rc = linear_forward(head, vec ? 1 : n_want, p.bf16_acts, s))) return rc;
        }
        return bpd_argmax_dim_cuda(b.logits, b.picked, n_want, p.cfg.vocab, 1, s);
    }
};

int check_layer(const Plan& p, int i)
{
    const bpdq_hybrid_layer& l = p.layers[i];
    auto pad_ok = [](int v, int pad) { return v >= 1 && pad >= v && pad % 16 == 0; };
    if (l.heads < 1 || !pad_ok(l.key_dim, l.key_pad) || !pad_ok(l.value_dim, l.value_pad)) return BPDQ_ERR_ARG;
    if (!l.w_in || !l.w_o || (l.ff_pad && (l.ff_pad % 16 || !l.w_gate_up || !l.w_down))) return BPDQ_ERR_ARG;
    switch (l.mixer) {
    case BPDQ_MIX_RETENTION:
        if (l.rot_dims % 2 || l.rot_dims < 0 || l.rot_dims > l.key_dim || !l.decay || !l.log_decay || (l.rot_dims && !l.rot_freq)) return BPDQ_ERR_ARG;
        return l.key_pad > 512 ? BPDQ_ERR_RANGE : 0;
    case BPDQ_MIX_MAMBA2:
        if (l.groups < 1 || l.heads % l.groups || l.conv < 1 || l.norm_groups < 1 || (l.heads * l.value_dim) % l.norm_groups) return BPDQ_ERR_ARG;
        if (!l.conv_w || !l.conv_b || !l.dt_bias || !l.neg_exp_a || !l.d_skip || !l.norm_w) return BPDQ_ERR_ARG;
        return l.key_pad > 512 ? BPDQ_ERR_RANGE : 0;
    case BPDQ_MIX_LATENT:
        if (!pad_ok(l.kv_rank, l.kv_rank_pad) || !pad_ok(l.q_rank, l.q_rank_pad) || !pad_ok(l.rot_dims, l.rot_pad) || l.rot_dims % 2) return BPDQ_ERR_ARG;
        if (!l.w_uq || !l.w_ukv || !l.rot_freq || !l.q_norm_w) return BPDQ_ERR_ARG;
        if (l.kv_from < 0) return l.kv_norm_w ? 0 : BPDQ_ERR_ARG;
        if (l.kv_from >= i) return BPDQ_ERR_ARG;
        {
            const bpdq_hybrid_layer& o = p.layers[l.kv_from];
            return o.mixer == BPDQ_MIX_LATENT && o.kv_from < 0 && o.kv_rank == l.kv_rank && o.rot_dims == l.rot_dims ? 0 : BPDQ_ERR_ARG;
        }
    case BPDQ_MIX_DELTA:
        if (l.groups < 1 || l.heads % l.groups || l.conv < 1 || l.gate_rank_pad < 16 || l.gate_rank_pad % 16) return BPDQ_ERR_ARG;
        if (!l.conv_w || !l.dt_bias || !l.neg_exp_a || !l.norm_w || !l.w_gates) return BPDQ_ERR_ARG;
        return l.key_pad > 512 ? BPDQ_ERR_RANGE : 0;
    case BPDQ_MIX_GROUPED: {
        if (l.groups < 1 || l.heads % l.groups || l.chunk < 0 || l.cache_rows < 1 || l.softcap < 0.0f) return BPDQ_ERR_ARG;
        if (l.kv_from < 0) return 0;
        if (l.kv_from >= i) return BPDQ_ERR_ARG;
        const bpdq_hybrid_layer& o = p.layers[l.kv_from];
        return o.mixer == BPDQ_MIX_GROUPED && o.kv_from < 0 && o.groups == l.groups && o.key_dim == l.key_dim && o.value_dim == l.value_dim &&
                       o.cache_rows == l.cache_rows ? 0 : BPDQ_ERR_ARG;
    }
    default: return BPDQ_ERR_ARG;
    }
}

// Rows of a cache that are still needed by a portion's first token must not be those that its last token takes.
bool rows_suffice(const Plan& p, int pos, int T)
{
    for (const auto& l : p.layers)
        if (l.mixer == BPDQ_MIX_GROUPED && pos + T > l.cache_rows && (l.chunk == 0 || T + l.chunk - 1 > l.cache_rows)) return false;
    return true;
}

}  // namespace

}  // namespace bpdq

using namespace bpdq;

extern "C" {

void* bpdq_hybrid_create(const bpdq_hybrid_config* cfg, const bpdq_hybrid_layer* layers)
{
    if (!cfg || !cfg->embed || !cfg->head || cfg->streams < 0 || cfg->streams > BPDQ_MAX_STREAMS || cfg->logit_cap < 0.0f || cfg->n_layers < 0 || (cfg->n_layers && !layers) || cfg->width < 1 || cfg->width_pad < cfg->width ||
        cfg->width_pad % 16 || cfg->vocab < 1) {
        latch(BPDQ_ERR_ARG);
        return nullptr;
    }
    Plan* p = new (std::nothrow) Plan();
    if (!p) return nullptr;
    p->cfg = *cfg;
    p->layers.assign(layers, layers + cfg->n_layers);
    p->bf16_acts = cfg->act_bf16 != 0;
    for (int i = 0; i < cfg->n_layers; i++) {
        const int rc = check_layer(*p, i);
        if (rc) {
            latch(rc);
            delete p;
            return nullptr;
        }
    }
    return p;
}

void bpdq_hybrid_destroy(void* plan)
{
    Plan* p = (Plan*)plan;
    if (!p) return;
    check_cuda(cudaDeviceSynchronize());
    for (auto& g : p->graphs) check_cuda(cudaGraphExecDestroy(g.second));
    for (Buffers* b : {&p->one, &p->many})
        if (b->base) check_cuda(cudaFree(b->base));
    delete p;
}

int bpdq_hybrid_forward(void* plan, const int32_t* token_ids, int n_tokens, int pos, void* state, const int32_t* want, int n_want,
                        float* residuals, int use_graph, void* stream)
{
    Plan* p = (Plan*)plan;
    cudaStream_t s = (cudaStream_t)stream;
    if (!p || !token_ids || n_tokens < 1 || pos < 0 || !state || n_want < 0 || (n_want && !want)) return latch(BPDQ_ERR_ARG);
    if (n_tokens > 65535 || !rows_suffice(*p, pos, n_tokens)) return latch(BPDQ_ERR_RANGE);       // (tokens are a grid dimension)
    bool all = n_want == n_tokens;
    for (int i = 0; i < n_want; i++) {
        if (want[i] < 0 || want[i] >= n_tokens) return latch(BPDQ_ERR_RANGE);
        all = all && want[i] == i;
    }
    for (int i = 0; i < n_tokens; i++)
        if (token_ids[i] < 0 || token_ids[i] >= p->cfg.vocab) return latch(BPDQ_ERR_RANGE);
    const bool single = n_tokens == 1 && n_want <= 1;
    Buffers& b = single ? p->one : p->many;
    int rc = 0;
    if (!single) rc = make_room(*p, b, n_tokens, pos + n_tokens, n_want, s);
    else if (!b.base) rc = make_room(*p, b, 1, 1, 1, s);
    if (rc) return rc;
    // (copies from pageable memory: staged before the calls return)
    if ((rc = check_cuda(cudaMemcpyAsync(b.ids, token_ids, (size_t)n_tokens * 4, cudaMemcpyHostToDevice, s)))) return rc;
    if ((rc = check_cuda(cudaMemcpyAsync(b.pos, &pos, 4, cudaMemcpyHostToDevice, s)))) return rc;
    if (n_want && !all && (rc = check_cuda(cudaMemcpyAsync(b.want, want, (size_t)n_want * 4, cudaMemcpyHostToDevice, s)))) return rc;
    p->last = &b;
    Runner r{*p, b, n_tokens, pos + n_tokens, (uint8_t*)state, s};
    if (!single || !use_graph || residuals || n_want == 0) {
        rc = r.run(residuals, n_want, all);
        return rc ? latch(rc) : 0;
    }
    auto it = p->graphs.find(state);
    if (it == p->graphs.end()) {
        // the first one-token step of a slot runs launch by launch, so that every kernel's attributes are set outside a capture
        if ((rc = r.run(nullptr, 1, true))) return latch(rc);
        if ((rc = check_cuda(cudaStreamBeginCapture(s, cudaStreamCaptureModeThreadLocal)))) return rc;
        const int run_rc = r.run(nullptr, 1, true);
        cudaGraph_t g = nullptr;
        rc = check_cuda(cudaStreamEndCapture(s, &g));
        if (run_rc || rc || !g) {
            if (g) cudaGraphDestroy(g);
            return latch(run_rc ? run_rc : rc ? rc : BPDQ_ERR_CUDA);
        }
        cudaGraphExec_t e = nullptr;
        rc = check_cuda(cudaGraphInstantiate(&e, g, 0));
        cudaGraphDestroy(g);
        if (rc) return rc;
        p->graphs[state] = e;
        return 0;
    }
    return check_cuda(cudaGraphLaunch(it->second, s));
}

float* bpdq_hybrid_logits(void* plan)
{
    Plan* p = (Plan*)plan;
    return p && p->last ? p->last->logits : nullptr;
}
void* bpdq_hybrid_picked(void* plan)
{
    Plan* p = (Plan*)plan;
    return p && p->last ? p->last->picked : nullptr;
}
size_t bpdq_hybrid_scratch_bytes(void* plan)
{
    Plan* p = (Plan*)plan;
    return p ? p->one.bytes + p->many.bytes : 0;
}

}  // extern "C"
