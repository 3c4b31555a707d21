// Forward pass of the hybrid decoder: a list of layers, each with one of three mixers (retention, state-space duality,
// latent attention) and an optional SwiGLU feed-forward, dynamic-tanh norms before and after every sublayer, the
// embedding table as output head.
//
//   x = embed[token]
//   x += norm1b(mixer(norm1(x)));  x += norm2b(ff(norm2(x)))          per layer
//   logits = embed norm(x)
//
// Norms have no launch of their own: the product that ends a sublayer adds to the residual through its post norm and
// writes the next sublayer's normed input (linear.cu).  Launches per layer for one token: 4 (retention: in, recurrence,
// gate + norm, out), 4 (state space: in with convolution and step sizes, recurrence, gate + norm, out), 7 (latent
// attention), 2 (feed-forward).  One-token steps are recorded as a CUDA graph per sequence slot and replayed; token and
// position are read from device memory.
#include "decayed_scan.cuh"
#include "latent_attention.cuh"
#include "launch.cuh"
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
    float *x, *dt, *partial, *logits;
    void *h, *u, *o, *y, *xbc, *act, *cq, *q, *q_latent, *expanded, *rows;
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

int in_rows(const bpdq_hybrid_layer& l)
{
    if (l.mixer == BPDQ_MIX_RETENTION) return 2 * l.heads * l.key_pad + 2 * l.heads * l.value_pad;
    if (l.mixer == BPDQ_MIX_MAMBA2) return 2 * l.heads * l.value_pad + 2 * l.groups * l.key_pad + l.heads;
    return l.q_rank_pad + (l.kv_from < 0 ? l.kv_rank_pad + l.rot_pad : 0);
}
int conv_channels(const bpdq_hybrid_layer& l) { return l.heads * l.value_pad + 2 * l.groups * l.key_pad; }

// Lays the buffers out (base == null: counts bytes).  A buffer is as large as the largest layer needs it.
size_t lay_out(const Plan& p, Buffers& b, uint8_t* base, int T, int context, int wanted)
{
    const size_t a = p.bf16_acts ? 2 : 4, t = (size_t)T;
    const int W = p.cfg.width_pad;
    size_t u = 0, o = 0, xbc = 0, dt = 0, act = 0, cq = 0, q = 0, ql = 0, part = 0, exp = 0;
    auto grow = [](size_t& m, size_t v) { if (v > m) m = v; };
    for (const auto& l : p.layers) {
        grow(u, t * ((in_rows(l) + 15) / 16 * 16));
        grow(o, t * l.heads * l.value_pad);
        grow(act, t * l.ff_pad);
        if (l.mixer == BPDQ_MIX_MAMBA2) {
            grow(xbc, t * conv_channels(l));
            grow(dt, t * l.heads);
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
    b.x = (float*)take(t * W * 4);
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
    // the product that ends a sublayer: residual add through the post norm, then the next sublayer's normed input
    int close(const uint16_t* W, int K, const void* in, const bpdq_dyn_tanh& post, const bpdq_dyn_tanh& next) const
    {
        Linear l = product(W, p.cfg.width_pad, K, in, K, b.h, p.cfg.width_pad, kLinResidual);
        l.x = b.x;
        l.ld_x = p.cfg.width_pad;
        l.post = norm_of(post);
        l.next = norm_of(next);
        return linear_forward(l, T, p.bf16_acts, s);
    }

    int retention(const bpdq_hybrid_layer& l, const bpdq_dyn_tanh& next) const
    {
        const int HD = l.heads * l.key_pad, HV = l.heads * l.value_pad, N = in_rows(l);
        int rc = linear_forward(product(l.w_in, N, p.cfg.width_pad, b.h, p.cfg.width_pad, b.u, N, kLinAct), T, p.bf16_acts, s);
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
        return close(l.w_o, HV, b.y, l.norm1b, next);
    }

    int mamba2(const bpdq_hybrid_layer& l, const bpdq_dyn_tanh& next) const
    {
        const int HV = l.heads * l.value_pad, GN = l.groups * l.key_pad, C = conv_channels(l), N = in_rows(l), ld = (N + 15) / 16 * 16;
        Linear in = product(l.w_in, N, p.cfg.width_pad, b.h, p.cfg.width_pad, b.u, ld, kLinSsmIn);
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
        return close(l.w_o, HV, b.y, l.norm1b, next);
    }

    int latent(const bpdq_hybrid_layer& l, const bpdq_dyn_tanh& next) const
    {
        const LatentShape sh = latent_shape(p, l);
        const bool own = l.kv_from < 0;
        const int N = in_rows(l);
        void* cache = state + (own ? l : p.layers[l.kv_from]).cache_offset;
        int rc = linear_forward(product(l.w_in, N, p.cfg.width_pad, b.h, p.cfg.width_pad, b.u, N, kLinAct), T, p.bf16_acts, s);
        if (rc) return rc;
        if ((rc = latent_prepare(sh, b.u, N, l.q_norm_w, l.kv_norm_w, b.cq, own ? cache : nullptr, b.pos, T, p.bf16_acts, s))) return rc;
        const int Q = sh.heads * sh.q_head();
        if ((rc = linear_forward(product(l.w_uq, Q, sh.q_rank_pad, b.cq, sh.q_rank_pad, b.q, Q, kLinAct), T, p.bf16_acts, s))) return rc;
        const LatentBuffers lb = {b.q_latent, b.partial, b.expanded};
        if ((rc = latent_attention(sh, b.q, reinterpret_cast<const bf16*>(l.w_ukv), cache, b.o, lb, b.pos, T, context, p.bf16_acts, s))) return rc;
        return close(l.w_o, sh.heads * sh.value_pad, b.o, l.norm1b, next);
    }

    int run(float* residuals, int n_want, bool all_wanted) const
    {
        const int W = p.cfg.width_pad, n = (int)p.layers.size();
        const bf16* table = reinterpret_cast<const bf16*>(p.cfg.embed);
        const DynTanh first = norm_of(n ? p.layers[0].norm1 : p.cfg.final_norm);
        int rc = p.bf16_acts ? launch_ordered(k_embed_norm<bf16>, dim3((W + 1023) / 1024, T), 256, 0, s, table, (const int32_t*)b.ids, b.x, (bf16*)b.h, first, W, p.cfg.vocab, device_error_flag())
                             : launch_ordered(k_embed_norm<float>, dim3((W + 1023) / 1024, T), 256, 0, s, table, (const int32_t*)b.ids, b.x, (float*)b.h, first, W, p.cfg.vocab, device_error_flag());
        if (rc) return rc;
        for (int i = 0; i < n; i++) {
            const bpdq_hybrid_layer& l = p.layers[i];
            const bpdq_dyn_tanh& after = i + 1 < n ? p.layers[i + 1].norm1 : p.cfg.final_norm;
            const bpdq_dyn_tanh& next = l.ff_pad ? l.norm2 : after;
            rc = l.mixer == BPDQ_MIX_RETENTION ? retention(l, next) : l.mixer == BPDQ_MIX_MAMBA2 ? mamba2(l, next) : latent(l, next);
            if (rc) return rc;
            if (l.ff_pad) {
                if ((rc = linear_forward(product(l.w_gate_up, 2 * l.ff_pad, W, b.h, W, b.act, l.ff_pad, kLinSwiglu), T, p.bf16_acts, s))) return rc;
                if ((rc = close(l.w_down, l.ff_pad, b.act, l.norm2b, after))) return rc;
            }
            if (residuals)
                if ((rc = check_cuda(cudaMemcpy2DAsync(residuals + (size_t)i * T * p.cfg.width, (size_t)p.cfg.width * 4, b.x, (size_t)W * 4,
                                                       (size_t)p.cfg.width * 4, T, cudaMemcpyDeviceToDevice, s))))
                    return rc;
        }
        if (n_want == 0) return 0;
        const void* rows = b.h;
        if (!all_wanted) {
            rc = p.bf16_acts ? launch_ordered(k_gather_rows<bf16>, grid_1d((long)n_want * W), 256, 0, s, (const bf16*)b.h, (const int32_t*)b.want, (bf16*)b.rows, W, n_want)
                             : launch_ordered(k_gather_rows<float>, grid_1d((long)n_want * W), 256, 0, s, (const float*)b.h, (const int32_t*)b.want, (float*)b.rows, W, n_want);
            if (rc) return rc;
            rows = b.rows;
        }
        if ((rc = linear_forward(product(p.cfg.embed, p.cfg.vocab, W, rows, W, b.logits, p.cfg.vocab, kLinF32), n_want, p.bf16_acts, s))) return rc;
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
    default: return BPDQ_ERR_ARG;
    }
}

}  // namespace

}  // namespace bpdq

using namespace bpdq;

extern "C" {

void* bpdq_hybrid_create(const bpdq_hybrid_config* cfg, const bpdq_hybrid_layer* layers)
{
    if (!cfg || !cfg->embed || cfg->n_layers < 0 || (cfg->n_layers && !layers) || cfg->width < 1 || cfg->width_pad < cfg->width ||
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
    if (n_tokens > 65535) return latch(BPDQ_ERR_RANGE);       // tokens are a grid dimension
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
