"""The Vuzelix decoder on the device against the plain oracle: every mechanism alone through the C ABI, then whole models through
the engine's own step: prompts, token-by-token decoding, portions, chunk edges, cache rows and slots used again, interleaved requests,
greedy generation."""
import ctypes as C
import io
import json

import numpy as np
import pytest

from bpd_substrate_b200 import capi, generate, hybrid, trace, vuzelix
from bpd_substrate_b200.engine import Engine
from oracle import hybrid_oracle as ho
from oracle import vuzelix_oracle as vo
from tests import hybrid_models as hm
from tests import vuzelix_models as vm
from tests.test_hybrid_gpu import Act, done, feed_portions, pad16, save_model
from tests.util import Dev, normwise

pytestmark = pytest.mark.gpu
ACTS = [0, 1]
F64 = np.float64


# ------------------------------------------------------------------ epilogues of the products

@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,N,K", [(1, 70, 48), (1, 513, 16), (3, 130, 64), (40, 96, 80), (70, 257, 144), (300, 20, 32)])
def test_mapped_products(lib, bf16, T, N, K):
    act, rng = Act(bf16), np.random.default_rng(T + N)
    W, x = hm.bf16_round(rng.standard_normal((N, K)) * 4 / np.sqrt(K)), act.host(rng.standard_normal((T, K)))
    W[:4] *= 8                                     # sums that saturate a cap, a gelu and a sigmoid
    v = x.astype(F64) @ W.T.astype(F64)
    bias, rate = rng.uniform(-9, 2, N).astype(np.float32), -rng.uniform(0.1, 3, N).astype(np.float32)
    dW, dx, db, dr = Dev(lib, hm.bf16_bits(W)), act.up(lib, x), Dev(lib, bias), Dev(lib, rate)
    fine = 2e-5 if bf16 and T > 1 else 2e-6
    for kind, want in ((capi.MAP_GELU, vo.gelu_tanh(v)), (capi.MAP_CAP, vo.soft_cap(v, 7.0)), (capi.MAP_LOG_DECAY, rate * ho.softplus(v + bias)),
                       (capi.MAP_SIGMOID, vo.sigmoid(v))):
        do = act.empty(lib, T * N) if kind == capi.MAP_GELU else Dev(lib, nbytes=4 * T * N, fill=0xFF)
        done(lib, lib.bpd_linear_map_cuda(dW.ptr, dx.ptr, do.ptr, T, N, K, kind, db.ptr, dr.ptr, 7.0, bf16, None))
        got = (act.read(do) if kind == capi.MAP_GELU else do.read(np.float32)).reshape(T, N)
        assert normwise(got, want) < (act.tol if kind == capi.MAP_GELU else fine), kind
        if kind == capi.MAP_LOG_DECAY:             # small decays are exact in themselves, not only beside large ones
            small = (np.abs(want) < 0.05) & (np.abs(want) > 1e-7)
            assert small.any() and np.max(np.abs(got[small] / want[small] - 1)) < 2e-4


# ------------------------------------------------------------------ gated delta rule

def delta_case(lib, bf16, T, H, G, D, V, seed, state_scale=1.0, cut=None):
    """Runs T tokens (as portions of `cut` tokens) and compares outputs and state."""
    act, rng = Act(bf16), np.random.default_rng(seed)
    Dp, Vp = pad16(D), pad16(V)
    q, k, v = (act.host(rng.standard_normal(s)) for s in ((T, G, D), (T, G, D), (T, H, V)))
    beta = rng.uniform(0.05, 1.0, (T, H)).astype(np.float32)
    lg = -(10.0 ** rng.uniform(-5, 0, (T, H, D))).astype(np.float32)
    lg[:, :, ::3] = -1e-5                          # channels that hardly forget
    if D > 4:
        lg[:, :, 4] = -30.0                        # and one that forgets everything
    lg[T // 2, :, 1] = -200.0                      # a decay that underflows
    if T > 3:
        k[T - 1] = k[1]                            # the key written second is written again at the end, and a late query reads it
        q[T - 2] = k[1]
        k[2] = act.host(k[1] * 3 + 0.01 * k[2])    # nearly the same direction: the write is the small error that is left
        beta[1] = beta[2] = 1.0
    state = (state_scale * rng.standard_normal((H, D, V))).astype(np.float32)
    s, want = state.astype(F64), np.empty((T, H, V))
    qn, kn = vo.unit(q.astype(F64)) * D ** -0.5, vo.unit(k.astype(F64))
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            s[h], want[t, h] = vo.delta_step(s[h], np.exp(lg[t, h].astype(F64)), float(beta[t, h]), kn[t, g], v[t, h].astype(F64), qn[t, g])
    ld = 2 * G * Dp + H * Vp
    u = np.zeros((T, ld), np.float32)
    u[:, :G * Dp].reshape(T, G, Dp)[:, :, :D] = q
    u[:, G * Dp:2 * G * Dp].reshape(T, G, Dp)[:, :, :D] = k
    u[:, 2 * G * Dp:].reshape(T, H, Vp)[:, :, :V] = v
    lgp, sp = np.zeros((T, H, Dp), np.float32), np.zeros((H, Dp, Vp), np.float32)
    lgp[:, :, :D], sp[:, :D, :V] = lg, state
    du, dl, db, ds = act.up(lib, u), Dev(lib, lgp), Dev(lib, beta), Dev(lib, sp)
    do, size = act.empty(lib, T * H * Vp), 2 if bf16 else 4
    at = 0
    while at < T:
        n = T if cut is None else cut[0]
        cut = None if cut is None else cut[1:] + cut[:1]
        n = min(n, T - at)
        base = du.ptr + at * ld * size
        done(lib, lib.bpd_delta_rule_cuda(base, base + G * Dp * size, base + 2 * G * Dp * size, ld, dl.ptr + 4 * at * H * Dp, db.ptr + 4 * at * H, D ** -0.5,
                                          1e-6, ds.ptr, do.ptr + at * H * Vp * size, None, None, 0.0, n, H, G, Dp, V, Vp, bf16, None))
        at += n
    got, got_s = act.read(do).reshape(T, H, Vp), ds.read(np.float32).reshape(H, Dp, Vp)
    assert not got[:, :, V:].any() and not got_s[:, D:].any() and not got_s[:, :, V:].any()
    for h in range(H):
        assert normwise(got[:, h, :V], want[:, h]) < act.tol, h
        # nothing of the recurrence is rounded to bf16
        assert normwise(got_s[h, :D, :V], s[h]) < (4e-5 if bf16 else 4e-6), h


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,H,G,D,V", [(1, 3, 3, 16, 16), (1, 4, 2, 40, 72), (2, 4, 1, 48, 80), (15, 2, 2, 24, 32), (16, 2, 1, 128, 64), (17, 3, 3, 64, 144),
                                       (31, 2, 2, 144, 40), (32, 2, 2, 16, 16), (33, 4, 2, 72, 24), (47, 1, 1, 128, 128), (64, 6, 3, 32, 48),
                                       (100, 2, 1, 256, 32), (130, 2, 2, 200, 16), (70, 1, 1, 272, 16)])
def test_delta_rule(lib, bf16, T, H, G, D, V):
    delta_case(lib, bf16, T, H, G, D, V, 100 * T + D)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("D,V", [(500, 24), (100, 300), (256, 256)])
def test_delta_rule_one_token_sizes(lib, bf16, D, V):
    delta_case(lib, bf16, 1, 2, 1, D, V, D)
    delta_case(lib, bf16, 4, 2, 1, D, V, V)


@pytest.mark.parametrize("bf16", ACTS)
def test_delta_rule_portions_of_any_size(lib, bf16):
    """The state goes on from portion to portion, whichever kernel takes which."""
    delta_case(lib, bf16, 240, 2, 2, 40, 24, 3, cut=[33, 2, 1, 64, 16, 1, 1, 45])
    delta_case(lib, bf16, 150, 2, 1, 24, 40, 4, cut=[1])


@pytest.mark.parametrize("bf16", ACTS)
def test_delta_rule_more_tokens_than_a_segment(lib, bf16):
    delta_case(lib, bf16, 1100, 1, 1, 16, 16, 5)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("H,D,V", [(3, 16, 16), (2, 48, 40), (2, 32, 72), (5, 128, 128), (1, 24, 200), (2, 100, 256)])
def test_delta_rule_with_norm_and_gate(lib, bf16, H, D, V):
    act, rng = Act(bf16), np.random.default_rng(V)
    Dp, Vp, eps = pad16(D), pad16(V), 0.01
    q, k, v, gate = (act.host(rng.standard_normal(s)) for s in ((H, D), (H, D), (H, V), (H, V)))
    w = (1 + 0.3 * rng.standard_normal(V)).astype(np.float32)
    beta, lg = rng.uniform(0.1, 1, H).astype(np.float32), -rng.uniform(0, 1, (H, D)).astype(np.float32)
    state = 0.3 * rng.standard_normal((H, D, V)).astype(np.float32)
    want = np.empty((H, V))
    for h in range(H):
        _, o = vo.delta_step(state[h].astype(F64), np.exp(lg[h].astype(F64)), float(beta[h]), vo.unit(k[h].astype(F64)), v[h].astype(F64),
                             vo.unit(q[h].astype(F64)) * D ** -0.5)
        want[h] = ho.rms(o, eps) * w * vo.sigmoid(gate[h].astype(F64))

    def pad(x, size):
        return np.pad(x, [(0, 0)] * (x.ndim - 1) + [(0, size - x.shape[-1])]).reshape(-1)
    u = np.concatenate([pad(q, Dp), pad(k, Dp), pad(v, Vp)])
    sp = np.zeros((H, Dp, Vp), np.float32)
    sp[:, :D, :V] = state
    du, dg, dw, dl, db, ds = act.up(lib, u), act.up(lib, pad(gate, Vp)), Dev(lib, np.tile(pad(w[None], Vp), H)), Dev(lib, pad(lg, Dp)), Dev(lib, beta), Dev(lib, sp)
    do, size = act.empty(lib, H * Vp), 2 if bf16 else 4
    done(lib, lib.bpd_delta_rule_cuda(du.ptr, du.ptr + H * Dp * size, du.ptr + 2 * H * Dp * size, u.size, dl.ptr, db.ptr, D ** -0.5, 1e-6, ds.ptr, do.ptr, dw.ptr,
                                      dg.ptr, eps, 1, H, H, Dp, V, Vp, bf16, None))
    got = act.read(do).reshape(H, Vp)
    assert not got[:, V:].any() and normwise(got[:, :V], want) < act.tol
    # the same by the norm's own kernel, for several tokens
    o64 = act.host(rng.standard_normal((3, H, V)))
    g3 = act.host(rng.standard_normal((3, H, V)))
    d1, d2, dy = act.up(lib, pad(o64, Vp)), act.up(lib, pad(g3, Vp)), act.empty(lib, 3 * H * Vp)
    done(lib, lib.bpd_gated_norm_cuda(d1.ptr, H * Vp, d2.ptr, H * Vp, dw.ptr, dy.ptr, H * Vp, 3, H, V, Vp, H, 2, eps, bf16, None))
    want = ho.rms(o64.astype(F64), eps) * w * vo.sigmoid(g3.astype(F64))
    got = act.read(dy).reshape(3, H, Vp)
    assert not got[:, :, V:].any() and normwise(got[:, :, :V], want) < act.tol


# ------------------------------------------------------------------ grouped attention

def attention_case(lib, bf16, T, pos, H, G, D, V, chunk, rows=None, seed=0, sink=1, cap=14.0):
    """Positions up to pos + T - 1 of which the last T are run; the cache is filled by earlier calls.  Some (query, head) look for one
    key that stands out: the first and the last of the chunk, far ones, block edges, and keys just outside the chunk, which
    must not be seen."""
    act, rng = Act(bf16), np.random.default_rng(seed + T + 7 * pos)
    Dp, Vp, L, eps = pad16(D), pad16(V), pos + T, 0.001
    rows, scale = rows or L + 5, 24.0 / D
    q, k, v = (act.host(rng.standard_normal(s)) for s in ((L, H, D), (L, G, D), (L, G, V)))
    for t in range(pos, L):
        lo = t // chunk * chunk if chunk else 0
        spots = [x for x in (lo, lo - 1, t, t - 1, lo + 1, (lo + t) // 2, lo + 63, lo + 64, lo + 16, 0) if 0 <= x <= t]
        for h in range(H):
            if lo and h == t % H:
                q[t, h] = act.host(k[lo - 1, h // (H // G)])
            elif (t + h) % 3:
                s = spots[(t + 2 * h) % len(spots)]
                q[t, h] = act.host(k[s, h // (H // G)] * (1 if (t + h) % 5 else -1))     # (or away from it: the sink takes over)
    qn, kn = ho.rms(q.astype(F64), eps), ho.rms(k.astype(F64), eps)
    want = np.empty((T, H, V))
    for t in range(pos, L):
        seen = [j for j in range(L) if vo.sees(t, j, chunk)]
        for h in range(H):
            g = h // (H // G)
            if sink:
                want[t - pos, h] = vo.attend(qn[t, h], kn[seen, g], v[seen, g].astype(F64), scale, cap)
            else:
                s = vo.soft_cap(kn[seen, g] @ qn[t, h] * scale, cap) if cap else kn[seen, g] @ qn[t, h] * scale
                e = np.exp(s - s.max())
                want[t - pos, h] = e / e.sum() @ v[seen, g]
    ld = H * Dp + G * (Dp + Vp)
    u = np.zeros((L, ld), np.float32)
    u[:, :H * Dp].reshape(L, H, Dp)[:, :, :D] = q
    u[:, H * Dp:(H + G) * Dp].reshape(L, G, Dp)[:, :, :D] = k
    u[:, (H + G) * Dp:].reshape(L, G, Vp)[:, :, :V] = v
    shape = capi.GroupedShape(H, G, D, Dp, Vp, chunk, rows, sink, scale, cap, eps)
    size = 2 if bf16 else 4
    du, dc, do = act.up(lib, u), act.empty(lib, rows * G * (Dp + Vp)), act.empty(lib, L * H * Vp)        # (the cache holds NaN before it is written)
    dp = Dev(lib, np.array([pos], np.int32))
    limit = rows - chunk + 1 if rows < L else L
    step = 0
    while step < pos:       # the tokens before, in portions that the cache's rows allow
        n = min(limit, pos - step, 50)
        d = Dev(lib, np.array([step], np.int32))
        done(lib, lib.bpd_grouped_attention_cuda(C.byref(shape), du.ptr + step * ld * size, ld, dc.ptr, 1, do.ptr, d.ptr, n, bf16, None))
        step += n
    done(lib, lib.bpd_grouped_attention_cuda(C.byref(shape), du.ptr + pos * ld * size, ld, dc.ptr, 1, do.ptr, dp.ptr, T, bf16, None))
    got = act.read(do)[:T * H * Vp].reshape(T, H, Vp)
    assert not got[:, :, V:].any()
    scale_of = np.abs(v).max()
    for t in range(T):
        for h in range(H):
            assert np.max(np.abs(got[t, h, :V] - want[t, h])) < scale_of * (1.2e-2 if bf16 else 1e-5), (t, h)
    # a layer that borrows the keys: its own queries, nothing appended
    q2 = act.host(rng.standard_normal((T, H, D)))
    u2 = np.zeros((T, H * Dp), np.float32)
    u2.reshape(T, H, Dp)[:, :, :D] = q2
    d2, before = act.up(lib, u2), dc.read(np.uint8).copy()
    done(lib, lib.bpd_grouped_attention_cuda(C.byref(shape), d2.ptr, H * Dp, dc.ptr, 0, do.ptr, dp.ptr, T, bf16, None))
    assert np.array_equal(dc.read(np.uint8), before)
    got = act.read(do)[:T * H * Vp].reshape(T, H, Vp)
    if sink:
        qn = ho.rms(q2.astype(F64), eps)
        for t in {0, T // 2, T - 1}:
            seen = [j for j in range(L) if vo.sees(pos + t, j, chunk)]
            for h in range(H):
                w = vo.attend(qn[t, h], kn[seen, h // (H // G)], v[seen, h // (H // G)].astype(F64), scale, cap)
                assert np.max(np.abs(got[t, h, :V] - w)) < scale_of * (1.2e-2 if bf16 else 1e-5), (t, h)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,pos", [(1, 0), (1, 36), (1, 37), (1, 38), (1, 73), (1, 74), (2, 36), (2, 35), (5, 0), (20, 60), (70, 0), (75, 30), (130, 36), (40, 111)])
def test_grouped_attention_at_chunk_edges(lib, bf16, T, pos):
    attention_case(lib, bf16, T, pos, 6, 2, 20, 28, 37)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,pos,H,G,D,V,chunk", [(1, 700, 4, 2, 32, 32, 0), (1, 900, 8, 1, 128, 128, 1000), (1, 300, 2, 2, 64, 16, 256), (3, 257, 16, 1, 16, 48, 128),
                                                 (2, 400, 40, 2, 24, 24, 300), (1, 150, 3, 3, 200, 256, 100), (1, 90, 2, 1, 264, 24, 64), (60, 100, 2, 1, 264, 24, 90),
                                                 (150, 40, 4, 1, 128, 136, 64), (90, 10, 5, 1, 40, 272, 1), (66, 0, 1, 1, 8, 8, 2), (40, 200, 4, 2, 144, 64, 0)])
def test_grouped_attention_sizes(lib, bf16, T, pos, H, G, D, V, chunk):
    attention_case(lib, bf16, T, pos, H, G, D, V, chunk)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,pos,chunk,rows", [(1, 200, 37, 70), (1, 200, 100, 128), (30, 170, 37, 70), (64, 260, 50, 113), (80, 300, 1, 80), (1, 333, 64, 64), (2, 190, 90, 91)])
def test_grouped_attention_rows_used_again(lib, bf16, T, pos, chunk, rows):
    attention_case(lib, bf16, T, pos, 6, 2, 24, 40, chunk, rows)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("cap", [2.0, 60.0, 90.0, 500.0])
def test_grouped_attention_caps(lib, bf16, cap):
    for T, pos in ((1, 70), (90, 20)):
        attention_case(lib, bf16, T, pos, 4, 2, 32, 72, 48, cap=cap)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,pos", [(1, 130), (90, 20)])
def test_grouped_attention_without_sink_or_cap(lib, bf16, T, pos):
    attention_case(lib, bf16, T, pos, 4, 2, 32, 32, 48, sink=0)
    attention_case(lib, bf16, T, pos, 4, 2, 32, 32, 48, sink=0, cap=0.0)


# ------------------------------------------------------------------ residual streams

@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,S,W", [(1, 1, 16), (3, 2, 40), (2, 3, 1030), (5, 4, 200), (2, 8, 4100), (2, 5, 72), (1, 4, 6000)])
def test_stream_step(lib, bf16, T, S, W):
    act, rng = Act(bf16), np.random.default_rng(W)
    Wp, eps, N = pad16(W), 0.01, capi.MAX_STREAMS
    x, y = np.zeros((T, S, Wp), np.float32), np.zeros((T, Wp), np.float32)
    x[:, :, :W], y[:, :W] = rng.standard_normal((T, S, W)), rng.standard_normal((T, W))
    mix, out, into = (rng.standard_normal(s).astype(np.float32) for s in ((S, S), (S,), (S,)))
    w = np.pad(1 + 0.2 * rng.standard_normal(W), (0, Wp - W)).astype(np.float32)
    d = capi.StreamMix()
    for s in range(S):
        d.out[s], d.in_[s] = out[s], into[s]
        for t in range(S):
            d.mix[s * N + t] = mix[s, t]
    dx, dy, dw, dh, du = Dev(lib, x), Dev(lib, y), Dev(lib, w), act.empty(lib, T * Wp), Dev(lib, nbytes=4 * T * Wp, fill=0xFF)
    done(lib, lib.bpd_stream_step_cuda(dy.ptr, dx.ptr, C.byref(d), S, dw.ptr, eps, T, W, Wp, dh.ptr, du.ptr, bf16, None))
    got_x, got_u, got_h = dx.read(np.float32).reshape(x.shape), du.read(np.float32).reshape(T, Wp), act.read(dh).reshape(T, Wp)
    for t in range(T):
        want = vo.write_streams(x[t].astype(F64), y[t].astype(F64), mix.astype(F64), out.astype(F64), 1.0)
        u = vo.read_streams(want, into.astype(F64))
        assert normwise(got_x[t], want) < 1e-6 and normwise(got_u[t], u) < 2e-6
        assert normwise(got_h[t, :W], ho.rms(u[:W], eps) * w[:W]) < act.tol and not got_h[t, W:].any()


# ------------------------------------------------------------------ whole models

LIMIT = {"float32": 4e-5, "bfloat16": 8e-2}


@pytest.fixture(scope="module", params=list(vm.CONFIGS))
def case(request):
    cfg = vm.CONFIGS[request.param]
    w = vm.weights(cfg, 11)
    toks = hm.tokens(cfg, 150, 4)
    logits, res = vo.Model(cfg, w).run(toks)
    return cfg, w, toks, logits, res


def device(cfg, w, lib, dtype, capacity=256, spec_class=vuzelix.VuzelixSpec, **kw):
    return hybrid.DeviceHybrid(spec_class(cfg), hybrid.ArrayTensors(w), dtype=dtype, capacity=capacity, lib=lib, **kw)


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_residual_stream_layer_by_layer(lib, case, dtype):
    cfg, w, toks, _, res = case
    m = device(cfg, w, lib, dtype)
    e = Engine(m)
    limit = 1.5e-5 if dtype == "float32" else 5e-2
    for one_by_one in (False, True):
        seq, n = e.slots.acquire(), 40 if one_by_one else 90
        got = np.concatenate([m.residuals(seq, [t]) for t in toks[:n]], 1) if one_by_one else m.residuals(seq, toks[:n])
        for i in range(len(cfg["layers"])):
            assert np.max(hm.row_errors(got[i], res[i][:n])) < limit, (one_by_one, i)
        e.slots.release(seq)
    e.close()
    m.close()


CUTS = ([150], [1] * 150, [118] + [1] * 32, [2] * 75, [33, 2, 37, 14, 22, 3, 1, 1, 37], [64, 64, 22], [65, 1, 63, 1, 20], [70, 80], [1, 149], [149, 1],
        [16, 17, 15, 31, 32, 39], [24, 16, 24, 24, 10, 2, 50])


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_prompt_portions_and_decoding(lib, case, dtype):
    """The logits of every position, however the sequence is cut; one slot, used again by every run."""
    cfg, w, toks, want, _ = case
    m = device(cfg, w, lib, dtype)
    e = Engine(m)
    for sizes in CUTS:
        err = hm.row_errors(feed_portions(e, "r", toks, sizes), want)
        assert np.max(err) < LIMIT[dtype], (sizes[:4], int(np.argmax(err)), float(np.max(err)))
    assert m.lib.bpdq_last_status() == 0
    e.close()
    m.close()


class ShortRows(vuzelix.VuzelixSpec):
    """Attention layers keep 20 rows beyond a chunk."""
    portion = 20


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_cache_rows_used_again(lib, case, dtype):
    """Caches that keep less than the sequence: portions as long as they allow, single tokens, and longer prompts cut by the engine."""
    cfg, w, toks, want, _ = case
    m = device(cfg, w, lib, dtype, spec_class=ShortRows)
    assert m.portion == 20 and any(p.limit and p.count(256) < 150 for p in m.parts)
    e = Engine(m)
    assert e.portion == 20
    for sizes in ([20] * 7 + [10], [150], [1] * 150, [7, 20, 20, 1, 1, 19, 2, 20, 60]):
        err = hm.row_errors(feed_portions(e, "r", toks, sizes), want)
        assert np.max(err) < LIMIT[dtype], (sizes[:4], int(np.argmax(err)), float(np.max(err)))
    seq = e.slots.acquire()
    with pytest.raises(ValueError, match="up to 20"):
        m.launch(seq, toks[:21])
    e.close()
    m.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_interleaved_requests_equal_each_alone(lib, dtype):
    """Live requests in several slots, steps taken in turn, slots given back and used again; recorded one-token steps
    and launch-by-launch ones give the same bits."""
    cfg = vm.CONFIGS["mixed"]
    w = vm.weights(cfg, 21)
    seqs = {k: hm.tokens(cfg, n, n) for k, n in (("a", 41), ("b", 7), ("c", 90), ("d", 23))}
    cuts = {"a": [30] + [1] * 11, "b": [1] * 7, "c": [2, 60, 3] + [1] * 25, "d": [5, 5, 5, 5, 3]}
    m = device(cfg, w, lib, dtype, capacity=128)
    e = Engine(m, slots=1)
    alone = {k: feed_portions(e, k, seqs[k], cuts[k]) for k in seqs}
    e.close()
    m.close()
    m = device(cfg, w, lib, dtype, capacity=128, use_graph=False)
    e = Engine(m, slots=2)
    got, at, live, waiting = {k: [] for k in seqs}, dict.fromkeys(seqs, 0), [], list(seqs)
    while live or waiting:
        while waiting and len(live) < 2:
            live.append(waiting.pop(0))
        for k in list(live):
            n = cuts[k][len(got[k])]
            lg, _ = e.feed(k, seqs[k][at[k]:at[k] + n], range(n))
            got[k].append(lg)
            at[k] += n
            if at[k] == len(seqs[k]):
                e.end(k)
                live.remove(k)
    for k in seqs:
        assert np.array_equal(np.concatenate(got[k]).view(np.uint32), alone[k].view(np.uint32)), k
    e.close()
    m.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_long_decoding(lib, dtype):
    cfg = vm.CONFIGS["square"]
    w, toks = vm.weights(cfg, 5), hm.tokens(cfg, 420, 6)
    want, _ = vo.Model(cfg, w).run(toks)
    m = device(cfg, w, lib, dtype, capacity=420)
    e = Engine(m)
    assert np.max(hm.row_errors(feed_portions(e, 0, toks, [20] + [1] * 400), want)) < LIMIT[dtype]
    lg, ids = e.feed(1, toks[:60], [59, 3, 3])              # places in any order, and twice
    assert np.max(hm.row_errors(lg, want[[59, 3, 3]])) < LIMIT[dtype] and np.array_equal(ids, lg.argmax(1))
    lg, _ = e.feed(1, toks[60:61], [0, 0])
    assert np.max(hm.row_errors(lg, want[[60, 60]])) < LIMIT[dtype]
    with pytest.raises(ValueError, match="room for 420"):
        e.feed(1, toks[:400])
    e.close()
    m.close()


def looking_model(kind, chunk=400):
    """One layer in which token 61 looks for what token 62 left: with attention the key of 62, with the delta rule the value written at
    its key into channels that do not decay."""
    mixer = vm.attention(2, 1, 32, 32, chunk, 1.0, 20.0) if kind == "attention" else vm.delta(2, 1, 32, 32, 1)
    cfg = vm.config(64, 48, 2, [vm.layer(kind, mixer)], mult=1.0)
    w, p = vm.weights(cfg, 9), "l0.mix."
    w64 = {k: v.astype(F64) for k, v in w.items()}

    def seen(tok):
        x = np.tile(w64["embed"][tok] * cfg["embedding"]["scale"], (2, 1))
        return ho.rms(vo.read_streams(x, w64["l0.hc1.in"]), cfg["norm"]["eps"]) * w64["l0.norm1"]
    h61, key = seen(61), w64[p + "k"] @ seen(62)
    q = np.stack([np.outer(key, h61)] * 2) if kind == "attention" else np.outer(key, h61)[None]
    w[p + "q"] = hm.bf16_round(q.reshape(-1, 48) * 40.0 / (h61 @ h61) + 0.05 * w64[p + "q"])
    if kind == "channel_delta":
        for n in "qkv":
            w[f"{p}{n}.conv"][:] = 1.0
        w[p + "dt_bias"][:], w[p + "b"] = -14.0, hm.bf16_round(w64[p + "b"] + 3.0 * np.outer(np.ones(2), seen(62)) / (seen(62) @ seen(62)))
    w[p + "o"] = hm.bf16_round(4.0 * w64[p + "o"])
    return cfg, w


def check_far_token(lib, cfg, w, toks, far, matters, sizes_of, fine):
    want, _ = vo.Model(cfg, w).run(toks)
    other = list(toks)
    other[far] = 63
    blind, _ = vo.Model(cfg, w).run(other)
    err = hm.row_errors(want[-1:], blind[-1:])[0]
    assert err > 0.1 if matters else err < 1e-9, err
    for dtype in LIMIT:
        m = device(cfg, w, lib, dtype, capacity=len(toks))
        e = Engine(m)
        for sizes in sizes_of(len(toks)):
            err = hm.row_errors(feed_portions(e, 0, toks, sizes), want)
            assert np.max(err) < (fine if dtype == "float32" else 0.15), (dtype, sizes[:2], int(np.argmax(err)))
        e.close()
        m.close()


@pytest.mark.parametrize("n,far,matters", [(400, 0, True), (401, 399, False), (430, 400, True), (800, 400, True), (450, 3, False)])
def test_a_far_key_shows_within_its_chunk_only(lib, n, far, matters):
    """The looking token at the end sees the other one from the far end of its chunk, and not one position beyond it."""
    cfg, w = looking_model("attention")
    toks = np.random.default_rng(0).integers(1, 60, n).tolist()
    toks[far], toks[-1] = 62, 61
    check_far_token(lib, cfg, w, toks, far, matters, lambda n: ([n], [n - 1, 1], [n - 20] + [1] * 20, [100] * (n // 100) + ([n % 100] if n % 100 else [])), 1e-4)


def test_a_far_write_shows_in_the_state(lib):
    cfg, w = looking_model("channel_delta")
    toks = np.random.default_rng(1).integers(1, 3, 300).tolist()         # a few directions only are written in between
    toks[0], toks[-1] = 62, 61
    check_far_token(lib, cfg, w, toks, 0, True, lambda n: ([n], [n - 1, 1], [100] + [1] * 200, [31, 33, 2, 234]), 1e-4)


def test_greedy_generation_through_the_command_line(lib, tmp_path, capsys):
    cfg = vm.CONFIGS["mixed"]
    w = vm.weights(cfg, 31)
    save_model(tmp_path, cfg, w)
    prompts = [hm.tokens(cfg, n, n) for n in (3, 40, 1, 17)]
    args = ["--model", str(tmp_path), "--max-new", "12", "--dtype", "float32", "--capacity", "64", "--slots", "2", "--portion", "16"]
    for p in prompts:
        args += ["--prompt", " ".join(map(str, p))]
    assert generate.main(args) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.splitlines()]
    ref = vo.Model(cfg, w)
    assert [x["prompt"] for x in lines] == prompts
    assert [x["output"] for x in lines] == [ref.greedy(p, 12) for p in prompts]


def test_trace_replay_from_a_folder(lib, tmp_path, monkeypatch):
    cfg = vm.CONFIGS["single"]
    w = vm.weights(cfg, 41)
    save_model(tmp_path, cfg, w)
    toks = hm.tokens(cfg, 30, 3)
    want, _ = vo.Model(cfg, w).run(toks)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": toks[:20], "want": [4, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": toks[20:], "want": [9]}], "end": ["q"]},
             {"step": 2, "entries": [{"id": "p", "tokens": toks[:1], "want": [0]}], "end": ["p"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "30"]) == 0
    for i, rows in enumerate(([4, 19], [29], [0])):
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(len(rows), cfg["vocab"])
        assert np.max(hm.row_errors(got, want[rows])) < LIMIT["float32"]


def test_refused_calls(lib):
    d = Dev(lib, nbytes=1 << 16)
    shape = capi.GroupedShape(3, 2, 16, 16, 16, 0, 8, 1, 1.0, 0.0, 1e-5)
    assert lib.bpd_grouped_attention_cuda(C.byref(shape), d.ptr, 96, d.ptr, 1, d.ptr, d.ptr, 1, 1, None) == -1
    assert lib.bpd_delta_rule_cuda(d.ptr, d.ptr, d.ptr, 64, d.ptr, d.ptr, 1.0, 1e-6, d.ptr, d.ptr, None, None, 0.0, 1, 3, 2, 16, 16, 16, 1, None) == -1
    mix = capi.StreamMix()
    assert lib.bpd_stream_step_cuda(d.ptr, d.ptr, C.byref(mix), 9, d.ptr, 1e-5, 1, 16, 16, d.ptr, None, 1, None) == -3
    assert lib.bpd_linear_map_cuda(d.ptr, d.ptr, d.ptr, 1, 4, 16, 9, None, None, 0.0, 1, None) == -1
    lib.bpdq_clear_status()
