"""The hybrid decoder on the device against the plain oracle: every mechanism alone through the C ABI, then whole models
through the engine's own step: prompts, token-by-token decoding, portions, slots used again, interleaved requests, greedy
generation."""
import ctypes as C
import io
import json

import numpy as np
import pytest

from bpd_substrate_b200 import capi, generate, hybrid, safetensors_load, trace
from bpd_substrate_b200.engine import Engine
from oracle import hybrid_oracle as ho
from tests import hybrid_models as hm
from tests.util import Dev, normwise

pytestmark = pytest.mark.gpu
ACTS = [0, 1]


class Act:
    """Activations of one type: values the device holds exactly, and how to read them back."""

    def __init__(self, bf16):
        self.bf16 = bf16
        self.tol = 6e-3 if bf16 else 2e-6         # of results stored in this type

    def host(self, x):
        return hm.bf16_round(x) if self.bf16 else np.asarray(x, np.float32)

    def up(self, lib, x):
        x = self.host(x)
        return Dev(lib, hm.bf16_bits(x) if self.bf16 else x)

    def empty(self, lib, n):
        return Dev(lib, nbytes=n * (2 if self.bf16 else 4), fill=0xFF)

    def read(self, d):
        return hm.bits_f32(d.read(np.uint16)) if self.bf16 else d.read(np.float32)


def pad16(n):
    return -(-n // 16) * 16


def done(lib, rc):
    assert rc == 0
    lib.bpdq_sync()
    assert lib.bpdq_last_status() == 0


# ------------------------------------------------------------------ matrix products

@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,N,K", [(1, 17, 16), (1, 700, 1040), (1, 5000, 48), (2, 130, 48), (7, 16, 4096), (33, 129, 80), (64, 1000, 336),
                                   (65, 130, 64), (129, 257, 144), (300, 96, 2064)])
def test_linear(lib, bf16, T, N, K):
    act, rng = Act(bf16), np.random.default_rng(T + N)
    W, x = hm.bf16_round(rng.standard_normal((N, K))), act.host(rng.standard_normal((T, K)))
    dW, dx, do = Dev(lib, hm.bf16_bits(W)), act.up(lib, x), Dev(lib, nbytes=4 * T * N, fill=0xFF)
    done(lib, lib.bpd_linear_bf16_cuda(dW.ptr, dx.ptr, do.ptr, T, N, K, bf16, None))
    # (the tensor cores keep fewer low-order bits of a long fp32 sum than a chain of fp32 additions)
    limit = 2e-5 if bf16 and T > 1 else 2e-6
    assert normwise(do.read(np.float32).reshape(T, N), x.astype(np.float64) @ W.T.astype(np.float64)) < limit


def test_linear_many_tiles_per_cta(lib):
    """More 128 x 256 tiles than CTAs: the persistent walk and both accumulators."""
    T, N, K = 700, 128 * 120 + 40, 208
    rng = np.random.default_rng(5)
    W, x = hm.bf16_round(rng.standard_normal((N, K))), hm.bf16_round(rng.standard_normal((T, K)))
    dW, dx, do = Dev(lib, hm.bf16_bits(W)), Dev(lib, hm.bf16_bits(x)), Dev(lib, nbytes=4 * T * N, fill=0xFF)
    done(lib, lib.bpd_linear_bf16_cuda(dW.ptr, dx.ptr, do.ptr, T, N, K, 1, None))
    assert normwise(do.read(np.float32).reshape(T, N), x @ W.T) < 1e-5


def test_linear_rejects_bad_arguments(lib):
    d = Dev(lib, nbytes=4096)
    assert lib.bpd_linear_bf16_cuda(d.ptr, d.ptr, d.ptr, 1, 4, 24, 1, None) == -1
    assert lib.bpd_linear_bf16_cuda(None, d.ptr, d.ptr, 1, 4, 16, 1, None) == -1
    assert lib.bpd_linear_bf16_cuda(d.ptr + 2, d.ptr, d.ptr, 1, 4, 16, 1, None) == -2
    lib.bpdq_clear_status()


# ------------------------------------------------------------------ decaying states

def scan_oracle(q, k, v, decay, dt, skip, state, groups):
    T, H, V = v.shape
    s, o = state.astype(np.float64), np.empty((T, H, V))
    for t in range(T):
        for h in range(H):
            g = h // (H // groups)
            s[h], o[t, h] = ho.decayed_recurrence(s[h], decay[t, h], dt[t, h] * k[t, g].astype(np.float64), v[t, h], q[t, g])
            o[t, h] += skip[h] * v[t, h]
    return o, s


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("ssm", [0, 1])
@pytest.mark.parametrize("T,H,G,N,V", [(1, 3, 1, 16, 16), (2, 4, 2, 48, 80), (23, 2, 2, 80, 48), (24, 4, 1, 16, 32), (63, 2, 1, 128, 64),
                                       (64, 3, 3, 64, 144), (65, 2, 2, 144, 64), (130, 2, 1, 256, 32), (200, 6, 3, 32, 16)])
def test_decayed_scan(lib, bf16, ssm, T, H, G, N, V):
    act, rng = Act(bf16), np.random.default_rng(100 * T + N)
    if not ssm:
        G = H
    q, k, v = (act.host(rng.standard_normal(s) / np.sqrt(s[-1])) for s in ((T, G, N), (T, G, N), (T, H, V)))
    v *= 8
    state = rng.standard_normal((H, N, V)).astype(np.float32)
    if T > 2:
        k[1] *= 16          # one early key and one late query that match: the far term stands out
        q[T - 1] = k[1]
    skip = rng.standard_normal(H).astype(np.float32) if ssm else np.zeros(H, np.float32)
    if ssm:
        dt = (0.001 + 0.2 * rng.random((T, H)) ** 3).astype(np.float32)
        dt[T // 2] = 6.0                              # a step that forgets nearly everything
        rate = -np.linspace(0.1, 3.0, H).astype(np.float32)
        decay = np.exp(rate.astype(np.float64) * dt)
    else:
        dt = np.ones((T, H), np.float32)
        fixed = np.linspace(0.7, 1.0, H).astype(np.float32)
        decay = np.tile(fixed.astype(np.float64), (T, 1))
    want, want_s = scan_oracle(q, k, v, decay, dt, skip, state, G)
    dq, dk, dv, ds, do = act.up(lib, q), act.up(lib, k), act.up(lib, v), Dev(lib, state), act.empty(lib, T * H * V)
    if ssm:
        ddt, drate, dskip = Dev(lib, dt), Dev(lib, rate), Dev(lib, skip)
        tail = (None, None, ddt.ptr, drate.ptr, dskip.ptr)
    else:
        dfix, dlog = Dev(lib, fixed), Dev(lib, np.log(fixed.astype(np.float64)).astype(np.float32))
        tail = (dfix.ptr, dlog.ptr, None, None, None)
    done(lib, lib.bpd_decayed_scan_cuda(dq.ptr, G * N, dk.ptr, G * N, dv.ptr, H * V, *tail, ds.ptr, do.ptr, H * V, T, H, G, N, V, bf16, None))
    got, got_s = act.read(do).reshape(want.shape), ds.read(np.float32).reshape(want_s.shape)
    for h in range(H):
        assert normwise(got[:, h], want[:, h]) < act.tol, h
        # nothing of the recurrence is rounded to bf16: the state is exact to 16 bits of its inputs' products
        assert normwise(got_s[h], want_s[h]) < (3e-5 if bf16 else 2e-6), h


@pytest.mark.parametrize("bf16", ACTS)
def test_rotate_half(lib, bf16):
    act, rng = Act(bf16), np.random.default_rng(2)
    T, H, D, pos = 5, 3, 48, 1000
    for dims in (48, 20, 2):
        q, k = act.host(rng.standard_normal((T, H, D))), act.host(rng.standard_normal((T, H, D)))
        both = np.concatenate([q.reshape(T, -1), k.reshape(T, -1)], 1)
        d, dp, df = act.up(lib, both), Dev(lib, np.array([pos], np.int32)), Dev(lib, hybrid.rotary_frequencies(dims, 700.0))
        size = 2 if bf16 else 4
        done(lib, lib.bpd_rotate_half_qk_cuda(d.ptr, d.ptr + H * D * size, 2 * H * D, T, H, D, dims, df.ptr, 0.25, dp.ptr, bf16, None))
        got = act.read(d).reshape(T, 2, H, D)
        for t in range(T):
            assert normwise(got[t, 0], ho.rotate_half(q[t].astype(np.float64), pos + t, 700.0, dims)) < (5e-3 if bf16 else 1e-4)
            assert normwise(got[t, 1], 0.25 * ho.rotate_half(k[t].astype(np.float64), pos + t, 700.0, dims)) < (5e-3 if bf16 else 1e-4)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_causal_conv(lib, bf16, taps):
    act, rng = Act(bf16), np.random.default_rng(taps)
    ch = 150
    w, b = rng.standard_normal((ch, taps)).astype(np.float32), rng.standard_normal(ch).astype(np.float32)
    x, tail = act.host(rng.standard_normal((110, ch))), act.host(rng.standard_normal((max(1, taps - 1), ch)))
    hist = np.concatenate([tail[:taps - 1], x]).astype(np.float64)
    want = np.array([ho.silu(ho.causal_conv(hist[t:t + taps], w, b)) for t in range(110)])
    dw, db, dt = Dev(lib, np.ascontiguousarray(w.T)), Dev(lib, b), Dev(lib, tail)
    at = 0
    for n in (1, 2, 33, 3, 1, 70):                    # every portion starts from the window the last one left
        dx, do = act.up(lib, x[at:at + n]), act.empty(lib, n * ch)
        done(lib, lib.bpd_causal_conv_silu_cuda(dx.ptr, ch, do.ptr, n, ch, taps, dw.ptr, db.ptr, dt.ptr, bf16, None))
        assert normwise(act.read(do).reshape(n, ch), want[at:at + n]) < act.tol, (at, n)
        at += n
    if taps > 1:
        assert np.array_equal(dt.read(np.float32).reshape(taps - 1, ch), x[110 - (taps - 1):])


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("heads,V,parts,first", [(40, 16, 40, 0), (40, 16, 10, 1), (24, 320, 24, 0), (80, 32, 1, 1), (3, 40, 3, 0), (1, 16, 1, 0), (6, 24, 4, 1), (4, 32, 1, 1), (2, 5000, 2, 1), (2, 2500, 2, 0)])
def test_gated_norm(lib, bf16, heads, V, parts, first):
    act, rng = Act(bf16), np.random.default_rng(V)
    T, Vp, eps = 3, pad16(V), 0.01
    o, g = act.host(0.1 * rng.standard_normal((T, heads, V))), act.host(rng.standard_normal((T, heads, V)))
    w = (1 + 0.3 * rng.standard_normal((heads, V))).astype(np.float32)
    o64, s = o.astype(np.float64).reshape(T, -1), ho.silu(g.astype(np.float64)).reshape(T, -1)
    if first:
        want = ho.rms((o64 * s).reshape(T, parts, -1), eps).reshape(T, -1) * w.reshape(-1)
    else:
        want = ho.rms(o64.reshape(T, parts, -1), eps).reshape(T, -1) * s

    def pad(x):
        return np.pad(x, [(0, 0)] * (x.ndim - 1) + [(0, Vp - V)])
    do, dg, dw, dy = act.up(lib, pad(o)), act.up(lib, pad(g)), Dev(lib, pad(w)), act.empty(lib, T * heads * Vp)
    ld = heads * Vp
    done(lib, lib.bpd_gated_norm_cuda(do.ptr, ld, dg.ptr, ld, dw.ptr, dy.ptr, ld, T, heads, V, Vp, parts, first, eps, bf16, None))
    got = act.read(dy).reshape(T, heads, Vp)
    assert not got[:, :, V:].any() and normwise(got[:, :, :V].reshape(T, -1), want) < act.tol


# ------------------------------------------------------------------ latent attention

def latent_case(lib, bf16, T, pos, H, D, r, V, R, seed, stand_out=True):
    act, rng = Act(bf16), np.random.default_rng(seed)
    Dp, rp, Vp, Rp = pad16(D), pad16(r), pad16(V), pad16(R)
    L, base, scale = pos + T, 400.0, 0.4 / np.sqrt(D)
    c, kr = act.host(rng.standard_normal((L, R))), act.host(rng.standard_normal((L, r)))
    q = act.host(rng.standard_normal((T, H, D + r)))
    uk, uv = hm.bf16_round(rng.standard_normal((H, D, R)) / np.sqrt(R)), hm.bf16_round(rng.standard_normal((H, V, R)) / np.sqrt(R))
    special, shown = {}, 0
    if stand_out:       # for some (query, head) one key carries nearly all the weight: near, far, at block edges, its own
        spots = sorted({0, 1, 31, 32, 63, 64, 65, 127, 128, pos - 1, pos, L - 1} & set(range(L)))
        c[spots] = act.host(2 * c[spots])
        for i, s in enumerate(spots):
            t = max(0, min(T - 1, s - pos + (i % 3)))
            h = i % H
            if (t, h) not in special and s <= pos + t:
                special[(t, h)] = s
                key = uk[h].astype(np.float64) @ c[s]
                q[t, h, :D] = act.host(key * (30.0 / scale / (key @ key)))
    cache = np.full((L + 70, Rp + rp), np.nan, np.float32)          # rows that are not there yet must not be read
    cache[:L, :] = 0
    cache[:L, :R], cache[:L, Rp:Rp + r] = c, kr
    qs = np.zeros((T, H, Dp + rp), np.float32)
    qs[:, :, :D], qs[:, :, Dp:Dp + r] = q[:, :, :D], q[:, :, D:]
    ukv = np.zeros((H * Dp + H * Vp, Rp), np.float32)
    ukv[:H * Dp].reshape(H, Dp, Rp)[:, :D, :R] = uk
    ukv[H * Dp:].reshape(H, Vp, Rp)[:, :V, :R] = uv
    c64, kr64 = c.astype(np.float64), kr.astype(np.float64)
    want = np.empty((T, H, V))
    for h in range(H):
        k, v = c64 @ uk[h].T, c64 @ uv[h].T
        for t in range(T):
            n = pos + t + 1
            qr = ho.rotate_interleaved(q[t, h, D:].astype(np.float64), pos + t, base, r)
            s = (k[:n] @ q[t, h, :D].astype(np.float64) + kr64[:n] @ qr) * scale
            e = np.exp(s - s.max())
            want[t, h] = e / e.sum() @ v[:n]
            if (t, h) in special:
                shown += e[special[(t, h)]] / e.sum() > 0.5
    assert shown >= len(special) / 2
    freq = Dev(lib, hybrid.rotary_frequencies(r, base))
    shape = capi.LatentShape(H, Dp, Vp, R, Rp, r, rp, 16, 16, scale, 1e-6, freq.ptr)
    bits = hm.bf16_bits(np.where(np.isnan(cache), 0, cache))
    if bf16:
        bits[np.isnan(cache)] = 0x7FC0
    dq, dc, dw = act.up(lib, qs), Dev(lib, bits) if bf16 else Dev(lib, cache), Dev(lib, hm.bf16_bits(ukv))
    do, dp = act.empty(lib, T * H * Vp), Dev(lib, np.array([pos], np.int32))
    done(lib, lib.bpd_latent_attention_cuda(C.byref(shape), dq.ptr, dw.ptr, dc.ptr, do.ptr, dp.ptr, T, L, bf16, None))
    got = act.read(do).reshape(T, H, Vp)
    assert not got[:, :, V:].any()
    for h in range(H):
        for t in range(T):
            assert normwise(got[t, h, :V], want[t, h]) < (2.5e-2 if bf16 else 2e-5), (t, h, special.get((t, h)))


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,pos", [(1, 0), (1, 63), (1, 64), (1, 700), (2, 127), (5, 0), (16, 60), (70, 0), (70, 58), (130, 0), (200, 65)])
def test_latent_attention(lib, bf16, T, pos):
    latent_case(lib, bf16, T, pos, 3, 24, 6, 40, 40, T + pos)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("T,pos,H,D,r,V,R", [(1, 300, 1, 16, 2, 16, 16), (1, 130, 20, 64, 32, 48, 208), (3, 90, 16, 40, 10, 72, 500),
                                             (1, 200, 33, 16, 16, 16, 640), (130, 40, 2, 128, 64, 136, 96), (140, 0, 1, 16, 16, 272, 32),
                                             (1, 100, 2, 16, 16, 16, 1000)])
def test_latent_attention_sizes(lib, bf16, T, pos, H, D, r, V, R):
    latent_case(lib, bf16, T, pos, H, D, r, V, R, R)


@pytest.mark.parametrize("bf16", ACTS)
@pytest.mark.parametrize("Q,R,r", [(300, 40, 6), (2048, 1000, 64), (2100, 40, 16), (40, 1100, 2)])
def test_latent_prepare(lib, bf16, Q, R, r):
    act, rng = Act(bf16), np.random.default_rng(8)
    T, pos = 4, 37
    Qp, Rp, rp = pad16(Q), pad16(R), pad16(r)
    u = act.host(rng.standard_normal((T, Q + R + r)) * 0.05)
    us = np.zeros((T, Qp + Rp + rp), np.float32)
    us[:, :Q], us[:, Qp:Qp + R], us[:, Qp + Rp:Qp + Rp + r] = u[:, :Q], u[:, Q:Q + R], u[:, Q + R:]
    qn, kn = (np.pad(1 + 0.3 * rng.standard_normal(n), (0, pad16(n) - n)).astype(np.float32) for n in (Q, R))
    eps, freq = 1e-2, Dev(lib, hybrid.rotary_frequencies(r, 90.0))
    shape = capi.LatentShape(1, 16, 16, R, Rp, r, rp, Q, Qp, 1.0, eps, freq.ptr)
    du, dqn, dkn, dcq = act.up(lib, us), Dev(lib, qn), Dev(lib, kn), act.empty(lib, T * Qp)
    row = Rp + rp
    dc, dp = act.empty(lib, 64 * row), Dev(lib, np.array([pos], np.int32))
    done(lib, lib.bpd_latent_prepare_cuda(C.byref(shape), du.ptr, Qp + Rp + rp, dqn.ptr, dkn.ptr, dcq.ptr, dc.ptr, dp.ptr, T, bf16, None))
    u64 = u.astype(np.float64)
    cq, cache = act.read(dcq).reshape(T, Qp), act.read(dc).reshape(64, row)
    assert normwise(cq[:, :Q], ho.rms(u64[:, :Q], eps) * qn[:Q]) < act.tol and not cq[:, Q:].any()
    mine = cache[pos:pos + T]
    assert normwise(mine[:, :R], ho.rms(u64[:, Q:Q + R], eps) * kn[:R]) < act.tol
    for t in range(T):
        assert normwise(mine[t, Rp:Rp + r], ho.rotate_interleaved(u64[t, Q + R:], pos + t, 90.0, r)) < max(act.tol, 1e-5)
    assert not mine[:, R:Rp].any() and not mine[:, Rp + r:].any()
    assert np.isnan(cache[:pos]).all() and np.isnan(cache[pos + T:]).all()      # nobody else's rows


# ------------------------------------------------------------------ whole models

LIMIT = {"float32": 2e-5, "bfloat16": 6e-2}


@pytest.fixture(scope="module", params=list(hm.CONFIGS))
def case(request):
    cfg = hm.CONFIGS[request.param]
    w = hm.weights(cfg, 11)
    toks = hm.tokens(cfg, 150, 4)
    logits, res = ho.Model(cfg, w).run(toks)
    return cfg, w, toks, logits, res


def device(cfg, w, lib, dtype, capacity=256, **kw):
    return hybrid.DeviceHybrid(hybrid.HybridSpec(cfg), hybrid.ArrayTensors(w), dtype=dtype, capacity=capacity, lib=lib, **kw)


def feed_portions(e, key, toks, sizes):
    out, at = [], 0
    for n in sizes:
        lg, picked = e.feed(key, toks[at:at + n], range(n))
        assert np.array_equal(picked, lg.argmax(1))
        out.append(lg)
        at += n
    assert at == len(toks)
    e.end(key)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_residual_stream_layer_by_layer(lib, case, dtype):
    cfg, w, toks, _, res = case
    m = device(cfg, w, lib, dtype)
    e = Engine(m)
    seq = e.slots.acquire()
    got = m.residuals(seq, toks[:90])
    for i in range(len(cfg["layers"])):
        assert np.max(hm.row_errors(got[i], res[i][:90])) < (1e-5 if dtype == "float32" else 4e-2), i
    e.slots.release(seq)
    seq = e.slots.acquire()
    got = np.concatenate([m.residuals(seq, [t]) for t in toks[:20]], 1)
    for i in range(len(cfg["layers"])):
        assert np.max(hm.row_errors(got[i], res[i][:20])) < (1e-5 if dtype == "float32" else 4e-2), i
    e.close()
    m.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_prompt_portions_and_decoding(lib, case, dtype):
    """The logits of every position, however the sequence is cut; one slot, used again by every run."""
    cfg, w, toks, want, _ = case
    m = device(cfg, w, lib, dtype)
    e = Engine(m)
    for sizes in ([150], [1] * 150, [118] + [1] * 32, [2] * 75, [33, 2, 37, 14, 22, 3, 1, 1, 37], [64, 64, 22], [65, 1, 63, 1, 20], [70, 80],
                  [1, 149], [149, 1]):
        err = hm.row_errors(feed_portions(e, "r", toks, sizes), want)
        assert np.max(err) < LIMIT[dtype], (sizes[:4], int(np.argmax(err)), float(np.max(err)))
    assert m.lib.bpdq_last_status() == 0
    e.close()
    m.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_interleaved_requests_equal_each_alone(lib, dtype):
    """Live requests in several slots, steps taken in turn, slots given back and used again; recorded one-token steps
    and launch-by-launch ones give the same bits."""
    cfg = hm.CONFIGS["mixed"]
    w = hm.weights(cfg, 21)
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
    cfg = hm.CONFIGS["square"]
    w, toks = hm.weights(cfg, 5), hm.tokens(cfg, 420, 6)
    want, _ = ho.Model(cfg, w).run(toks)
    m = device(cfg, w, lib, dtype, capacity=420)
    e = Engine(m)
    got = feed_portions(e, 0, toks, [20] + [1] * 400)
    assert np.max(hm.row_errors(got, want)) < LIMIT[dtype]
    with pytest.raises(ValueError, match="room for 420"):
        e.feed(1, toks[:400])
        e.feed(1, toks[:21])
    with pytest.raises(ValueError, match="token ids"):
        e.end(1)
        e.feed(2, [cfg["vocab"]])
    e.close()
    m.close()


def far_key_case():
    cfg = hm.config(64, 48, [hm.layer("latent_attention", hm.latent(2, 32, 4, 32, 48, 48, 1.0))])
    w, p = hm.weights(cfg, 9), "l0.mix."
    w[p + "dq"], w[p + "dq.norm"] = w[p + "dkv"][:48], w[p + "dkv.norm"]         # query latent = key latent
    w64 = {k: v.astype(np.float64) for k, v in w.items()}

    def latent(tok):
        h = ho.dynamic_tanh(w64["embed"][tok], w64, "l0.norm1")
        return ho.rms(w64[p + "dq"] @ h, cfg["norm"]["eps"]) * w64[p + "dq.norm"]
    uq, c = np.zeros((2, 36, 48)), latent(61)
    for head in range(2):
        key = w64[p + "uk"].reshape(2, 32, 48)[head] @ latent(62)
        uq[head, :32] = np.outer(key, c) * (24.0 / (key @ key) / (c @ c))
    w[p + "uq"] = hm.bf16_round(uq.reshape(72, 48))
    toks = np.random.default_rng(0).integers(1, 60, 330).tolist()
    toks[3], toks[329] = 62, 61
    return cfg, w, toks


def test_a_far_key_shows_through_the_whole_model(lib):
    """A single attention layer in which one token's query looks for another token's key, hundreds of keys away: in prompts
    and in decoding."""
    cfg, w, toks = far_key_case()
    want, _ = ho.Model(cfg, w).run(toks)
    other = list(toks)
    other[3] = 63
    blind, _ = ho.Model(cfg, w).run(other)
    assert hm.row_errors(want[329:], blind[329:])[0] > 0.1           # the far token matters
    for dtype in LIMIT:
        m = device(cfg, w, lib, dtype, capacity=330)
        e = Engine(m)
        for sizes in ([330], [329, 1], [100] + [1] * 230):
            err = hm.row_errors(feed_portions(e, 0, toks, sizes), want)
            assert np.max(err) < (1e-4 if dtype == "float32" else 0.15), (dtype, sizes[:2])
        e.close()
        m.close()


def save_model(folder, cfg, w):
    (folder / "config.json").write_text(json.dumps(cfg))
    safetensors_load.save_bf16(str(folder / "model.safetensors"), {k: np.asarray(v, np.float32) for k, v in w.items()})


def test_greedy_generation_through_the_command_line(lib, tmp_path, capsys):
    cfg = hm.CONFIGS["mixed"]
    w = hm.weights(cfg, 31)
    save_model(tmp_path, cfg, w)
    prompts = [hm.tokens(cfg, n, n) for n in (3, 40, 1, 17)]
    args = ["--model", str(tmp_path), "--max-new", "12", "--dtype", "float32", "--capacity", "64", "--slots", "2", "--portion", "16"]
    for p in prompts:
        args += ["--prompt", " ".join(map(str, p))]
    assert generate.main(args) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.splitlines()]
    ref = ho.Model(cfg, w)
    assert [x["prompt"] for x in lines] == prompts
    assert [x["output"] for x in lines] == [ref.greedy(p, 12) for p in prompts]


def test_trace_replay_from_a_folder(lib, tmp_path, monkeypatch):
    cfg = hm.CONFIGS["conv1"]
    w = hm.weights(cfg, 41)
    save_model(tmp_path, cfg, w)
    toks = hm.tokens(cfg, 30, 3)
    want, _ = ho.Model(cfg, w).run(toks)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": toks[:20], "want": [4, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": toks[20:], "want": [9]}], "end": ["q"]},
             {"step": 2, "entries": [{"id": "p", "tokens": toks[:1], "want": [0]}], "end": ["p"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "30"]) == 0
    for i, rows in enumerate(([4, 19], [29], [0])):
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(len(rows), cfg["vocab"])
        assert np.max(hm.row_errors(got, want[rows])) < 2e-5


def test_the_llama_family_runs_in_the_same_engine(lib):
    """Greedy generation of the Q8_0 Llama through the engine equals its own forward, two sequences taking turns."""
    from bpd_substrate_b200 import llama
    cfg = llama.make_config(n_layers=2, n_heads=4, n_kv_heads=2, head_dim=32, ffn_dim=256, vocab_size=96, max_seq_len=48)
    dev = llama.DeviceLlama(llama.SyntheticLlama(cfg, seed=3), lib)
    prompts, n = [[5, 9, 33, 2], [7]], 6
    want = []
    for p in prompts:
        dev.reset_cache()
        toks, kv, out = list(p), 0, []
        while len(out) < n:
            _, ids = dev.forward(toks, np.arange(kv, kv + len(toks), dtype=np.int32), kv)
            kv += len(toks)
            out.append(int(ids[-1]))
            toks = [out[-1]]
        want.append(out)
    e = Engine(dev, slots=2, portion=3)
    assert e.generate(prompts, n) == want
    e.close()
    dev.close()
