"""Host side of the hybrid decoder and of generation, without a GPU: configuration checks, weight packing, checkpoint files,
sequence slots, the engine's scheduling, trace replay, registry, and the oracle against closed forms."""
import ctypes as C
import io
import json
import os

import numpy as np
import pytest

from bpd_substrate_b200 import capi, hybrid, registry, safetensors_load, trace
from bpd_substrate_b200.engine import Engine, Request
from bpd_substrate_b200.sequences import ALIGN, SequenceSlots, StatePart, lay_out
from oracle import hybrid_oracle as ho
from tests import hybrid_models as hm


# ------------------------------------------------------------------ oracle

def test_oracle_retention_equals_the_sum_over_earlier_tokens():
    rng = np.random.default_rng(0)
    T, D, V, decay = 9, 6, 5, 0.8
    q, k, v = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, V))
    s = np.zeros((D, V))
    for t in range(T):
        s, o = ho.decayed_recurrence(s, decay, k[t], v[t], q[t])
        want = sum(decay ** (t - j) * (q[t] @ k[j]) * v[j] for j in range(t + 1))
        assert np.allclose(o, want, atol=1e-12)


def test_oracle_rotations_depend_on_the_distance_only():
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal(10), rng.standard_normal(10)
    for rot in (ho.rotate_half, ho.rotate_interleaved):
        a = rot(q, 7, 50.0, 8) @ rot(k, 4, 50.0, 8)
        b = rot(q, 103, 50.0, 8) @ rot(k, 100, 50.0, 8)
        assert abs(a - b) < 1e-10 and abs(a - q @ k) > 1e-3
        assert np.array_equal(rot(q, 5, 50.0, 8)[8:], q[8:]) and np.array_equal(rot(q, 0, 50.0, 8), q)


def test_oracle_convolution_is_a_dot_product_with_the_newest_tap_last():
    x, taps = np.arange(12, dtype=float).reshape(4, 3), np.array([[1, 10], [2, 20], [3, 30]], float)
    assert np.array_equal(ho.causal_conv(x[1:3], taps, np.array([0.5, 0, 0])), taps[:, 0] * x[1] + taps[:, 1] * x[2] + [0.5, 0, 0])


# ------------------------------------------------------------------ configuration and packing

@pytest.mark.parametrize("name", list(hm.CONFIGS))
def test_tensor_shapes(name):
    cfg = hm.CONFIGS[name]
    want = {k: v.shape for k, v in hm.weights(cfg).items()}
    assert hybrid.HybridSpec(cfg).tensor_shapes() == want


def test_rejected_configurations():
    def bad(change):
        cfg = json.loads(json.dumps(hm.CONFIGS["mixed"]))
        change(cfg)
        with pytest.raises((ValueError, KeyError)):
            hybrid.HybridSpec(cfg)
    bad(lambda c: c.update(architecture="Other"))
    bad(lambda c: c.update(width=0))
    bad(lambda c: c["layers"][0].update(type="window"))
    bad(lambda c: c["layers"][0]["mlp"].update(kind="experts"))
    bad(lambda c: c["layers"][1]["mixer"].update(groups=4))
    bad(lambda c: c["layers"][1]["mixer"].update(norm_groups=5))
    bad(lambda c: c["layers"][2]["mixer"].update(decay=[0.5]))
    bad(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=50))
    bad(lambda c: c["layers"][3]["mixer"].update(kv_from=1))       # not latent attention
    bad(lambda c: c["layers"][3]["mixer"].update(kv_from=4))       # later
    bad(lambda c: c["layers"][3]["mixer"].update(kv_rank=48))      # other latents
    bad(lambda c: c["layers"][3]["mixer"]["rot"].update(base=1.0))


def test_packed_products_equal_the_tensors():
    """The padded, stacked and interleaved matrices give the same products, zeros at the pads."""
    cfg = hm.CONFIGS["mixed"]
    spec, w = hybrid.HybridSpec(cfg), hm.weights(cfg, 3)
    get = hybrid.ArrayTensors(w)
    h = np.random.default_rng(0).standard_normal(spec.width)
    hp = np.zeros(spec.width_pad)
    hp[:spec.width] = h
    f = hm.bits_f32
    # latent attention: layer 0
    pk, m = hybrid.pack_layer(spec, 0, get), cfg["layers"][0]["mixer"]
    u = f(pk.mats["w_in"]) @ hp
    qp, rp, pp = pk.ints["q_rank_pad"], pk.ints["kv_rank_pad"], pk.ints["rot_pad"]
    assert (qp, rp, pp) == (64, 48, 16) and u.size == qp + rp + pp
    assert np.allclose(u[:56], w["l0.mix.dq"] @ h) and not u[56:64].any()
    kv = w["l0.mix.dkv"] @ h
    assert np.allclose(u[64:104], kv[:40]) and np.allclose(u[112:118], kv[40:]) and not u[118:].any()
    c = np.random.default_rng(1).standard_normal(56)
    q = (f(pk.mats["w_uq"]) @ np.pad(c, (0, 8))).reshape(3, 32 + 16)
    want = (w["l0.mix.uq"] @ c).reshape(3, 30)
    assert np.allclose(q[:, :24], want[:, :24]) and np.allclose(q[:, 32:38], want[:, 24:]) and not q[:, 24:32].any()
    # state space: layer 1, heads of 24 values (32 stored), 3 groups of 20 (32 stored)
    pk = hybrid.pack_layer(spec, 1, get)
    u, want = f(pk.mats["w_in"]) @ hp, w["l1.mix.in"] @ h
    assert u.size == 2 * 6 * 32 + 2 * 3 * 32 + 6
    assert np.allclose(u[:192].reshape(6, 32)[:, :24].ravel(), want[:144])
    assert np.allclose(u[192:384].reshape(6, 32)[:, :24].ravel(), want[144:288])
    assert np.allclose(u[384:480].reshape(3, 32)[:, :20].ravel(), want[288:348])
    assert np.allclose(u[480:576].reshape(3, 32)[:, :20].ravel(), want[348:408]) and np.allclose(u[576:], want[408:])
    assert pk.vecs["conv_w"].shape == (4, 384) and np.array_equal(pk.vecs["conv_w"][:, 192:212], w["l1.mix.conv"][144:164].T)
    y = np.random.default_rng(2).standard_normal((6, 24))
    o = f(pk.mats["w_o"]) @ np.pad(y, ((0, 0), (0, 8))).ravel()
    assert np.allclose(o[:72], w["l1.mix.o"] @ y.ravel()) and not o[72:].any()
    # feed-forward of layer 0: gate and up rows alternate
    pk = hybrid.pack_layer(spec, 0, get)
    gu = f(pk.mats["w_gate_up"]) @ hp
    assert np.allclose(gu[0:176:2], w["l0.mlp.gate"] @ h) and np.allclose(gu[1:176:2], w["l0.mlp.up"] @ h)


def test_struct_layout_matches_the_header():
    """ctypes mirrors of the descriptor structs against a compiler's view of the header."""
    import shutil
    import subprocess
    import tempfile
    if not shutil.which("gcc"):
        pytest.skip("no C compiler")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    src = ('#include <stdio.h>\n#include <stddef.h>\n#include <stdint.h>\n#include "bpdq.h"\nint main(void){printf("%zu %zu %zu %zu %zu",'
           "sizeof(bpdq_hybrid_layer),sizeof(bpdq_hybrid_config),sizeof(bpdq_latent_shape),offsetof(bpdq_hybrid_layer,norm1),"
           "offsetof(bpdq_hybrid_layer,state_offset));return 0;}")
    with tempfile.TemporaryDirectory() as d:
        with open(os.path.join(d, "a.c"), "w") as f:
            f.write(src)
        subprocess.check_call(["gcc", "-I", os.path.join(root, "include"), os.path.join(d, "a.c"), "-o", os.path.join(d, "a")])
        got = subprocess.check_output([os.path.join(d, "a")], text=True).split()
    want = [C.sizeof(capi.HybridLayer), C.sizeof(capi.HybridConfig), C.sizeof(capi.LatentShape), capi.HybridLayer.norm1.offset,
            capi.HybridLayer.state_offset.offset]
    assert [int(v) for v in got] == want


# ------------------------------------------------------------------ checkpoint files, registry

def test_safetensors_round_trip(tmp_path):
    path = str(tmp_path / "m.safetensors")
    a = hm.bf16_round(np.random.default_rng(0).standard_normal((3, 5)))
    safetensors_load.save_bf16(path, {"a": a, "s": np.float32(0.5), "t": np.arange(4, dtype=np.int32)})
    f = safetensors_load.SafetensorsFile(path)
    assert np.array_equal(f.f32("a"), a) and f.f32("s").shape == () and float(f.f32("s")) == 0.5
    assert np.array_equal(f.raw("t"), [0, 1, 2, 3]) and f.bf16("a").dtype == np.uint16 and "b" not in f
    with pytest.raises(KeyError):
        f.raw("b")
    f.close()
    data = open(path, "rb").read()
    with open(path, "wb") as g:
        g.write(data[:-3])
    with pytest.raises(ValueError):
        safetensors_load.SafetensorsFile(path)


def test_registry(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ValueError, match="Nothing"):
        registry.load_model(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps(hm.CONFIGS["conv1"]))
    assert registry.architecture_of(str(tmp_path)) == "Gurusun" and registry.architecture_of("x.gguf") == "llama"
    with pytest.raises(ValueError):
        registry.architecture_of("x.bin")


# ------------------------------------------------------------------ slots and engine, on a fake device

class FakeLib:
    def __init__(self):
        self.cleared = []

    def bpdq_alloc(self, n):
        self.block = n
        return 1 << 20

    def bpdq_free(self, p):
        assert p == 1 << 20

    def bpdq_memset_async(self, p, value, n, stream):
        self.cleared.append((p, value, n))
        return 0


class FakeModel:
    """Next token = (sum of the sequence so far) mod vocab; keeps what a slot was fed to check the scheduling."""
    vocab, stream = 50, None

    def __init__(self, capacity=64):
        self.lib, self.capacity, self.steps, self.sums = FakeLib(), capacity, [], {}

    def state_parts(self):
        return [StatePart("cache", 10, rows=True, zero=False), StatePart("s", 100)]

    def step(self, seq, tokens, want, logits=True):
        if seq.length == 0:
            self.sums[seq.slot] = []
        assert seq.length == len(self.sums[seq.slot])
        self.steps.append((seq.slot, len(tokens)))
        self.sums[seq.slot] += [int(t) for t in tokens]
        base = seq.length
        seq.length += len(tokens)
        picked = np.array([sum(self.sums[seq.slot][:base + w + 1]) % self.vocab for w in want], np.int64)
        return (np.eye(self.vocab, dtype=np.float32)[picked] if logits else None), picked


def expected_output(prompt, n, vocab=50):
    seq = list(prompt)
    for _ in range(n):
        seq.append(sum(seq) % vocab)
    return seq[len(prompt):]


def test_slots_are_cleared_and_used_again():
    m = FakeModel()
    lay = lay_out(m.state_parts(), 64)
    assert lay.offsets["s"] == 0 and lay.offsets["cache"] == ALIGN and lay.slot_bytes == ALIGN + 768
    s = SequenceSlots(m.lib, m.state_parts(), 64, 2)
    a, b = s.acquire(), s.acquire()
    assert s.acquire() is None and b.base - a.base == lay.slot_bytes
    s.release(a)
    with pytest.raises(ValueError):
        s.release(a)
    c = s.acquire()
    assert c.base == m.lib.cleared[0][0] and c.length == 0
    assert m.lib.cleared == [(p.base, 0, ALIGN) for p in (c, b, c)]       # the cache rows are not cleared
    s.close()


@pytest.mark.parametrize("slots,portion", [(1, 4), (2, 3), (3, 100)])
def test_engine_generates_every_request(slots, portion):
    m = FakeModel()
    e = Engine(m, slots, portion)
    prompts = [[3, 4, 5, 6, 7, 8, 9], [1], [2, 2], [9] * 12, [7, 1, 1]]
    assert e.generate(prompts, 6) == [expected_output(p, 6) for p in prompts]
    assert not e.live and len(e.slots.free) == slots
    assert max(n for _, n in m.steps) <= portion
    if slots > 1:
        assert any(m.steps[i][0] != m.steps[i + 1][0] for i in range(len(m.steps) - 1))      # live requests take turns


def test_engine_stops_and_checks_sizes():
    e = Engine(FakeModel(capacity=10), 1, 4)
    out = expected_output([5, 6], 8)
    assert e.generate([[5, 6]], 8, stop=[out[2]]) == [out[:3]]
    for r in (Request([], 3), Request([1], 0), Request([1] * 8, 4)):
        with pytest.raises(ValueError):
            e.run([r])
    e.feed("a", [1, 2])
    with pytest.raises(RuntimeError):
        e.feed("b", [1])
    with pytest.raises(ValueError):
        e.feed("a", [1], [1])


def test_trace_replay(tmp_path):
    e = Engine(FakeModel(), 1, 4)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": [1, 2, 3, 4, 5, 6], "want": [0, 3, 5]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": [7, 8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": [9], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": [2], "want": [0]}], "end": ["y"]}]
    said = []
    trace.replay(e, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32", "3.f32"]
    got = np.fromfile(tmp_path / "0.f32", "<f4").reshape(3, 50).argmax(1)
    assert got.tolist() == [1, 10, 21] and np.fromfile(tmp_path / "2.f32", "<f4").argmax() == 45
    assert np.fromfile(tmp_path / "3.f32", "<f4").argmax() == 2 and not e.live
