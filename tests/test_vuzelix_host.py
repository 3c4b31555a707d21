"""Host side of the Vuzelix decoder, without a GPU: configuration checks, weight packing, caches with limited rows, registry, and the
oracle against closed forms."""
import ctypes as C
import json
import os
import shutil
import subprocess

import numpy as np
import pytest

from bpd_substrate_b200 import capi, hybrid, registry, vuzelix
from bpd_substrate_b200.engine import Engine
from bpd_substrate_b200.sequences import ALIGN, StatePart, lay_out
from oracle import vuzelix_oracle as vo
from tests import hybrid_models as hm
from tests import vuzelix_models as vm
from tests.test_hybrid_host import FakeModel, expected_output


# ------------------------------------------------------------------ oracle

def test_oracle_delta_step_stores_and_replaces():
    """With beta 1 and no decay a key reads back what was last written at it, and other directions are left alone."""
    rng = np.random.default_rng(0)
    D, V = 6, 4
    k1, k2 = np.linalg.qr(rng.standard_normal((D, 2)))[0].T
    v1, v2, v3 = rng.standard_normal((3, V))
    s, one = np.zeros((D, V)), np.ones(D)
    s, o = vo.delta_step(s, one, 1.0, k1, v1, k1)
    assert np.allclose(o, v1)
    s, _ = vo.delta_step(s, one, 1.0, k2, v2, k2)
    s, o = vo.delta_step(s, one, 1.0, k1, v3, k1)
    assert np.allclose(o, v3) and np.allclose(s.T @ k2, v2)
    s, o = vo.delta_step(s, one, 0.25, k1, v1, k1)
    assert np.allclose(o, 0.75 * v3 + 0.25 * v1)
    assert np.allclose(vo.delta_step(s, np.zeros(D), 1.0, k2, v1, k1)[1], 0)      # everything forgotten, nothing written at k1


def test_oracle_decays_act_on_key_channels():
    s = np.arange(12, dtype=float).reshape(3, 4)
    decay = np.array([1.0, 0.5, 0.0])
    got, o = vo.delta_step(s, decay, 0.0, np.ones(3), np.ones(4), np.array([0, 1.0, 0]))
    assert np.array_equal(got, s * decay[:, None]) and np.array_equal(o, 0.5 * s[1])


def test_oracle_attention_has_a_sink_and_a_cap():
    q, keys, values = np.array([2.0, 0]), np.array([[3.0, 1], [-50, 0]]), np.array([[1.0, 10], [2, 20]])
    a, b = np.exp(4 * np.tanh(3.0 / 4)), np.exp(4 * np.tanh(-50.0 / 4))
    assert np.allclose(vo.attend(q, keys, values, 0.5, 4.0), (a * values[0] + b * values[1]) / (1 + a + b))
    assert np.allclose(vo.attend(q, keys[:1], values[:1], 0.0, 4.0), values[0] / 2)         # a lone score of 0 shares with the sink


def test_oracle_chunks_are_counted_from_the_first_position():
    seen = [[j for j in range(10) if vo.sees(i, j, 4)] for i in (0, 3, 4, 7, 9)]
    assert seen == [[0], [0, 1, 2, 3], [4], [4, 5, 6, 7], [8, 9]]
    assert all(vo.sees(9, j, 0) for j in range(10)) and not vo.sees(3, 4, 0)


def test_oracle_streams_mix_from_row_to_column():
    x, y = np.array([[1.0, 2], [10, 20]]), np.array([100.0, 200])
    mix = np.array([[1.0, 2], [3, 4]])
    got = vo.write_streams(x, y, mix, np.array([1.0, -1]), 0.5)
    assert np.array_equal(got, [1 * x[0] + 3 * x[1] + 0.5 * y, 2 * x[0] + 4 * x[1] - 0.5 * y])
    assert np.array_equal(vo.read_streams(x, np.array([2.0, -1])), 2 * x[0] - x[1])


def test_oracle_elementwise():
    z = np.linspace(-4, 4, 9)
    assert np.allclose(vo.gelu_tanh(z) - vo.gelu_tanh(-z), z) and vo.gelu_tanh(np.array(0.0)) == 0
    assert np.allclose(vo.soft_cap(1e-4 * z, 5.0), 1e-4 * z) and np.all(np.abs(vo.soft_cap(1e3 * z, 5.0)) <= 5)
    assert abs(np.linalg.norm(vo.unit(np.arange(1.0, 9))) - 1) < 1e-6


# ------------------------------------------------------------------ configuration and packing

def spec_of(name, w=None):
    cfg = vm.CONFIGS[name]
    spec, get = vuzelix.VuzelixSpec(cfg), hybrid.ArrayTensors(w or vm.weights(cfg, 3))
    spec.read_shapes(get.shape)
    return spec, get


@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_tensor_shapes(name):
    spec, _ = spec_of(name)
    assert spec.tensor_shapes() == {k: v.shape for k, v in vm.weights(vm.CONFIGS[name]).items()}


def test_rejected_configurations():
    def bad(change):
        cfg = json.loads(json.dumps(vm.CONFIGS["mixed"]))
        change(cfg)
        with pytest.raises((ValueError, KeyError)):
            vuzelix.VuzelixSpec(cfg)
    bad(lambda c: c.update(architecture="Gurusun"))
    bad(lambda c: c.update(streams=0))
    bad(lambda c: c.update(streams=9))
    bad(lambda c: c.update(logit_softcap=0.0))
    bad(lambda c: c.pop("embedding"))
    bad(lambda c: c.pop("residual_mult"))
    bad(lambda c: c["layers"][0].update(type="mamba2"))
    bad(lambda c: c["layers"][0]["mlp"].update(kind="experts"))
    bad(lambda c: c["layers"][0]["mixer"].update(kv_heads=4))
    bad(lambda c: c["layers"][0]["mixer"].update(conv=0))
    bad(lambda c: c["layers"][1]["mixer"].update(softcap=-1.0))
    bad(lambda c: c["layers"][1]["mixer"]["mask"].update(size=0))
    bad(lambda c: c["layers"][2]["mixer"].update(kv_from=0))       # not attention
    bad(lambda c: c["layers"][2]["mixer"].update(kv_from=4))       # later
    bad(lambda c: c["layers"][2]["mixer"].update(vdim=24))         # other sizes
    bad(lambda c: c["layers"][4]["mixer"].update(kv_from=2))       # no keys of its own


def test_packed_delta_layer():
    """The padded and stacked matrices give the same products, zeros at the pads."""
    w = vm.weights(vm.CONFIGS["mixed"], 3)
    spec, get = spec_of("mixed", w)
    f, rng = hm.bits_f32, np.random.default_rng(0)
    h = rng.standard_normal(72)
    hp = np.pad(h, (0, 8))
    pk, p = spec.pack_layer(0, get), "l0.mix."              # 6 heads on 2 key heads, 24 keys (32 stored), 40 values (48 stored)
    u = f(pk.mats["w_in"]) @ hp
    a, g = spec.ranks[0]
    assert (a, g) == (w[p + "a1"].shape[0], w[p + "g1"].shape[0]) and a != g
    R = pk.ints["gate_rank_pad"]
    assert R == 32 and u.size == 2 * 2 * 32 + 6 * 48 + 2 * R + 6
    assert np.allclose(u[:64].reshape(2, 32)[:, :24].ravel(), w[p + "q"] @ h) and np.allclose(u[64:128].reshape(2, 32)[:, :24].ravel(), w[p + "k"] @ h)
    v = u[128:416].reshape(6, 48)
    assert np.allclose(v[:, :40].ravel(), w[p + "v"] @ h) and not v[:, 40:].any()
    low, gate = u[416:416 + R], u[416 + R:416 + 2 * R]
    assert np.allclose(low[:a], w[p + "a1"] @ h) and np.allclose(gate[:g], w[p + "g1"] @ h) and not low[a:].any() and not gate[g:].any()
    assert np.allclose(u[-6:], w[p + "b"] @ h)
    x = rng.standard_normal(R)
    both = f(pk.mats["w_gates"]) @ x
    assert np.allclose(both[:192].reshape(6, 32)[:, :24].ravel(), w[p + "a2"] @ x[:a]) and np.allclose(both[192:].reshape(6, 48)[:, :40].ravel(), w[p + "g2"] @ x[:g])
    assert pk.vecs["conv_w"].shape == (4, 416) and np.array_equal(pk.vecs["conv_w"][:, 128 + 48:128 + 88], w[p + "v.conv"][40:80].T)
    assert np.allclose(pk.vecs["neg_exp_a"].reshape(6, 32)[:, :24], np.repeat(-np.exp(w[p + "A_log"].astype(float))[:, None], 24, 1))
    assert np.array_equal(pk.vecs["norm_w"].reshape(6, 48)[:, :40], np.tile(w[p + "norm"], (6, 1)))
    y = rng.standard_normal((6, 40))
    o = f(pk.mats["w_o"]) @ np.pad(y, ((0, 0), (0, 8))).ravel()
    assert np.allclose(o[:72], w[p + "o"] @ y.ravel()) and not o[72:].any()
    assert pk.floats["scale"] == 24 ** -0.5


def test_packed_attention_layers_and_connections():
    w = vm.weights(vm.CONFIGS["mixed"], 3)
    spec, get = spec_of("mixed", w)
    f = hm.bits_f32
    own, lent = spec.pack_layer(1, get), spec.pack_layer(2, get)
    assert own.mats["w_in"].shape == ((6 + 3) * 32 + 3 * 32, 80) and lent.mats["w_in"].shape == (6 * 32, 80)
    assert (own.ints["kv_from"], lent.ints["kv_from"]) == (-1, 1) and (own.ints["chunk"], lent.ints["chunk"]) == (24, 40)
    assert (lent.floats["scale"], lent.floats["softcap"]) == (0.3, 25.0) and "ff_pad" not in own.ints
    assert lent.ints["ff_pad"] == 64 and lent.ints["ff_kind"] == capi.FF_GELU
    up, down = f(lent.mats["w_gate_up"]), f(lent.mats["w_down"])
    assert np.array_equal(up[:50, :72], w["l2.mlp.up"]) and not up[50:].any() and np.array_equal(down[:72, :50], w["l2.mlp.down"]) and not down[:, 50:].any()
    d = lent.mixes["mix2"]
    assert all(d.mix[s * capi.MAX_STREAMS + t] == w["l2.hc2.mix"][s, t] for s in range(2) for t in range(2))
    assert np.allclose(d.out[:2], 0.6 * w["l2.hc2.out"]) and np.allclose(d.in_[:2], w["l2.hc2.in"]) and d.out[2] == 0
    ends = spec.pack_ends(get)
    assert np.array_equal(f(ends.head)[:, :72], w["head"]) and ends.numbers == {"streams": 2, "embed_scale": 3.0, "logit_cap": 12.0}


def test_caches_hold_what_every_reader_can_still_see():
    spec, _ = spec_of("mixed")
    parts = {p.name: p for p in spec.state_parts(True)}
    assert set(parts) == {"l0.state", "l0.tail", "l1.cache", "l3.state", "l3.tail", "l4.cache"}       # layer 2 reads layer 1's
    assert parts["l1.cache"].limit == 40 + spec.portion and parts["l4.cache"].limit == 17 + spec.portion
    assert parts["l1.cache"].nbytes == 2 * 3 * 64 and parts["l0.state"].nbytes == 4 * 6 * 32 * 48 and parts["l0.tail"].nbytes == 4 * 3 * 416
    assert parts["l4.cache"].count(100) == 100 and parts["l4.cache"].count(10 ** 6) == 17 + spec.portion
    spec, _ = spec_of("wide")
    assert {p.name: p.limit for p in spec.state_parts(False) if p.rows} == {"l1.cache": 90 + spec.portion, "l2.cache": 33 + spec.portion, "l3.cache": 0}


def test_layout_of_limited_parts():
    parts = [StatePart("cache", 100, rows=True, zero=False, limit=10), StatePart("s", 8)]
    assert lay_out(parts, 50).slot_bytes == ALIGN + 4 * ALIGN and lay_out(parts, 5).slot_bytes == ALIGN + 2 * ALIGN


def test_engine_keeps_to_the_models_portion():
    m = FakeModel()
    m.portion = 3
    e = Engine(m, 2, 100)
    prompts = [[3, 4, 5, 6, 7, 8, 9], [1], [9] * 12]
    assert e.generate(prompts, 4) == [expected_output(p, 4) for p in prompts]
    assert max(n for _, n in m.steps) == 3


def test_struct_layout_matches_the_header(tmp_path):
    if not shutil.which("gcc"):
        pytest.skip("no C compiler")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    (tmp_path / "a.c").write_text('#include <stdio.h>\n#include <stddef.h>\n#include <stdint.h>\n#include "bpdq.h"\nint main(void){printf("%zu %zu %zu %zu %zu %d",'
                                  "sizeof(bpdq_stream_mix),sizeof(bpdq_grouped_shape),offsetof(bpdq_hybrid_layer,mix1),offsetof(bpdq_hybrid_layer,w_gates),"
                                  "offsetof(bpdq_hybrid_config,head),BPDQ_MAX_STREAMS);return 0;}")
    subprocess.check_call(["gcc", "-I", os.path.join(root, "include"), str(tmp_path / "a.c"), "-o", str(tmp_path / "a")])
    got = subprocess.check_output([str(tmp_path / "a")], text=True).split()
    want = [C.sizeof(capi.StreamMix), C.sizeof(capi.GroupedShape), capi.HybridLayer.mix1.offset, capi.HybridLayer.w_gates.offset, capi.HybridConfig.head.offset,
            capi.MAX_STREAMS]
    assert [int(v) for v in got] == want


def test_registry(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(vm.CONFIGS["single"]))
    assert registry.architecture_of(str(tmp_path)) == "Vuzelix" and "Vuzelix" in registry.FAMILIES
