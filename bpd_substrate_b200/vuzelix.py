"""Vuzelix: a hybrid decoder of gated-delta-rule layers with a decay per key channel and grouped-query attention layers (chunks, capped
scores, a sink; some layers on an earlier layer's keys and values), GELU feed-forwards, and several residual streams joined by
hyper-connections around every sublayer.  Configuration and packing; ``hybrid.DeviceHybrid`` runs it.
"""
import numpy as np

from . import capi
from .hybrid import DecoderSpec, Ends, Pack, _blocks, _cols, _positive, _spread, _vec, pad16
from .sequences import StatePart

MIXERS = {"channel_delta": capi.MIX_DELTA, "attention": capi.MIX_GROUPED}


def _number(where, d, key, positive=False):
    v = d.get(key)
    if not isinstance(v, (int, float)) or isinstance(v, bool) or (positive and not v > 0):
        raise ValueError(f"{where}: '{key}' must be a {'positive ' if positive else ''}number, not {v!r}")
    return float(v)


def _chunk(m):
    return m["mask"]["size"] if m.get("mask") is not None else 0


class VuzelixSpec(DecoderSpec):
    architecture = "Vuzelix"
    portion = 4096          # attention layers keep this many rows beyond a chunk: a step of as many tokens overwrites none it needs

    def check(self):
        c = self.config
        _positive("config", c, "streams")
        if c["streams"] > capi.MAX_STREAMS:
            raise ValueError(f"{c['streams']} residual streams; up to {capi.MAX_STREAMS} are supported")
        self.streams = c["streams"]
        self.embed_scale = _number("embedding", c["embedding"], "scale")
        self.residual_mult = _number("config", c, "residual_mult")
        self.logit_cap = _number("config", c, "logit_softcap", True)
        self.ranks = {}         # delta-rule layer -> ranks of its decays and gates
        for i, layer in enumerate(self.layers):
            where, kind, m = f"layer {i}", layer.get("type"), layer.get("mixer")
            if kind not in MIXERS:
                raise ValueError(f"{where}: unknown mixer {kind!r}")
            _positive(where, m, "heads", "kv_heads", "dim", "vdim")
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"{where}: {m['kv_heads']} key heads do not divide {m['heads']} heads")
            if kind == "channel_delta":
                _positive(where, m, "conv")
            else:
                _number(where, m, "scale")
                _number(where, m, "softcap", True)
                if m.get("mask") is not None:       # without one a position sees everything before it
                    _positive(where, m["mask"], "size")
                j = m.get("kv_from")
                if j is not None:
                    own = self.layers[j] if isinstance(j, int) and 0 <= j < i else None
                    if own is None or own["type"] != "attention" or own["mixer"].get("kv_from") is not None:
                        raise ValueError(f"{where}: kv_from {j!r} is not an earlier layer with keys of its own")
                    if any(own["mixer"][k] != m[k] for k in ("heads", "kv_heads", "dim", "vdim")):
                        raise ValueError(f"{where}: keys of layer {j} have other sizes")
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")
                _positive(where, mlp, "ff")

    def read_shapes(self, shape):
        for i, layer in enumerate(self.layers):
            if layer["type"] == "channel_delta":
                self.ranks[i] = (int(shape(f"l{i}.mix.a1")[0]), int(shape(f"l{i}.mix.g1")[0]))

    def tensor_shapes(self):
        """Every tensor of a checkpoint, in order: {name: shape}."""
        W, S, out = self.width, self.streams, {"embed": (self.vocab, self.width)}
        for i, layer in enumerate(self.layers):
            p, m, subs = f"l{i}.mix.", layer["mixer"], 2 if layer.get("mlp") else 1
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({f"l{i}.norm{q}": (W,) for q in range(1, subs + 1)})
            if layer["type"] == "attention":
                out[p + "q"] = (H * D, W)
                if m.get("kv_from") is None:
                    out.update({p + "k": (G * D, W), p + "v": (G * V, W)})
            else:
                a, g = self.ranks[i]
                for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                    out.update({p + n: (rows, W), f"{p}{n}.conv": (rows, m["conv"])})
                out.update({p + "b": (H, W), p + "A_log": (H,), p + "norm": (V,), p + "a1": (a, W), p + "a2": (H * D, a), p + "dt_bias": (H * D,),
                            p + "g1": (g, W), p + "g2": (H * V, g)})
            out[p + "o"] = (W, H * V)
            if layer.get("mlp"):
                out.update({f"l{i}.mlp.up": (layer["mlp"]["ff"], W), f"l{i}.mlp.down": (W, layer["mlp"]["ff"])})
            for q in range(1, subs + 1):
                out.update({f"l{i}.hc{q}.in": (S,), f"l{i}.hc{q}.out": (S,), f"l{i}.hc{q}.mix": (S, S)})
        out.update({"final.norm": (W,), "head": (self.vocab, W)})
        return out

    def state_parts(self, act_bf16):
        """What a sequence holds, layer by layer."""
        parts, a = [], 2 if act_bf16 else 4
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            D, V = pad16(m["dim"]), pad16(m["vdim"])
            if layer["type"] == "channel_delta":
                parts.append(StatePart(f"l{i}.state", 4 * m["heads"] * D * V))
                parts.append(StatePart(f"l{i}.tail", 4 * max(1, m["conv"] - 1) * (2 * m["kv_heads"] * D + m["heads"] * V)))
            elif m.get("kv_from") is None:
                reach = [_chunk(u["mixer"]) for j, u in enumerate(self.layers) if u["type"] == "attention" and i in (j, u["mixer"].get("kv_from"))]
                parts.append(StatePart(f"l{i}.cache", a * m["kv_heads"] * (D + V), rows=True, zero=False,
                                       limit=max(reach) + self.portion if all(reach) else 0))
        return parts

    def pack_layer(self, i, get):
        layer, Wp = self.layers[i], self.width_pad
        m, p, out = layer["mixer"], f"l{i}.mix.", Pack()
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        Dp, Vp = pad16(D), pad16(V)
        out.ints.update(mixer=MIXERS[layer["type"]], heads=H, groups=G, key_dim=D, key_pad=Dp, value_dim=V, value_pad=Vp, kv_from=-1)

        def rows(name, heads, size, cols=Wp):
            return _cols(_spread(get.bf16(p + name), 0, _blocks(heads, size, pad16(size)), heads * pad16(size)), cols)

        def channels(a, heads, size):
            return _spread(a, 0, _blocks(heads, size, pad16(size)), heads * pad16(size))

        out.mats["w_o"] = _spread(_spread(get.bf16(p + "o"), 1, _blocks(H, V, Vp), H * Vp), 0, np.arange(self.width), Wp)
        if layer["type"] == "attention":
            w_in = [rows("q", H, D)]
            if m.get("kv_from") is None:
                w_in += [rows("k", G, D), rows("v", G, V)]
            else:
                out.ints["kv_from"] = m["kv_from"]
            out.mats["w_in"] = np.concatenate(w_in)
            out.ints["chunk"] = _chunk(m)
            out.floats.update(scale=float(m["scale"]), softcap=float(m["softcap"]))
        else:
            a, g = self.ranks[i]
            R = pad16(max(a, g))

            def low(name, rank):
                return _spread(_cols(get.bf16(p + name), Wp), 0, np.arange(rank), R)
            out.mats["w_in"] = np.concatenate([rows("q", G, D), rows("k", G, D), rows("v", H, V), low("a1", a), low("g1", g), _cols(get.bf16(p + "b"), Wp)])
            out.mats["w_gates"] = np.concatenate([rows("a2", H, D, R), rows("g2", H, V, R)])
            conv = [channels(get.f32(p + n + ".conv"), heads, size) for n, heads, size in (("q", G, D), ("k", G, D), ("v", H, V))]
            rate = np.repeat(-np.exp(get.f32(p + "A_log").astype(np.float64)), D)
            out.vecs.update(conv_w=np.concatenate(conv).T, dt_bias=channels(get.f32(p + "dt_bias"), H, D), neg_exp_a=channels(rate, H, D),
                            norm_w=channels(np.tile(get.f32(p + "norm"), H), H, V))
            out.ints.update(conv=m["conv"], gate_rank_pad=R)
            out.floats["scale"] = D ** -0.5
        out.norms["norm1"] = (_vec(get, f"l{i}.norm1", Wp), None, 0.0)
        out.mixes["mix1"] = self._mix(get, f"l{i}.hc1")
        if layer.get("mlp"):
            F = layer["mlp"]["ff"]
            Fp = pad16(F)
            out.mats["w_gate_up"] = _spread(_cols(get.bf16(f"l{i}.mlp.up"), Wp), 0, np.arange(F), Fp)
            out.mats["w_down"] = _spread(_cols(get.bf16(f"l{i}.mlp.down"), Fp), 0, np.arange(self.width), Wp)
            out.ints.update(ff_pad=Fp, ff_kind=capi.FF_GELU)
            out.norms["norm2"] = (_vec(get, f"l{i}.norm2", Wp), None, 0.0)
            out.mixes["mix2"] = self._mix(get, f"l{i}.hc2")
        return out

    def _mix(self, get, name):
        """Connections of a sublayer; its output's share carries the residual multiplier."""
        d, n = capi.StreamMix(), capi.MAX_STREAMS
        mix = get.f32(name + ".mix")
        for s in range(self.streams):
            for t in range(self.streams):
                d.mix[s * n + t] = float(mix[s, t])
            d.out[s] = self.residual_mult * float(get.f32(name + ".out")[s])
            d.in_[s] = float(get.f32(name + ".in")[s])
        return d

    def pack_ends(self, get):
        return Ends(_cols(get.bf16("embed"), self.width_pad), _cols(get.bf16("head"), self.width_pad), (_vec(get, "final.norm", self.width_pad), None, 0.0),
                    {"streams": self.streams, "embed_scale": self.embed_scale, "logit_cap": self.logit_cap})

    def synthetic_value(self, name, leaf, shape, rng):
        if name == "embed":
            return rng.standard_normal(shape, dtype=np.float32) / np.float32(self.embed_scale)
        if "norm" in leaf:
            return 1.0 + 0.1 * rng.standard_normal(shape, dtype=np.float32)
        if leaf == "A_log":
            return np.log(rng.uniform(1.0, 4.0, shape)).astype(np.float32)
        if leaf == "dt_bias":
            return rng.uniform(-4.0, -1.0, shape).astype(np.float32)
        if leaf == "conv":
            return (0.5 * rng.standard_normal(shape)).astype(np.float32)
        if leaf == "mix":
            return np.eye(shape[0], dtype=np.float32) + 0.05 * rng.standard_normal(shape, dtype=np.float32)
        if leaf in ("in", "out"):
            return 1.0 / shape[0] + 0.1 * rng.standard_normal(shape, dtype=np.float32)
        return None
