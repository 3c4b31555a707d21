"""Hybrid decoders: a list of layers whose mixers differ.  This file holds what their designs share and one of them: layers of
retention, state-space duality (Mamba-2) or latent attention, with dynamic-tanh norms around every sublayer and the embedding
table as output head (Gurusun).  vuzelix.py holds the other.

A spec reads config.json (sizes and constants, checked), lists the checkpoint's tensors and what a sequence holds, and packs
tensors into what the kernels read (inner sizes padded to multiples of 16 with zero weights, products that share an input
stacked, gate and up rows interleaved); ``DeviceHybrid`` uploads them and runs ``bpdq_hybrid_forward``.  There is no CPU path.
"""
import ctypes as C
import json
import os

import numpy as np

from . import capi
from .safetensors_load import SafetensorsFile, bf16_to_f32
from .sequences import StatePart, lay_out

MAX_TOKENS = 65535      # of one step
MIXERS = {"retention": capi.MIX_RETENTION, "mamba2": capi.MIX_MAMBA2, "latent_attention": capi.MIX_LATENT}


def pad16(n):
    return -(-n // 16) * 16


def _positive(where, d, *keys):
    for k in keys:
        if not isinstance(d.get(k), int) or isinstance(d.get(k), bool) or d[k] < 1:
            raise ValueError(f"{where}: '{k}' must be a positive integer, not {d.get(k)!r}")


def _rotation(where, m, limit):
    rot = m.get("rot")
    if not isinstance(rot, dict):
        raise ValueError(f"{where}: no rotation ('rot')")
    dims = rot.get("dims")
    if not isinstance(dims, int) or dims < 2 or dims % 2 or dims > limit:
        raise ValueError(f"{where}: {dims!r} rotated dimensions of {limit}")
    return dims, float(rot["base"])


class DecoderSpec:
    """What every design of a hybrid decoder has.  A subclass names its architecture, checks its layers, and brings
    ``tensor_shapes``, ``state_parts``, ``pack_layer`` and ``pack_ends``."""
    architecture = None
    portion = None          # most tokens of a step once cache rows are used again

    def __init__(self, config):
        self.config = config
        if config.get("architecture") != self.architecture:
            raise ValueError(f"architecture {config.get('architecture')!r} is not {self.architecture}")
        _positive("config", config, "vocab", "width")
        self.vocab, self.width = config["vocab"], config["width"]
        self.width_pad = pad16(self.width)
        self.eps = float(config["norm"]["eps"])
        self.layers = config["layers"]
        self.check()

    def read_shapes(self, shape):
        """Sizes that only the checkpoint's tensors tell; shape(name) gives one."""

    @classmethod
    def from_folder(cls, folder):
        with open(os.path.join(folder, "config.json")) as f:
            return cls(json.load(f))


class HybridSpec(DecoderSpec):
    architecture = "Gurusun"

    def check(self):
        for i, layer in enumerate(self.layers):
            where, kind, m = f"layer {i}", layer.get("type"), layer.get("mixer")
            if kind not in MIXERS:
                raise ValueError(f"{where}: unknown mixer {kind!r}")
            if kind == "retention":
                _positive(where, m, "heads", "dim", "vdim")
                _rotation(where, m, m["dim"])
                if len(m["decay"]) != m["heads"] or not all(0.0 < d <= 1.0 for d in m["decay"]):
                    raise ValueError(f"{where}: needs a decay in (0, 1] for each of {m['heads']} heads")
            elif kind == "mamba2":
                _positive(where, m, "heads", "vdim", "state", "groups", "conv", "norm_groups")
                if m["heads"] % m["groups"] or (m["heads"] * m["vdim"]) % m["norm_groups"]:
                    raise ValueError(f"{where}: groups do not divide the heads, or norm_groups the channels")
            else:
                _positive(where, m, "heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")
                dims, base = _rotation(where, m, m["rot_dim"])
                if dims != m["rot_dim"]:
                    raise ValueError(f"{where}: rotates {dims} of a rotated part of {m['rot_dim']}")
                j = m.get("kv_from")
                if j is not None:
                    own = self.layers[j] if isinstance(j, int) and 0 <= j < i else None
                    if own is None or own["type"] != "latent_attention" or own["mixer"].get("kv_from") is not None:
                        raise ValueError(f"{where}: kv_from {j!r} is not an earlier layer with latents of its own")
                    o = own["mixer"]
                    if (o["kv_rank"], o["rot_dim"], o["rot"]) != (m["kv_rank"], m["rot_dim"], m["rot"]):
                        raise ValueError(f"{where}: latents of layer {j} have other sizes or another rotation")
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")
                _positive(where, mlp, "ff")

    def state_parts(self, act_bf16):
        """What a sequence holds, layer by layer."""
        parts, a = [], 2 if act_bf16 else 4
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            if layer["type"] == "retention":
                parts.append(StatePart(f"l{i}.state", 4 * m["heads"] * pad16(m["dim"]) * pad16(m["vdim"])))
            elif layer["type"] == "mamba2":
                channels = m["heads"] * pad16(m["vdim"]) + 2 * m["groups"] * pad16(m["state"])
                parts.append(StatePart(f"l{i}.state", 4 * m["heads"] * pad16(m["state"]) * pad16(m["vdim"])))
                parts.append(StatePart(f"l{i}.tail", 4 * max(1, m["conv"] - 1) * channels))
            elif m.get("kv_from") is None:
                parts.append(StatePart(f"l{i}.cache", a * (pad16(m["kv_rank"]) + pad16(m["rot_dim"])), rows=True, zero=False))
        return parts

    def tensor_shapes(self):
        """Every tensor of a checkpoint, in order: {name: shape}."""
        W, out = self.width, {"embed": (self.vocab, self.width)}

        def norm(name):
            out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

        for i, layer in enumerate(self.layers):
            p, m, mlp = f"l{i}.mix.", layer["mixer"], layer.get("mlp")
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp else ()):
                norm(f"l{i}.{n}")
            H = m["heads"]
            if layer["type"] == "retention":
                out.update({p + "q": (H * m["dim"], W), p + "k": (H * m["dim"], W), p + "v": (H * m["vdim"], W),
                            p + "g": (H * m["vdim"], W), p + "o": (W, H * m["vdim"])})
            elif layer["type"] == "mamba2":
                inner, gn = H * m["vdim"], m["groups"] * m["state"]
                out.update({p + "in": (2 * inner + 2 * gn + H, W), p + "conv": (inner + 2 * gn, m["conv"]), p + "conv.b": (inner + 2 * gn,),
                            p + "dt_bias": (H,), p + "A_log": (H,), p + "D": (H,), p + "norm": (inner,), p + "o": (W, inner)})
            else:
                out.update({p + "dq": (m["q_rank"], W), p + "dq.norm": (m["q_rank"],), p + "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"])})
                if m.get("kv_from") is None:
                    out.update({p + "dkv": (m["kv_rank"] + m["rot_dim"], W), p + "dkv.norm": (m["kv_rank"],)})
                out.update({p + "uk": (H * m["dim"], m["kv_rank"]), p + "uv": (H * m["vdim"], m["kv_rank"]), p + "o": (W, H * m["vdim"])})
            if mlp:
                out.update({f"l{i}.mlp.gate": (mlp["ff"], W), f"l{i}.mlp.up": (mlp["ff"], W), f"l{i}.mlp.down": (W, mlp["ff"])})
        norm("final.norm")
        return out

    def pack_layer(self, i, get):
        return pack_layer(self, i, get)

    def pack_ends(self, get):
        """Embedding, head and final norm; numbers of the model's descriptor."""
        return Ends(_cols(get.bf16("embed"), self.width_pad), None, _norm(get, "final.norm", self.width_pad), {})

    def synthetic_value(self, name, leaf, shape, rng):
        """Random values of a tensor that is no matrix of a product, or None."""
        if name == "embed":
            return rng.standard_normal(shape, dtype=np.float32)
        if leaf == "alpha":
            return np.float32(0.5)
        if name.endswith(".conv.b") or (leaf == "b" and "norm" in name):
            return 0.05 * rng.standard_normal(shape, dtype=np.float32)
        if leaf in ("D",) or "norm" in leaf:
            return 1.0 + 0.1 * rng.standard_normal(shape, dtype=np.float32)
        if leaf == "A_log":
            return np.log(rng.uniform(1.0, 4.0, shape)).astype(np.float32)
        if leaf == "dt_bias":
            return rng.uniform(-4.0, -1.0, shape).astype(np.float32)
        if leaf == "conv":
            return (0.5 * rng.standard_normal(shape)).astype(np.float32)
        return None


# ---- packing: zero padding of inner sizes

def _blocks(n_blocks, size, size_pad):
    """Places of n_blocks runs of `size` entries when every run is stored size_pad apart."""
    return (np.arange(n_blocks)[:, None] * size_pad + np.arange(size)[None, :]).reshape(-1)


def _spread(a, axis, places, total):
    """Entries of `a` along `axis` moved to `places` of an axis of `total`, zeros elsewhere."""
    if a.shape[axis] == total:         # nothing to pad: the places are 0, 1, ...
        return a
    shape = list(a.shape)
    shape[axis] = total
    out = np.zeros(shape, a.dtype)
    if axis == 0:
        out[places] = a
    else:
        out[:, places] = a
    return out


def _cols(a, total):
    return _spread(a, 1, np.arange(a.shape[1]), total)


def rotary_frequencies(dims, base):
    return (float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)).astype(np.float32)


class Pack:
    """Host arrays of one layer as the kernels read them: `mats` (uint16 bf16 bits), `vecs` (fp32), `norms` (w, b or None, alpha),
    `mixes` (capi.StreamMix), and the descriptor's numbers: `ints`, `floats`."""

    def __init__(self):
        self.mats, self.vecs, self.ints, self.norms, self.mixes, self.floats = {}, {}, {}, {}, {}, {"scale": 1.0}


class Ends:
    """What lies around the layers: bf16 bits of the embedding and the head (None: the embedding again), the final norm, and
    further numbers of the descriptor."""

    def __init__(self, embed, head, norm, numbers):
        self.embed, self.head, self.norm, self.numbers = embed, head, norm, numbers


def _vec(get, name, total):
    v = np.zeros(total, np.float32)
    a = get.f32(name)
    v[:a.size] = a
    return v


def _norm(get, name, width_pad):
    return _vec(get, name, width_pad), _vec(get, name + ".b", width_pad), float(get.f32(name + ".alpha").reshape(()))


def pack_layer(spec, i, get):
    layer, Wp = spec.layers[i], spec.width_pad
    m, p, out = layer["mixer"], f"l{i}.mix.", Pack()
    H, kind = m["heads"], layer["type"]
    key = {"retention": "dim", "mamba2": "state", "latent_attention": "dim"}[kind]
    D, V = m[key], m["vdim"]
    Dp, Vp = pad16(D), pad16(V)
    out.ints.update(mixer=MIXERS[kind], heads=H, groups=H, key_dim=D, key_pad=Dp, value_dim=V, value_pad=Vp, kv_from=-1)
    rows_d, rows_v = _blocks(H, D, Dp), _blocks(H, V, Vp)

    def mat(name):
        return get.bf16(p + name)

    def padded_rows(name, places, total, cols=Wp):
        return _cols(_spread(mat(name), 0, places, total), cols)

    out.mats["w_o"] = _spread(_spread(mat("o"), 1, rows_v, H * Vp), 0, np.arange(spec.width), Wp)
    if kind == "retention":
        dims, base = m["rot"]["dims"], m["rot"]["base"]
        out.mats["w_in"] = np.concatenate([padded_rows("q", rows_d, H * Dp), padded_rows("k", rows_d, H * Dp),
                                           padded_rows("v", rows_v, H * Vp), padded_rows("g", rows_v, H * Vp)])
        decay = np.asarray(m["decay"], np.float64)
        out.vecs.update(rot_freq=rotary_frequencies(dims, base), decay=decay, log_decay=np.log(decay))
        out.ints.update(rot_dims=dims)
        out.floats["scale"] = D ** -0.5
    elif kind == "mamba2":
        G = m["groups"]
        inner, gn, taps = H * V, G * D, m["conv"]
        w = _cols(mat("in"), Wp)
        rows_n = _blocks(G, D, Dp)
        cuts = np.cumsum([inner, inner, gn, gn])
        z, x, b, c, dt = np.split(w, cuts)
        out.mats["w_in"] = np.concatenate([_spread(z, 0, rows_v, H * Vp), _spread(x, 0, rows_v, H * Vp), _spread(b, 0, rows_n, G * Dp),
                                           _spread(c, 0, rows_n, G * Dp), dt])
        places = np.concatenate([rows_v, H * Vp + rows_n, H * Vp + G * Dp + rows_n])
        channels = H * Vp + 2 * G * Dp
        out.vecs.update(conv_w=_spread(get.f32(p + "conv"), 0, places, channels).T, conv_b=_spread(get.f32(p + "conv.b"), 0, places, channels),
                        dt_bias=get.f32(p + "dt_bias"), neg_exp_a=-np.exp(get.f32(p + "A_log").astype(np.float64)), d_skip=get.f32(p + "D"),
                        norm_w=_spread(get.f32(p + "norm"), 0, rows_v, H * Vp))
        out.ints.update(groups=G, conv=taps, norm_groups=m["norm_groups"])
    else:
        Q, R, r = m["q_rank"], m["kv_rank"], m["rot_dim"]
        Qp, Rp, rp = pad16(Q), pad16(R), pad16(r)
        w_in = [padded_rows("dq", np.arange(Q), Qp)]
        if m.get("kv_from") is None:
            dkv = _cols(mat("dkv"), Wp)
            w_in += [_spread(dkv[:R], 0, np.arange(R), Rp), _spread(dkv[R:], 0, np.arange(r), rp)]
            out.vecs["kv_norm_w"] = _spread(get.f32(p + "dkv.norm"), 0, np.arange(R), Rp)
        else:
            out.ints["kv_from"] = m["kv_from"]
        out.mats["w_in"] = np.concatenate(w_in)
        head = np.concatenate([np.arange(D), Dp + np.arange(r)])
        rows_q = (np.arange(H)[:, None] * (Dp + rp) + head[None, :]).reshape(-1)
        out.mats["w_uq"] = padded_rows("uq", rows_q, H * (Dp + rp), Qp)
        out.mats["w_ukv"] = np.concatenate([padded_rows("uk", rows_d, H * Dp, Rp), padded_rows("uv", rows_v, H * Vp, Rp)])
        out.vecs.update(q_norm_w=_spread(get.f32(p + "dq.norm"), 0, np.arange(Q), Qp), rot_freq=rotary_frequencies(r, m["rot"]["base"]))
        out.ints.update(rot_dims=r, rot_pad=rp, q_rank=Q, q_rank_pad=Qp, kv_rank=R, kv_rank_pad=Rp)
        out.floats["scale"] = float(m["scale"])
    out.norms["norm1"] = _norm(get, f"l{i}.norm1", Wp)
    out.norms["norm1b"] = _norm(get, f"l{i}.norm1b", Wp)
    if layer.get("mlp"):
        F = layer["mlp"]["ff"]
        Fp = pad16(F)
        gate_up = np.zeros((2 * Fp, Wp), np.uint16)
        gate_up[0:2 * F:2] = _cols(get.bf16(f"l{i}.mlp.gate"), Wp)
        gate_up[1:2 * F:2] = _cols(get.bf16(f"l{i}.mlp.up"), Wp)
        out.mats["w_gate_up"] = gate_up
        out.mats["w_down"] = _spread(_cols(get.bf16(f"l{i}.mlp.down"), Fp), 0, np.arange(spec.width), Wp)
        out.ints["ff_pad"] = Fp
        out.norms["norm2"] = _norm(get, f"l{i}.norm2", Wp)
        out.norms["norm2b"] = _norm(get, f"l{i}.norm2b", Wp)
    return out


class ArrayTensors:
    """Tensors of a model held in memory: {name: float32 array or uint16 bf16 bits}."""

    def __init__(self, tensors):
        from .safetensors_load import f32_to_bf16
        self._bits = {k: (v if np.asarray(v).dtype == np.uint16 else f32_to_bf16(v)) for k, v in tensors.items()}

    def bf16(self, name):
        return self._bits[name]

    def f32(self, name):
        return bf16_to_f32(self._bits[name])

    def shape(self, name):
        return self._bits[name].shape


def synthetic_tensors(spec, seed=0):
    """Random weights of the right shapes (bf16 bits): products keep activations O(1)."""
    rng = np.random.default_rng(seed)
    from .safetensors_load import f32_to_bf16
    out, pool = {}, rng.standard_normal(1 << 20, dtype=np.float32)
    pools = {}

    def matrix(shape):
        """Large matrices repeat a pool of a million numbers (every row at another place of it)."""
        if shape[0] * shape[1] <= pool.size:
            return f32_to_bf16(rng.standard_normal(shape, dtype=np.float32) / np.float32(np.sqrt(shape[1])))
        bits = pools.setdefault(shape[1], f32_to_bf16(pool / np.float32(np.sqrt(shape[1]))))
        start = int(rng.integers(0, pool.size))
        return np.resize(np.roll(bits, start)[:pool.size - 7], shape)

    for name, shape in spec.tensor_shapes().items():
        v = spec.synthetic_value(name, name.rsplit(".", 1)[-1], shape, rng)
        out[name] = matrix(shape) if v is None else f32_to_bf16(np.asarray(v, np.float32))
    return out


class DeviceHybrid:
    """A hybrid decoder resident on the device.  `step` is the one entry that generation, the trace runner and the
    tests drive: some tokens of one sequence, logits where they are asked for."""

    def __init__(self, spec, get, dtype="bfloat16", capacity=4096, lib=None, stream=None, use_graph=True):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
        self.lib = lib = lib or capi.load()
        self.spec, self.vocab, self.dtype, self.capacity, self.use_graph = spec, spec.vocab, dtype, capacity, use_graph
        self._own_stream = stream is None
        self.stream = lib.bpdq_stream_create() if stream is None else stream
        self._allocs, self.weight_bytes = [], 0
        spec.read_shapes(get.shape)
        self.parts = spec.state_parts(dtype == "bfloat16")
        offsets, rows = lay_out(self.parts, capacity).offsets, {p.name: p.count(capacity) for p in self.parts}
        self.layers = (capi.HybridLayer * max(1, len(spec.layers)))()
        for i in range(len(spec.layers)):
            pk, dst = spec.pack_layer(i, get), self.layers[i]
            for k, v in list(pk.ints.items()) + list(pk.floats.items()) + list(pk.mixes.items()):
                setattr(dst, k, v)
            for k, v in pk.mats.items():
                setattr(dst, k, self._up(np.ascontiguousarray(v, np.uint16)))
            for k, v in pk.vecs.items():
                setattr(dst, k, self._up(np.ascontiguousarray(v, np.float32)))
            for k, (w, b, alpha) in pk.norms.items():
                setattr(dst, k, self._norm_of(w, b, alpha))
            dst.cache_rows = rows.get(f"l{i if dst.kv_from < 0 else dst.kv_from}.cache", 0)
            for part in ("state", "tail", "cache"):
                setattr(dst, part + "_offset", offsets.get(f"l{i}.{part}", 0))
        ends = spec.pack_ends(get)
        self.config = capi.HybridConfig(n_layers=len(spec.layers), width=spec.width, width_pad=spec.width_pad, vocab=spec.vocab,
                                        act_bf16=int(dtype == "bfloat16"), eps=spec.eps, final_norm=self._norm_of(*ends.norm), **ends.numbers)
        self.config.embed = self._up(ends.embed)
        self.config.head = self.config.embed if ends.head is None else self._up(ends.head)
        self.plan = lib.bpdq_hybrid_create(C.byref(self.config), self.layers)
        capi.check(lib.bpdq_last_status(), "hybrid decoder set-up")
        if not self.plan:
            raise capi.BpdqError("bpdq_hybrid_create refused the model")
        # most tokens of one step: less where a layer keeps only its latest rows
        self.portion = spec.portion if any(p.rows and p.count(capacity) < capacity for p in self.parts) else MAX_TOKENS

    @classmethod
    def from_folder(cls, folder, spec_class=HybridSpec, **kw):
        spec = spec_class.from_folder(folder)
        f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
        try:
            spec.read_shapes(f.shape)
            for name, shape in spec.tensor_shapes().items():
                got = tuple(f.tensors[name]["shape"]) if name in f else None
                if got != tuple(shape):
                    raise ValueError(f"{f.path}: tensor {name} has shape {got}, config.json says {tuple(shape)}")
            return cls(spec, f, **kw)
        finally:
            f.close()

    def _up(self, arr):
        arr = np.ascontiguousarray(arr)
        p = self.lib.bpdq_alloc(max(arr.nbytes, 16))
        if not p:
            raise MemoryError(f"device allocation of {arr.nbytes} bytes failed")
        self.lib.bpdq_h2d(p, arr.ctypes.data, arr.nbytes)
        self._allocs.append(p)
        self.weight_bytes += arr.nbytes
        return p

    def _norm_of(self, w, b, alpha):
        return capi.DynTanh(self._up(w), None if b is None else self._up(b), alpha)

    def state_parts(self):
        return self.parts

    def launch(self, seq, tokens, want=(), residuals=None):
        """Queues the tokens of `seq`; results stay on the device until the next call."""
        tokens = np.ascontiguousarray(tokens, np.int32)
        want = np.ascontiguousarray(want, np.int32)
        n = tokens.size
        if n == 0:
            raise ValueError("a step needs at least one token")
        if seq.length + n > seq.capacity:
            raise ValueError(f"the sequence would hold {seq.length + n} tokens, its slot has room for {seq.capacity}")
        if n > self.portion:
            raise ValueError(f"a step of {n} tokens; this model takes up to {self.portion}")
        if tokens.min() < 0 or tokens.max() >= self.vocab:
            raise ValueError(f"token ids run from 0 to {self.vocab - 1}")
        capi.check(self.lib.bpdq_hybrid_forward(self.plan, tokens.ctypes.data, n, seq.length, seq.base, want.ctypes.data, want.size, residuals,
                                                int(self.use_graph), self.stream), "bpdq_hybrid_forward")
        seq.length += n

    def step(self, seq, tokens, want=(), logits=True):
        """Runs the tokens; returns (logits [len(want), vocab] or None, greedy token ids [len(want)])."""
        self.launch(seq, tokens, want)
        n = len(want)
        out = np.empty((n, self.vocab), np.float32) if logits else None
        picked = np.empty(n, np.int64)
        if n:
            if logits:
                capi.check(self.lib.bpdq_d2h_async(out.ctypes.data, self.lib.bpdq_hybrid_logits(self.plan), out.nbytes, self.stream))
            capi.check(self.lib.bpdq_d2h_async(picked.ctypes.data, self.lib.bpdq_hybrid_picked(self.plan), picked.nbytes, self.stream))
        capi.check(self.lib.bpdq_stream_sync(self.stream), "hybrid step")
        return out, picked

    def residuals(self, seq, tokens):
        """The residual stream after every layer, [layers, tokens, width]."""
        n, L = len(tokens), len(self.spec.layers)
        out = np.empty((L, n, self.spec.width), np.float32)
        d = self.lib.bpdq_alloc(max(out.nbytes, 16))
        try:
            self.launch(seq, tokens, (), d)
            capi.check(self.lib.bpdq_stream_sync(self.stream))
            self.lib.bpdq_d2h(out.ctypes.data, d, out.nbytes)
        finally:
            self.lib.bpdq_free(d)
        return out

    def close(self):
        self.lib.bpdq_stream_sync(self.stream)
        self.lib.bpdq_hybrid_destroy(self.plan)
        for p in self._allocs:
            self.lib.bpdq_free(p)
        self._allocs = []
        if self._own_stream:
            self.lib.bpdq_stream_destroy(self.stream)
