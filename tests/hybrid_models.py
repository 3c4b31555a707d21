"""Small hybrid decoders for the tests: configurations that differ in every size, and seeded weights whose shapes are
written out here a second time.  Weights are bf16-representable fp32 arrays, so oracle and product read the same numbers."""
import numpy as np


def bf16_round(x):
    u = np.array(x, np.float32, order="C").view(np.uint32)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def bf16_bits(x):
    return (bf16_round(x).view(np.uint32) >> 16).astype(np.uint16)


def bits_f32(b):
    return (np.asarray(b, np.uint16).astype(np.uint32) << 16).view(np.float32)


def retention(heads, dim, vdim, rot, decay, base=500.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"dims": rot, "base": base}}


def mamba2(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=3000.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Gurusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# every mixer with and without a feed-forward; partial rotations, groups, parts that cut through heads, shared latents
# with other head sizes than their owner's, sizes that are no multiples of anything
CONFIGS = {
    "mixed": config(301, 72, [
        layer("latent_attention", latent(3, 24, 6, 40, 40, 56, 0.31), 88),
        layer("mamba2", mamba2(6, 24, 20, 3, 4, 4), 50),
        layer("retention", retention(3, 40, 24, 12, [0.5, 0.98, 0.999])),
        layer("latent_attention", latent(5, 16, 6, 20, 40, 24, 0.12, kv_from=0)),
        layer("mamba2", mamba2(2, 48, 72, 2, 2, 1)),
        layer("retention", retention(2, 16, 130, 16, [1.0, 0.9], base=1e4), 33),
    ]),
    "square": config(128, 64, [
        layer("retention", retention(4, 32, 32, 32, [0.9, 0.95, 0.99, 0.997]), 96),
        layer("latent_attention", latent(16, 32, 16, 32, 64, 48, 0.2)),
        layer("mamba2", mamba2(4, 32, 32, 1, 3, 2), 64),
        layer("latent_attention", latent(20, 32, 16, 64, 64, 64, 0.25, base=100.0), 32),
    ], eps=1e-6),
    "conv1": config(97, 40, [
        layer("mamba2", mamba2(3, 16, 150, 1, 1, 3)),
        layer("mamba2", mamba2(1, 8, 8, 1, 6, 1), 24),
    ]),
}


def weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    W, out = cfg["width"], {}

    def put(name, v):
        out[name] = bf16_round(np.asarray(v, np.float32))

    def mat(name, rows, cols, gain=1.0):
        put(name, gain * rng.standard_normal((rows, cols)) / np.sqrt(cols))

    def norm(name, w=1.0):
        put(name, w * (1.0 + 0.2 * rng.standard_normal(W)))
        put(name + ".b", 0.1 * rng.standard_normal(W))
        put(name + ".alpha", rng.uniform(0.4, 0.9))

    put("embed", rng.standard_normal((cfg["vocab"], W)))
    for i, la in enumerate(cfg["layers"]):
        p, m, H = f"l{i}.mix", la["mixer"], la["mixer"]["heads"]
        norm(f"l{i}.norm1")
        norm(f"l{i}.norm1b", 0.7)
        if la["type"] == "retention":
            mat(p + ".q", H * m["dim"], W, 1.5)
            mat(p + ".k", H * m["dim"], W, 1.5)
            mat(p + ".v", H * m["vdim"], W)
            mat(p + ".g", H * m["vdim"], W)
            mat(p + ".o", W, H * m["vdim"], 2.0)
        elif la["type"] == "mamba2":
            inner, ch = H * m["vdim"], H * m["vdim"] + 2 * m["groups"] * m["state"]
            mat(p + ".in", inner + ch + H, W, 1.5)
            put(p + ".conv", rng.standard_normal((ch, m["conv"])) / np.sqrt(m["conv"]))
            put(p + ".conv.b", 0.2 * rng.standard_normal(ch))
            put(p + ".dt_bias", rng.uniform(-3.0, 0.0, H))
            put(p + ".A_log", np.log(rng.uniform(0.05, 2.0, H)))
            put(p + ".D", 1.0 + 0.3 * rng.standard_normal(H))
            put(p + ".norm", 1.0 + 0.2 * rng.standard_normal(inner))
            mat(p + ".o", W, inner, 2.0)
        else:
            mat(p + ".dq", m["q_rank"], W)
            put(p + ".dq.norm", 1.0 + 0.2 * rng.standard_normal(m["q_rank"]))
            mat(p + ".uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], 2.0)
            if m.get("kv_from") is None:
                mat(p + ".dkv", m["kv_rank"] + m["rot_dim"], W, 1.5)
                put(p + ".dkv.norm", 1.0 + 0.2 * rng.standard_normal(m["kv_rank"]))
            mat(p + ".uk", H * m["dim"], m["kv_rank"], 1.5)
            mat(p + ".uv", H * m["vdim"], m["kv_rank"])
            mat(p + ".o", W, H * m["vdim"], 2.0)
        if la["mlp"]:
            norm(f"l{i}.norm2")
            norm(f"l{i}.norm2b", 0.7)
            mat(f"l{i}.mlp.gate", la["mlp"]["ff"], W, 1.5)
            mat(f"l{i}.mlp.up", la["mlp"]["ff"], W)
            mat(f"l{i}.mlp.down", W, la["mlp"]["ff"], 2.0)
    norm("final.norm")
    return out


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def row_errors(got, want):
    """Per row: rms of the difference (mean taken off) over the rms of the expected row."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1) / (w ** 2).mean(-1).mean())
