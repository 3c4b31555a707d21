"""Small Vuzelix decoders for the tests: configurations that differ in every size, and seeded weights whose shapes are written out
here a second time.  Weights are bf16-representable fp32 arrays, so oracle and product read the same numbers."""
import numpy as np

from .hybrid_models import bf16_round


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attention(heads, kv_heads, dim, vdim, chunk, scale, softcap, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap}
    if chunk:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, streams, layers, eps=1e-5, embed=3.0, mult=0.6, cap=12.0):
    return {"architecture": "Vuzelix", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "residual_mult": mult, "logit_softcap": cap, "layers": layers}


# both mixers with and without a feed-forward; shared key heads, other chunks than the owner of the keys, value sizes above and below
# key sizes, sizes that are no multiples of anything; no convolution window, no chunks; one stream and the most streams
CONFIGS = {
    "mixed": config(211, 72, 2, [
        layer("channel_delta", delta(6, 2, 24, 40, 4), 88),
        layer("attention", attention(6, 3, 20, 28, 24, 0.5, 9.0)),
        layer("attention", attention(6, 3, 20, 28, 40, 0.3, 25.0, kv_from=1), 50),
        layer("channel_delta", delta(3, 3, 40, 24, 2)),
        layer("attention", attention(4, 1, 16, 72, 17, 0.7, 6.0), 33),
    ]),
    "square": config(128, 64, 4, [
        layer("attention", attention(4, 4, 32, 32, 64, 0.4, 15.0), 96),
        layer("channel_delta", delta(4, 4, 32, 32, 3), 64),
        layer("attention", attention(4, 4, 32, 32, 64, 0.4, 15.0, kv_from=0), 64),
        layer("channel_delta", delta(8, 4, 64, 64, 3), 64),
    ], eps=1e-6, embed=1.0, mult=1.0, cap=30.0),
    "single": config(97, 40, 1, [
        layer("channel_delta", delta(1, 1, 8, 8, 1)),
        layer("attention", attention(1, 1, 8, 24, 5, 1.5, 4.0), 24),
        layer("channel_delta", delta(2, 1, 72, 136, 6), 20),
    ], mult=0.9),
    "wide": config(150, 88, 8, [
        layer("channel_delta", delta(2, 2, 136, 264, 3), 40),
        layer("attention", attention(2, 1, 120, 200, 90, 0.2, 20.0), 40),
        layer("attention", attention(3, 1, 264, 24, 33, 0.15, 8.0)),
        layer("attention", attention(2, 2, 16, 32, 0, 0.6, 8.0)),
        layer("channel_delta", delta(2, 1, 264, 16, 4), 30),
    ]),
}


def weights(cfg, seed=0, gain=1.0):
    rng = np.random.default_rng(seed)
    W, S, out = cfg["width"], cfg["streams"], {}

    def put(name, v):
        out[name] = bf16_round(np.asarray(v, np.float32))

    def mat(name, rows, cols, g=1.0):
        put(name, g * rng.standard_normal((rows, cols)) / np.sqrt(cols))

    put("embed", rng.standard_normal((cfg["vocab"], W)) / cfg["embedding"]["scale"])
    for i, la in enumerate(cfg["layers"]):
        p, m, H = f"l{i}.mix", la["mixer"], la["mixer"]["heads"]
        G, D, V = m["kv_heads"], m["dim"], m["vdim"]
        subs = 2 if la["mlp"] else 1
        for q in range(1, subs + 1):
            put(f"l{i}.norm{q}", 1.0 + 0.2 * rng.standard_normal(W))
        if la["type"] == "attention":
            mat(p + ".q", H * D, W, 2.0 * gain)
            if m.get("kv_from") is None:
                mat(p + ".k", G * D, W, 2.0 * gain)
                mat(p + ".v", G * V, W)
        else:
            a, g = 3 + 5 * i % 13, 17 - 4 * i % 11
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                mat(f"{p}.{n}", rows, W, 1.5)
                put(f"{p}.{n}.conv", rng.standard_normal((rows, m["conv"])) / np.sqrt(m["conv"]))
            mat(p + ".b", H, W, 2.0)
            put(p + ".A_log", np.log(rng.uniform(0.02, 3.0, H)))
            put(p + ".norm", 1.0 + 0.2 * rng.standard_normal(V))
            mat(p + ".a1", a, W)
            mat(p + ".a2", H * D, a)
            put(p + ".dt_bias", rng.uniform(-6.0, 1.0, H * D))
            mat(p + ".g1", g, W)
            mat(p + ".g2", H * V, g, 2.0)
        mat(p + ".o", W, H * V, 2.0)
        if la["mlp"]:
            mat(f"l{i}.mlp.up", la["mlp"]["ff"], W, 1.5)
            mat(f"l{i}.mlp.down", W, la["mlp"]["ff"], 2.0)
        for q in range(1, subs + 1):
            put(f"l{i}.hc{q}.in", 1.0 / S + 0.3 * rng.standard_normal(S))
            put(f"l{i}.hc{q}.out", 1.0 + 0.3 * rng.standard_normal(S))
            put(f"l{i}.hc{q}.mix", 0.9 * np.eye(S) + 0.25 * rng.standard_normal((S, S)) / np.sqrt(S))
    put("final.norm", 1.0 + 0.2 * rng.standard_normal(W))
    mat("head", cfg["vocab"], W, 4.0)
    return out
