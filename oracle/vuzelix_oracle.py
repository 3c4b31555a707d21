"""Plain, slow restatement of the Vuzelix decoder's mechanisms in numpy, one function per mechanism: gated delta rule with a
decay per key channel, chunked attention with a capped score and a sink, residual streams joined by hyper-connections.

Everything is written token by token from the equations, in binary64 unless another dtype is asked for, and shares nothing
with the product path.  Used by the tests only.
"""
import numpy as np

from .hybrid_oracle import causal_conv, rms, silu, softplus


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def unit(x):
    """x over its length along the last axis."""
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_step(state, decay, beta, k, v, q):
    """One token of one head: the state [key, value] decays row by row, the value it predicts for k moves towards v by a
    share beta, then q reads it.  Returns (state, output)."""
    state = decay[:, None] * state
    u = beta * (v - state.T @ k)
    state = state + np.outer(k, u)
    return state, state.T @ q


def sees(i, j, size):
    """Whether position i sees position j: no later than i, in the same chunk of `size` counted from position 0 (size 0:
    no chunks)."""
    return j <= i and (not size or i // size == j // size)


def attend(q, keys, values, scale, cap):
    """One query over the keys it sees; one more score of 0 that has no value."""
    s = np.array([soft_cap((q @ k) * scale, cap) for k in keys])
    top = max(0.0, s.max())
    e = np.exp(s - top)
    p = e / (np.exp(-top) + e.sum())
    return sum(p[j] * values[j] for j in range(len(values)))


def read_streams(x, weights):
    """The sublayer's input: a weighted sum of the streams x [streams, width]."""
    return weights @ x


def write_streams(x, y, mix, out, mult):
    """Stream t becomes sum_s mix[s, t] x_s + mult out[t] y."""
    return mix.T @ x + mult * np.outer(out, y)


class DeltaState:
    def __init__(self, m, dtype):
        self.s = np.zeros((m["heads"], m["dim"], m["vdim"]), dtype)
        sizes = {"q": m["kv_heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["heads"] * m["vdim"]}
        self.tails = {n: np.zeros((m["conv"] - 1, c), dtype) for n, c in sizes.items()}


class CacheState:
    def __init__(self, m, dtype):
        self.k, self.v = [], []


def channel_delta(m, w, p, h, st, eps):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    u = {}
    for n in "qkv":
        history = np.concatenate([st.tails[n], (w[f"{p}.{n}"] @ h)[None]], axis=0)
        st.tails[n] = history[1:]
        u[n] = silu(causal_conv(history, w[f"{p}.{n}.conv"], 0.0))
    q = unit(u["q"].reshape(G, D)) * float(D) ** -0.5
    k = unit(u["k"].reshape(G, D))
    v = u["v"].reshape(H, V)
    beta = sigmoid(w[p + ".b"] @ h)
    step = softplus(w[p + ".a2"] @ (w[p + ".a1"] @ h) + w[p + ".dt_bias"]).reshape(H, D)
    o = np.empty((H, V), h.dtype)
    for n in range(H):
        g = n // (H // G)
        st.s[n], o[n] = delta_step(st.s[n], np.exp(-np.exp(w[p + ".A_log"][n]) * step[n]), beta[n], k[g], v[n], q[g])
    gate = sigmoid(w[p + ".g2"] @ (w[p + ".g1"] @ h)).reshape(H, V)
    return w[p + ".o"] @ (rms(o, eps) * w[p + ".norm"] * gate).reshape(-1)


def attention_append(m, w, p, h, st, eps):
    """Adds this token's keys and values to the layer's own cache."""
    G = m["kv_heads"]
    st.k.append(rms((w[p + ".k"] @ h).reshape(G, m["dim"]), eps))
    st.v.append((w[p + ".v"] @ h).reshape(G, m["vdim"]))


def attention(m, w, p, h, pos, st, eps):
    """st: the cache of the layer whose keys are used; its newest entry is this token's."""
    H, G = m["heads"], m["kv_heads"]
    q = rms((w[p + ".q"] @ h).reshape(H, m["dim"]), eps)
    seen = [j for j in range(pos + 1) if sees(pos, j, m["mask"]["size"] if m.get("mask") else 0)]
    o = []
    for n in range(H):
        g = n // (H // G)
        o.append(attend(q[n], [st.k[j][g] for j in seen], [st.v[j][g] for j in seen], m["scale"], m["softcap"]))
    return w[p + ".o"] @ np.concatenate(o)


STATES = {"channel_delta": DeltaState, "attention": CacheState}


class Model:
    """Runs one sequence token by token."""

    def __init__(self, config, weights, dtype=np.float64):
        self.cfg, self.dtype = config, dtype
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}
        self.reset()

    def reset(self):
        self.pos = 0
        self.states = [STATES[layer["type"]](layer["mixer"], self.dtype) for layer in self.cfg["layers"]]

    def mixer(self, i, h):
        layer, eps, p = self.cfg["layers"][i], self.cfg["norm"]["eps"], f"l{i}.mix"
        m, st = layer["mixer"], self.states[i]
        if layer["type"] == "channel_delta":
            return channel_delta(m, self.w, p, h, st, eps)
        if m.get("kv_from") is None:
            attention_append(m, self.w, p, h, st, eps)
        else:
            st = self.states[m["kv_from"]]
        return attention(m, self.w, p, h, self.pos, st, eps)

    def feed_forward(self, i, h):
        return self.w[f"l{i}.mlp.down"] @ gelu_tanh(self.w[f"l{i}.mlp.up"] @ h)

    def layer(self, i, x):
        w, eps = self.w, self.cfg["norm"]["eps"]
        for q, run in ((1, self.mixer), (2, self.feed_forward)):
            if q == 2 and self.cfg["layers"][i]["mlp"] is None:
                break
            hc = f"l{i}.hc{q}."
            h = rms(read_streams(x, w[hc + "in"]), eps) * w[f"l{i}.norm{q}"]
            x = write_streams(x, run(i, h), w[hc + "mix"], w[hc + "out"], self.cfg["residual_mult"])
        return x

    def token(self, tok):
        """Returns (logits, sum of the streams after every layer)."""
        x = np.tile(self.w["embed"][tok] * self.dtype(self.cfg["embedding"]["scale"]), (self.cfg["streams"], 1))
        after = []
        for i in range(len(self.cfg["layers"])):
            x = self.layer(i, x)
            after.append(x.sum(axis=0))
        self.pos += 1
        h = rms(x.sum(axis=0), self.cfg["norm"]["eps"]) * self.w["final.norm"]
        return soft_cap(self.w["head"] @ h, self.cfg["logit_softcap"]), after

    def run(self, tokens):
        """Logits [n, vocab] and residuals [layers, n, width] of a whole sequence from the start."""
        self.reset()
        out = [self.token(t) for t in tokens]
        return np.array([o[0] for o in out]), np.array([o[1] for o in out]).swapaxes(0, 1)

    def greedy(self, prompt, n):
        self.reset()
        for t in prompt:
            logits, _ = self.token(t)
        out = []
        for i in range(n):
            out.append(int(np.argmax(logits)))
            if i + 1 < n:
                logits, _ = self.token(out[-1])
        return out
