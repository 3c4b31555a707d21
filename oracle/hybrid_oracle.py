"""Plain, slow restatement of the hybrid decoder's mechanisms in numpy, one function per mechanism.

Everything is written token by token from the equations, in binary64 unless another dtype is asked for,
and shares nothing with the product path.  Used by the tests only.

A weight dictionary maps tensor names ('embed', 'l0.mix.q', ...) to arrays; linear weights are
[out, in] and applied as W @ x.
"""
import numpy as np


def rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dynamic_tanh(x, w, name):
    """tanh(alpha x) * w + b; no statistics."""
    return np.tanh(float(w[name + ".alpha"]) * x) * w[name] + w[name + ".b"]


def silu(z):
    return z / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def rotate_half(x, pos, base, dims):
    """Pairs (i, i + dims/2) of the first `dims` entries of the last axis turn by pos * base^(-2i/dims)."""
    out = np.array(x)
    half = dims // 2
    for i in range(half):
        a = pos * float(base) ** (-2.0 * i / dims)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * np.cos(a) - v * np.sin(a)
        out[..., i + half] = v * np.cos(a) + u * np.sin(a)
    return out


def rotate_interleaved(x, pos, base, dims):
    """The same with pairs (2i, 2i + 1)."""
    out = np.array(x)
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def decayed_recurrence(state, decay, k, v, q):
    """One token of one head: S <- decay S + k v^T; returns (S, S^T q)."""
    state = decay * state + np.outer(k, v)
    return state, state.T @ q


def causal_conv(history, taps, bias):
    """history [taps, channels], oldest first, the last row is the current token."""
    return np.sum(history * taps.T, axis=0) + bias


class RetentionState:
    def __init__(self, m, dtype):
        self.s = np.zeros((m["heads"], m["dim"], m["vdim"]), dtype)


class Mamba2State:
    def __init__(self, m, dtype):
        self.s = np.zeros((m["heads"], m["state"], m["vdim"]), dtype)
        channels = m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
        self.tail = np.zeros((m["conv"] - 1, channels), dtype)


class LatentState:
    def __init__(self, m, dtype):
        self.c, self.r = [], []


def retention(m, w, p, h, pos, st, eps):
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (w[p + ".q"] @ h).reshape(H, D)
    k = (w[p + ".k"] @ h).reshape(H, D)
    v = (w[p + ".v"] @ h).reshape(H, V)
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = rotate_half(q, pos, base, dims)
    k = rotate_half(k, pos, base, dims) * float(D) ** -0.5
    o = np.empty((H, V), h.dtype)
    for n in range(H):
        st.s[n], o[n] = decayed_recurrence(st.s[n], m["decay"][n], k[n], v[n], q[n])
    return w[p + ".o"] @ (rms(o, eps).reshape(-1) * silu(w[p + ".g"] @ h))


def mamba2(m, w, p, h, st, eps):
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    u = w[p + ".in"] @ h
    z, xbc, dt = u[:inner], u[inner:2 * inner + 2 * G * N], u[2 * inner + 2 * G * N:]
    history = np.concatenate([st.tail, xbc[None]], axis=0)
    st.tail = history[1:]
    xbc = silu(causal_conv(history, w[p + ".conv"], w[p + ".conv.b"]))
    x = xbc[:inner].reshape(H, V)
    B = xbc[inner:inner + G * N].reshape(G, N)
    C = xbc[inner + G * N:].reshape(G, N)
    dt = softplus(dt + w[p + ".dt_bias"])
    y = np.empty((H, V), h.dtype)
    for n in range(H):
        g = n // (H // G)
        decay = np.exp(-np.exp(w[p + ".A_log"][n]) * dt[n])
        st.s[n], y[n] = decayed_recurrence(st.s[n], decay, dt[n] * B[g], x[n], C[g])
        y[n] += w[p + ".D"][n] * x[n]
    y = y.reshape(-1) * silu(z)
    y = rms(y.reshape(m["norm_groups"], -1), eps).reshape(-1) * w[p + ".norm"]
    return w[p + ".o"] @ y


def latent_append(m, w, p, h, pos, st, eps):
    """Adds this token's latent and rotated key part to the layer's own cache."""
    R, r = m["kv_rank"], m["rot_dim"]
    u = w[p + ".dkv"] @ h
    st.c.append(rms(u[:R], eps) * w[p + ".dkv.norm"])
    st.r.append(rotate_interleaved(u[R:R + r], pos, m["rot"]["base"], m["rot"]["dims"]))


def latent_attention(m, w, p, h, pos, st, eps):
    """st: the cache of the layer whose latents are used; its newest entry is this token's."""
    H, D, r, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    cq = rms(w[p + ".dq"] @ h, eps) * w[p + ".dq.norm"]
    q = (w[p + ".uq"] @ cq).reshape(H, D + r)
    q_rot = rotate_interleaved(q[:, D:], pos, m["rot"]["base"], m["rot"]["dims"])
    c, kr = np.array(st.c), np.array(st.r)
    k = (c @ w[p + ".uk"].T).reshape(-1, H, D)
    v = (c @ w[p + ".uv"].T).reshape(-1, H, V)
    o = np.empty((H, V), h.dtype)
    for n in range(H):
        s = (k[:, n] @ q[n, :D] + kr @ q_rot[n]) * m["scale"]
        s = np.exp(s - s.max())
        o[n] = (s / s.sum()) @ v[:, n]
    return w[p + ".o"] @ o.reshape(-1)


def feed_forward(w, p, h):
    return w[p + ".down"] @ (silu(w[p + ".gate"] @ h) * (w[p + ".up"] @ h))


STATES = {"retention": RetentionState, "mamba2": Mamba2State, "latent_attention": LatentState}


class Model:
    """Runs one sequence token by token."""

    def __init__(self, config, weights, dtype=np.float64):
        self.cfg, self.dtype = config, dtype
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}
        self.reset()

    def reset(self):
        self.pos = 0
        self.states = [STATES[layer["type"]](layer["mixer"], self.dtype) for layer in self.cfg["layers"]]

    def layer(self, i, x):
        layer, w, eps = self.cfg["layers"][i], self.w, self.cfg["norm"]["eps"]
        p, m, st = f"l{i}", layer["mixer"], self.states[i]
        h = dynamic_tanh(x, w, p + ".norm1")
        if layer["type"] == "retention":
            y = retention(m, w, p + ".mix", h, self.pos, st, eps)
        elif layer["type"] == "mamba2":
            y = mamba2(m, w, p + ".mix", h, st, eps)
        else:
            if m.get("kv_from") is None:
                latent_append(m, w, p + ".mix", h, self.pos, st, eps)
            else:
                st = self.states[m["kv_from"]]
            y = latent_attention(m, w, p + ".mix", h, self.pos, st, eps)
        x = x + dynamic_tanh(y, w, p + ".norm1b")
        if layer["mlp"] is not None:
            y = feed_forward(w, p + ".mlp", dynamic_tanh(x, w, p + ".norm2"))
            x = x + dynamic_tanh(y, w, p + ".norm2b")
        return x

    def token(self, tok):
        """Returns (logits, residual after every layer)."""
        x = self.w["embed"][tok]
        after = []
        for i in range(len(self.cfg["layers"])):
            x = self.layer(i, x)
            after.append(x)
        self.pos += 1
        return self.w["embed"] @ dynamic_tanh(x, self.w, "final.norm"), after

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
