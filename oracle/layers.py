"""Plain, slow reference of the mechanisms of layered decoder designs (numpy), one function per mechanism.

Test infrastructure: it shares no code with the CUDA library and is written token by token from the equations,
so that an error of the chunked, paged or batched product path cannot also be an error here.  Arrays are
[tokens, features]; ``dtype`` float64 gives a reference far below float32 rounding, float32 the product's own
32-bit arithmetic.  Notation: t = token, d = key channel, e = value channel.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1 / (1 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1 + np.exp(-np.abs(z))))


def log_sigmoid(z):
    return np.minimum(z, 0) - np.log1p(np.exp(-np.abs(z)))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    """x / sqrt(mean x^2 + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dyt_norm(x, alpha, w, b):
    """Dynamic Tanh: tanh(alpha x) w + b, no statistics."""
    return np.tanh(alpha * x) * w + b


def linear(w, x):
    return x @ w.T


def gated_mlp(x, gate, up, down):
    return linear(down, gelu_tanh(linear(gate, x)) * linear(up, x))


def rotate_interleaved(x, positions, dims, base):
    """x [tokens, heads, dim]: the pairs (2i, 2i+1), i < dims/2, turn by position * base^(-2i/dims); the rest passes."""
    out = x.copy()
    for i in range(dims // 2):
        a = np.asarray(positions, np.float64) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(a).astype(x.dtype)[:, None], np.sin(a).astype(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def window_softmax(q, k, v, scale, window):
    """One head, one map: token t sees the tokens s with 0 <= t - s < window (all s <= t if window is None)."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        lo = 0 if window is None else max(0, t - window + 1)
        s = (k[lo:t + 1] @ q[t]) * scale
        p = np.exp(s - s.max())
        out[t] = (p / p.sum()) @ v[lo:t + 1]
    return out


def differential_lambda(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff


def differential_attention(h, w, heads, kv_heads, dim, vdim, rot_dims, rot_base, scale, window, diff, eps):
    """w: dict q, k, v, o, lq1, lk1, lq2, lk2.  Two attention maps per head over the same values; the second is
    subtracted lambda times, the difference is scaled to unit root mean square and by 1 - diff."""
    T = h.shape[0]
    pos = np.arange(T)
    q = rotate_interleaved(linear(w["q"], h).reshape(T, heads * 2, dim), pos, rot_dims, rot_base)
    k = rotate_interleaved(linear(w["k"], h).reshape(T, kv_heads * 2, dim), pos, rot_dims, rot_base)
    v = linear(w["v"], h).reshape(T, kv_heads, vdim)
    lam = differential_lambda(w["lq1"], w["lk1"], w["lq2"], w["lk2"], diff)
    o = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        g = n // (heads // kv_heads)
        a = [window_softmax(q[:, 2 * n + j], k[:, 2 * g + j], v[:, g], scale, window) for j in (0, 1)]
        o[:, n] = unit_rms(a[0] - lam * a[1], eps) * (1 - diff)
    return linear(w["o"], o.reshape(T, heads * vdim))


def gla_scan(q, k, v, log_decay, state):
    """One head.  S_t = diag(exp(log_decay_t)) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  -> (o [T, vdim], S)."""
    S = state.copy()
    o = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        S = np.exp(log_decay[t])[:, None] * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o, S


def gla(h, w, heads, dim, vdim, tau, eps):
    """w: dict q, k, v, g, o, norm, a1, a2, a2.b."""
    T = h.shape[0]
    q = linear(w["q"], h).reshape(T, heads, dim) * dim ** -0.5
    k = linear(w["k"], h).reshape(T, heads, dim)
    v = linear(w["v"], h).reshape(T, heads, vdim)
    z = (linear(w["a2"], linear(w["a1"], h)) + w["a2.b"]).reshape(T, heads, dim)
    o = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        o[:, n], _ = gla_scan(q[:, n], k[:, n], v[:, n], log_sigmoid(z[:, n]) / tau, np.zeros((dim, vdim), h.dtype))
    o = unit_rms(o, eps) * w["norm"]
    return linear(w["o"], o.reshape(T, heads * vdim) * silu(linear(w["g"], h)))


def mlstm_scan(q, k, v, log_i, log_f, state, n, m):
    """One head.  m_t = max(f + m, i); S, n decay by exp(f + m - m_t) and take exp(i - m_t) k (v^T, 1);
    o = S^T q / (max(|n.q|, exp(-m_t)) + 1e-6).  -> (o, S, n, m)."""
    S, n = state.copy(), n.copy()
    o = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        m_new = max(log_f[t] + m, log_i[t])
        keep, put = np.exp(log_f[t] + m - m_new), np.exp(log_i[t] - m_new)
        S = keep * S + put * np.outer(k[t], v[t])
        n = keep * n + put * k[t]
        m = m_new
        o[t] = (S.T @ q[t]) / (max(abs(n @ q[t]), np.exp(-m)) + 1e-6)
    return o, S, n, m


def mlstm_gates(h, w, cap):
    """(log input gate, log forget gate), each [tokens, heads]."""
    i = cap * np.tanh((linear(w["i"], h) + w["i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((linear(w["f"], h) + w["f.b"]) / cap))
    return i, f


def mlstm(h, w, heads, dim, vdim, cap, eps):
    """w: dict q, k, v, g, o, norm, i, i.b, f, f.b."""
    T = h.shape[0]
    q = linear(w["q"], h).reshape(T, heads, dim) * dim ** -0.5
    k = linear(w["k"], h).reshape(T, heads, dim)
    v = linear(w["v"], h).reshape(T, heads, vdim)
    i, f = mlstm_gates(h, w, cap)
    o = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        o[:, n] = mlstm_scan(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n], np.zeros((dim, vdim), h.dtype), np.zeros(dim, h.dtype), 0.0)[0]
    o = unit_rms(o, eps).reshape(T, heads * vdim) * w["norm"]
    return linear(w["o"], o * sigmoid(linear(w["g"], h)))


class Sumosun:
    """The whole design from a config dict and a dict of float arrays under the checkpoint's tensor names."""

    def __init__(self, config: dict, tensors: dict, dtype=np.float64):
        self.c = config
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.dtype = dtype

    def norm(self, name, x):
        return dyt_norm(x, self.t[name + ".alpha"], self.t[name], self.t[name + ".b"])

    def mixer(self, i, layer, h):
        p = f"l{i}.mix."
        w = {k[len(p):]: v for k, v in self.t.items() if k.startswith(p)}
        m, eps = layer["mixer"], self.c["norm"]["eps"]
        if layer["type"] == "attention":
            return differential_attention(h, w, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]["dims"], m["rot"]["base"],
                                          m["scale"], m["mask"]["size"], m["diff"], eps)
        if layer["type"] == "gla":
            return gla(h, w, m["heads"], m["dim"], m["vdim"], m["tau"], eps)
        if layer["type"] == "mlstm":
            return mlstm(h, w, m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps)
        raise ValueError(f"unknown mixer {layer['type']}")

    def forward(self, tokens, layer_outputs: list | None = None):
        """Logits [tokens, vocab] of one sequence from its first token."""
        x = self.t["embed"][np.asarray(tokens)]
        for i, layer in enumerate(self.c["layers"]):
            l = f"l{i}"
            x = x + self.norm(l + ".norm1b", self.mixer(i, layer, self.norm(l + ".norm1", x)))
            if layer.get("mlp"):
                h = self.norm(l + ".norm2", x)
                x = x + self.norm(l + ".norm2b", gated_mlp(h, self.t[l + ".mlp.gate"], self.t[l + ".mlp.up"], self.t[l + ".mlp.down"]))
            if layer_outputs is not None:
                layer_outputs.append(x.copy())
        return linear(self.t["embed"], self.norm("final.norm", x))
