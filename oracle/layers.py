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


# ---- mechanisms of Lilosun ------------------------------------------------------------------------------------------
# Notation: c = latent channel, n = state channel, e = value channel.

def softplus(z):
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


def layer_norm(x, w, eps):
    """Zero mean and unit variance over the last axis, times w; no bias."""
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w


def yarn_frequencies(dims, base, scaling):
    """(angle per position of every pair, factor of cos and sin).  ``scaling`` None: base^(-2i/dims) and 1."""
    i = np.arange(dims // 2)
    f = float(base) ** (-2.0 * i / dims)
    if scaling is None:
        return f, 1.0

    def pair_that_turns(times):   # (fractional) pair index that makes this many turns within the original length
        return dims * np.log(scaling["original"] / (2 * np.pi * times)) / (2 * np.log(base))

    lo = max(np.floor(pair_that_turns(scaling["fast"])), 0)
    hi = min(np.ceil(pair_that_turns(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0, 1)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * np.log(scaling["factor"]) + 1


def rotate_pairs(x, positions, frequencies, gain):
    """x [tokens, heads, dim]: the pairs (2i, 2i+1) turn by position * frequencies[i] and grow by ``gain``; the rest passes."""
    out = x.copy()
    for i, f in enumerate(frequencies):
        a = np.asarray(positions, np.float64) * f
        c, s = (gain * np.cos(a)).astype(x.dtype)[:, None], (gain * np.sin(a)).astype(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def latent_attention(h, w, heads, dim, rot_dim, vdim, rank, rot_base, scaling, scale, window, eps):
    """w: dict q, dkv, dkv.norm, uk, uv, g, o.  Every head's keys and values are spelled out from the latent vector; the last
    rot_dim key channels, rotated, are common to the heads."""
    T = h.shape[0]
    pos = np.arange(T)
    f, gain = yarn_frequencies(rot_dim, rot_base, scaling)
    q = linear(w["q"], h).reshape(T, heads, dim + rot_dim)
    q_rot = rotate_pairs(q[:, :, dim:], pos, f, gain)
    down = linear(w["dkv"], h)
    c = unit_rms(down[:, :rank], eps) * w["dkv.norm"]
    k_rot = rotate_pairs(down[:, None, rank:], pos, f, gain)[:, 0]
    k = linear(w["uk"], c).reshape(T, heads, dim)
    v = linear(w["uv"], c).reshape(T, heads, vdim)
    o = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        o[:, n] = window_softmax(np.concatenate([q[:, n, :dim], q_rot[:, n]], -1), np.concatenate([k[:, n], k_rot], -1), v[:, n], scale, window)
    return linear(w["o"], o.reshape(T, heads * vdim) * sigmoid(linear(w["g"], h)))


def causal_conv(x, w, b):
    """Per channel: y_t = b + sum_j w[:, j] x_(t - taps + 1 + j), zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    past = np.concatenate([np.zeros((taps - 1, x.shape[1]), x.dtype), x])
    y = np.zeros_like(x) + b
    for j in range(taps):
        y = y + w[:, j] * past[j:j + T]
    return y


def ssd_scan(x, B, C, dt, a_log, state):
    """One head.  S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t B_t x_t^T, y_t = S_t^T C_t.  -> (y [T, vdim], S)."""
    S = state.copy()
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(-np.exp(a_log) * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        y[t] = S.T @ C[t]
    return y, S


def grouped_unit_rms(x, groups, eps):
    T, n = x.shape
    return unit_rms(x.reshape(T, groups, n // groups), eps).reshape(T, n)


def mamba2(h, w, heads, vdim, state, groups, norm_groups, eps):
    """w: dict in, conv, conv.b, dt_bias, A_log, D, norm, o."""
    T, inner, gn = h.shape[0], heads * vdim, groups * state
    p = linear(w["in"], h)
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * gn], p[:, 2 * inner + 2 * gn:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].reshape(T, heads, vdim)
    B = xbc[:, inner:inner + gn].reshape(T, groups, state)
    C = xbc[:, inner + gn:].reshape(T, groups, state)
    dt = softplus(dt + w["dt_bias"])
    y = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        g = n // (heads // groups)
        y[:, n] = ssd_scan(x[:, n], B[:, g], C[:, g], dt[:, n], w["A_log"][n], np.zeros((state, vdim), h.dtype))[0] + w["D"][n] * x[:, n]
    return linear(w["o"], grouped_unit_rms(y.reshape(T, inner) * silu(z), norm_groups, eps) * w["norm"])


def silu_mlp(x, gate, up, down):
    return linear(down, silu(linear(gate, x)) * linear(up, x))


def clamped_mlp(x, gate, up, down, limit):
    """g sigmoid(1.702 g) (u + 1) with g cut from above and u on both sides."""
    g, u = np.minimum(linear(gate, x), limit), np.clip(linear(up, x), -limit, limit)
    return linear(down, g * sigmoid(1.702 * g) * (u + 1))


def route(z, correction, top, groups, keep):
    """Router logits [tokens, experts] -> (chosen experts [tokens, top], their weights).  Groups of neighbouring experts compete
    by the sum of their two best corrected scores; the weights are the plain scores of the chosen, brought to sum 1."""
    s = sigmoid(z)
    choice = s + correction
    T, E = z.shape
    n = E // groups
    ids = np.zeros((T, top), np.int64)
    for t in range(T):
        best = [np.sort(choice[t, g * n:(g + 1) * n])[-2:].sum() for g in range(groups)]
        kept = set(np.argsort(best)[::-1][:keep].tolist())
        allowed = [(choice[t, e], -e) for e in range(E) if e // n in kept]
        ids[t] = [-e for _, e in sorted(allowed, reverse=True)[:top]]
    w = np.take_along_axis(s, ids, 1)
    return ids, w / (w.sum(-1, keepdims=True) + 1e-20)


def route_margin(z, correction, top, groups, keep):
    """By how much the choice scores of every token would have to move to change what ``route`` chooses: the gap behind the
    last group that is kept, or behind the last expert that is chosen."""
    choice = sigmoid(z) + correction
    n = z.shape[1] // groups
    out = np.full(z.shape[0], np.inf)
    for t in range(z.shape[0]):
        best = np.array([np.sort(choice[t, g * n:(g + 1) * n])[-2:].sum() for g in range(groups)])
        order = np.argsort(best)[::-1]
        if keep < groups:
            out[t] = (best[order[keep - 1]] - best[order[keep]]) / 2
        c = np.sort(np.concatenate([choice[t, g * n:(g + 1) * n] for g in order[:keep]]))[::-1]
        if top < len(c):
            out[t] = min(out[t], c[top - 1] - c[top])
    return out


def moe(h, w, top, groups, keep, limit, shared_limit):
    """w: dict router, correction, e<i>.gate/up/down and, with a shared expert, shared.gate/up/down/sg."""
    ids, weights = route(linear(w["router"], h), w["correction"], top, groups, keep)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t], weights[t]):
            n = f"e{e}."
            out[t] += p * clamped_mlp(h[t], w[n + "gate"], w[n + "up"], w[n + "down"], limit)
    if shared_limit is not None:
        out = out + sigmoid(linear(w["shared.sg"], h)) * clamped_mlp(h, w["shared.gate"], w["shared.up"], w["shared.down"], shared_limit)
    return out


class Lilosun:
    """The whole design from a config dict and a dict of float arrays under the checkpoint's tensor names."""

    def __init__(self, config: dict, tensors: dict, dtype=np.float64):
        self.c = config
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.margin = None    # per token of the last forward: the closest call of any router

    def part(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def mixer(self, i, layer, h):
        w, m, eps = self.part(f"l{i}.mix."), layer["mixer"], self.c["norm"]["eps"]
        if layer["type"] == "latent_attention":
            rot, mask = m["rot"], m.get("mask")
            return latent_attention(h, w, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], rot["base"], rot.get("scaling"), m["scale"],
                                    mask["size"] if mask else None, eps)
        if layer["type"] == "mamba2":
            return mamba2(h, w, m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"], eps)
        raise ValueError(f"unknown mixer {layer['type']}")

    def feed_forward(self, i, mlp, h):
        w = self.part(f"l{i}.mlp.")
        if mlp["kind"] == "dense":
            return silu_mlp(h, w["gate"], w["up"], w["down"])
        r, g = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}
        shared = mlp.get("shared")
        self.margin = np.minimum(self.margin, route_margin(linear(w["router"], h), w["correction"], r["top"], g["count"], g["keep"]))
        return moe(h, w, r["top"], g["count"], g["keep"], mlp["expert"]["limit"], shared["limit"] if shared else None)

    def forward(self, tokens, layer_outputs: list | None = None):
        """Logits [tokens, vocab] of one sequence from its first token."""
        eps = self.c["norm"]["eps"]
        x = self.t["embed"][np.asarray(tokens)]
        self.margin = np.full(len(tokens), np.inf)
        for i, layer in enumerate(self.c["layers"]):
            l = f"l{i}."
            x = x + self.t[l + "ls1"] * self.mixer(i, layer, layer_norm(x, self.t[l + "norm1"], eps))
            if layer.get("mlp"):
                x = x + self.t[l + "ls2"] * self.feed_forward(i, layer["mlp"], layer_norm(x, self.t[l + "norm2"], eps))
            if layer_outputs is not None:
                layer_outputs.append(x.copy())
        return linear(self.t["head"], layer_norm(x, self.t["final.norm"], eps)) * self.c["logit_scale"]


# ---- mechanisms of Rubuvik ------------------------------------------------------------------------------------------

def rms_around_one(x, w, eps):
    """Unit root mean square, times 1 + w: the stored weight says by how much a channel differs from 1."""
    return unit_rms(x, eps) * (1 + w)


def distance_slopes(heads):
    """How much a head takes off a score per token of distance: 2^(-8 (n + 1) / heads), n = 0, 1, ..."""
    return 2.0 ** (-8.0 * (np.arange(heads) + 1) / heads)


def query_temperature(positions, coef, every):
    """1 + coef ln(1 + number of whole stretches of ``every`` tokens up to and with the position)."""
    return 1 + coef * np.log(np.floor((np.asarray(positions, np.float64) + 1) / every) + 1)


def biased_window_softmax(q, k, v, scale, slope, window, sink=None):
    """One head: scores scale (q_t . k_s) - slope (t - s) over 0 <= t - s < window; ``sink`` adds exp(sink) to the sum of weights."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        lo = 0 if window is None else max(0, t - window + 1)
        s = (k[lo:t + 1] @ q[t]) * scale - slope * (t - np.arange(lo, t + 1))
        top = s.max() if sink is None else max(s.max(), sink)
        p = np.exp(s - top)
        out[t] = (p @ v[lo:t + 1]) / (p.sum() + (0 if sink is None else np.exp(sink - top)))
    return out


def mixed_values(v, first, lam):
    """Values drawn towards those that the first layer of the kind gave the same token."""
    return (1 - lam) * v + lam * first


def biased_attention(h, w, heads, kv_heads, dim, vdim, scale, window, eps, temperature=None, biases=False, unit_qk=False, sink=False, gate=False,
                     first=None):
    """w: dict q, k, v, o and what the options need (q.b, k.b, v.b; sink; g; vmix).  ``temperature``: (coef, every).  ``first``: the first
    layer's values [T, kv_heads, vdim] to mix in.  -> (output, this layer's values before mixing)."""
    T = h.shape[0]

    def part(name, n, d):
        return (linear(w[name], h) + (w[name + ".b"] if biases else 0)).reshape(T, n, d)

    q, k, v = part("q", heads, dim), part("k", kv_heads, dim), part("v", kv_heads, vdim)
    own = v
    if unit_qk:
        q, k = unit_rms(q, eps), unit_rms(k, eps)
    if temperature is not None:
        q = q * query_temperature(np.arange(T), *temperature)[:, None, None].astype(q.dtype)
    if first is not None:
        v = mixed_values(v, first, w["vmix"])
    slopes = distance_slopes(heads)
    o = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        g = n // (heads // kv_heads)
        o[:, n] = biased_window_softmax(q[:, n], k[:, g], v[:, g], scale, slopes[n], window, w["sink"][n] if sink else None)
    if gate:
        o = o * sigmoid(linear(w["g"], h))[:, :, None]
    return linear(w["o"], o.reshape(T, heads * vdim)), own


def decayed_scan(q, k, v, decay, state):
    """One head.  S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  -> (o [T, vdim], S)."""
    S = state.copy()
    o = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o, S


def lightning(h, w, heads, dim, vdim, decay, eps):
    """w: dict q, k, v, g, o, norm.  The heads are normalised together, the gate follows the norm."""
    T = h.shape[0]
    q, k = silu(linear(w["q"], h)).reshape(T, heads, dim), silu(linear(w["k"], h)).reshape(T, heads, dim)
    v = silu(linear(w["v"], h)).reshape(T, heads, vdim)
    o = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        o[:, n] = decayed_scan(q[:, n], k[:, n], v[:, n], decay[n], np.zeros((dim, vdim), h.dtype))[0]
    return linear(w["o"], unit_rms(o.reshape(T, heads * vdim), eps) * w["norm"] * sigmoid(linear(w["g"], h)))


def softmax_scores(z):
    p = np.exp(z - z.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def route_softmax(z, correction, top, groups, keep, scale):
    """Router logits [tokens, experts] -> (chosen experts [tokens, top], their weights).  Groups of neighbouring experts compete
    by their best corrected score; the weights are the plain scores of the chosen times ``scale``."""
    s = softmax_scores(z)
    choice = s + correction
    T, E = z.shape
    n = E // groups
    ids = np.zeros((T, top), np.int64)
    for t in range(T):
        best = choice[t].reshape(groups, n).max(-1)
        kept = np.argsort(-best, kind="stable")[:keep]
        masked = np.full(E, -np.inf)
        for g in kept:
            masked[g * n:(g + 1) * n] = choice[t, g * n:(g + 1) * n]
        ids[t] = np.argsort(-masked, kind="stable")[:top]
    return ids, np.take_along_axis(s, ids, 1) * scale


def route_softmax_margin(z, correction, top, groups, keep):
    """As route_margin, for ``route_softmax``."""
    choice = softmax_scores(z) + correction
    out = np.full(z.shape[0], np.inf)
    for t in range(z.shape[0]):
        by_group = choice[t].reshape(groups, -1)
        order = np.argsort(-by_group.max(-1))
        if keep < groups:
            best = by_group.max(-1)
            out[t] = best[order[keep - 1]] - best[order[keep]]
        c = np.sort(by_group[order[:keep]].ravel())[::-1]
        if top < len(c):
            out[t] = min(out[t], c[top - 1] - c[top])
    return out


def softmax_moe(h, w, top, groups, keep, scale, shared):
    """w: dict router, correction, e<i>.gate/up/down and, with a shared expert, shared.gate/up/down."""
    ids, weights = route_softmax(linear(w["router"], h), w["correction"], top, groups, keep, scale)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t], weights[t]):
            n = f"e{e}."
            out[t] += p * silu_mlp(h[t], w[n + "gate"], w[n + "up"], w[n + "down"])
    if shared:
        out = out + silu_mlp(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return out


def token_side(x, e, w, eps):
    """What a layer's own row of the token table adds: w: dict gate, proj, norm; e [tokens, dim]."""
    return unit_rms(linear(w["proj"], gelu_tanh(linear(w["gate"], x)) * e), eps) * w["norm"]


class Rubuvik:
    """The whole design from a config dict and a dict of float arrays under the checkpoint's tensor names."""

    def __init__(self, config: dict, tensors: dict, dtype=np.float64):
        self.c = config
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.margin = None    # per token of the last forward: the closest call of any router

    def part(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def norm(self, name, x):
        return rms_around_one(x, self.t[name], self.c["norm"]["eps"])

    def mixer(self, i, layer, h):
        w, m, eps = self.part(f"l{i}.mix."), layer["mixer"], self.c["norm"]["eps"]
        if layer["type"] == "lightning":
            return lightning(h, w, m["heads"], m["dim"], m["vdim"], m["decay"], eps)
        more = {"attention": {}, "attention_2": dict(biases=True, unit_qk=True, sink=True, gate=True)}[layer["type"]]
        mask, temp, mix = m.get("mask"), m.get("q_temp"), m.get("v_mix", False)
        y, v = biased_attention(h, w, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], mask["size"] if mask else None, eps,
                                temperature=(temp["coef"], temp["every"]) if temp else None, first=self.first_values if mix else None, **more)
        if mix and self.first_values is None:
            self.first_values = v
        return y

    def feed_forward(self, i, mlp, h):
        w = self.part(f"l{i}.mlp.")
        if mlp["kind"] == "dense":
            return silu_mlp(h, w["gate"], w["up"], w["down"])
        r, g = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}
        self.margin = np.minimum(self.margin, route_softmax_margin(linear(w["router"], h), w["correction"], r["top"], g["count"], g["keep"]))
        return softmax_moe(h, w, r["top"], g["count"], g["keep"], r["scale"], bool(mlp.get("shared")))

    def forward(self, tokens, layer_outputs: list | None = None):
        """Logits [tokens, vocab] of one sequence from its first token."""
        tokens, eps, m, side = np.asarray(tokens), self.c["norm"]["eps"], self.c["residual_mult"], self.c["token_side"]
        x = self.t["embed"][tokens] * self.c["embedding"]["scale"]
        self.margin = np.full(len(tokens), np.inf)
        self.first_values = None
        for i, layer in enumerate(self.c["layers"]):
            l = f"l{i}."
            x = x + m * self.norm(l + "norm1b", self.mixer(i, layer, self.norm(l + "norm1", x)))
            if layer.get("mlp"):
                x = x + m * self.norm(l + "norm2b", self.feed_forward(i, layer["mlp"], self.norm(l + "norm2", x)))
            if side:
                d = side["dim"]
                x = x + m * token_side(x, self.t["side.embed"][tokens, i * d:(i + 1) * d], self.part(l + "side."), eps)
            if layer_outputs is not None:
                layer_outputs.append(x.copy())
        return linear(self.t["embed"], self.norm("final.norm", x))


# ---- mechanisms of Noresun ------------------------------------------------------------------------------------------

def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the table of token pairs for every token of a sequence; the last row, number ``buckets``, for the first token."""
    t = [int(x) for x in tokens]
    return np.array([buckets] + [(t[i - 1] * mul_prev + t[i] * mul_cur) % buckets for i in range(1, len(t))], np.int64)


def banded_frequencies(dims, base, scaling):
    """Angle per position of every pair.  ``scaling``: pairs with a wavelength under original / high keep theirs, those over
    original / low are slowed by ``factor``, those in between are blended by where original / wavelength lies between the two."""
    f = float(base) ** (-2.0 * np.arange(dims // 2) / dims)
    if scaling is None:
        return f
    out = f.copy()
    for i in range(len(f)):
        turns = scaling["original"] * f[i] / (2 * np.pi)          # within the original length
        if turns > scaling["high"]:
            continue
        if turns < scaling["low"]:
            out[i] = f[i] / scaling["factor"]
        else:
            s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
            out[i] = (1 - s) * f[i] / scaling["factor"] + s * f[i]
    return out


def window_sigmoid(q, k, v, scale, bias, window):
    """One head: every visible key weighs sigmoid(scale (q_t . k_s) + bias), whatever the others weigh; 0 <= t - s < window."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        lo = 0 if window is None else max(0, t - window + 1)
        out[t] = sigmoid((k[lo:t + 1] @ q[t]) * scale + bias) @ v[lo:t + 1]
    return out


def keys_and_values(h, w, kv_heads, dim, vdim, frequencies, eps):
    """k normalised over the whole projection, then rotated; v as it is."""
    T = h.shape[0]
    k = (unit_rms(linear(w["k"], h), eps) * w["k.norm"]).reshape(T, kv_heads, dim)
    return rotate_pairs(k, np.arange(T), frequencies, 1.0), linear(w["v"], h).reshape(T, kv_heads, vdim)


def sigmoid_attention(h, w, heads, dim, frequencies, scale, window, eps, k, v):
    """w: dict q, q.norm, pb, o; k, v: of this layer or of the one it shares them with."""
    T, kv_heads, vdim = v.shape
    q = (unit_rms(linear(w["q"], h), eps) * w["q.norm"]).reshape(T, heads, dim)
    q = rotate_pairs(q, np.arange(T), frequencies, 1.0)
    o = np.zeros((T, heads, vdim), h.dtype)
    for n in range(heads):
        g = n // (heads // kv_heads)
        o[:, n] = window_sigmoid(q[:, n], k[:, g], v[:, g], scale, w["pb"][n], window)
    return linear(w["o"], o.reshape(T, heads * vdim))


def positive_candidate(u):
    """u + 1/2 from zero up, sigmoid(u) below: positive and continuous."""
    return np.where(u >= 0, u + 0.5, sigmoid(u))


def min_gru_scan(z, candidate, state):
    """S_t = (1 - z_t) S_(t-1) + z_t candidate_t, element by element.  -> (S of every token, the last S)."""
    S = state.copy()
    out = np.zeros_like(z)
    for t in range(z.shape[0]):
        S = (1 - z[t]) * S + z[t] * candidate[t]
        out[t] = S
    return out, S


def min_gru(h, w):
    """w: dict z, z.b, x, x.b, g, o."""
    z, u = sigmoid(linear(w["z"], h) + w["z.b"]), linear(w["x"], h) + w["x.b"]
    s, _ = min_gru_scan(z, positive_candidate(u), np.zeros(z.shape[1], h.dtype))
    return linear(w["o"], s * silu(linear(w["g"], h)))


def route_chosen(z, top):
    """Router logits [tokens, experts] -> (the ``top`` largest [tokens, top], softmax over these alone)."""
    ids = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return ids, softmax_scores(np.take_along_axis(z, ids, 1))


def relu2_moe(h, w, top):
    """w: dict router, router.b, e<i>.up/down."""
    ids, weights = route_chosen(linear(w["router"], h) + w["router.b"], top)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t], weights[t]):
            out[t] += p * linear(w[f"e{e}.down"], np.maximum(linear(w[f"e{e}.up"], h[t]), 0) ** 2)
    return out


class Noresun:
    """The whole design from a config dict and a dict of float arrays under the checkpoint's tensor names."""

    def __init__(self, config: dict, tensors: dict, dtype=np.float64):
        self.c = config
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.margin = None    # per token of the last forward: the closest call of any router, in logits

    def part(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def embed(self, tokens):
        e = self.c["embedding"]
        x = self.t["embed"][tokens] * e["scale"]
        if e.get("bigram"):
            b = e["bigram"]
            x = x + self.t["bigram"][bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]
        return x

    def mixer(self, i, layer, h):
        w, m, eps = self.part(f"l{i}.mix."), layer["mixer"], self.c["norm"]["eps"]
        if layer["type"] == "mingru":
            return min_gru(h, w)
        if layer["type"] != "attention":
            raise ValueError(f"unknown mixer {layer['type']}")
        rot, mask = m.get("rot"), m.get("mask")
        f = banded_frequencies(rot["dims"], rot["base"], rot.get("scaling")) if rot else []
        if m.get("kv_from") is None:
            self.kv[i] = keys_and_values(h, w, m["kv_heads"], m["dim"], m["vdim"], f, eps)
        k, v = self.kv[i if m.get("kv_from") is None else m["kv_from"]]
        return sigmoid_attention(h, w, m["heads"], m["dim"], f, m["scale"], mask["size"] if mask else None, eps, k, v)

    def feed_forward(self, i, mlp, h):
        w, top = self.part(f"l{i}.mlp."), mlp["router"]["top"]
        if mlp["kind"] != "moe":
            raise ValueError(f"unknown feed-forward {mlp['kind']}")
        z = np.sort(linear(w["router"], h) + w["router.b"], axis=-1)[:, ::-1]
        if top < z.shape[1]:
            self.margin = np.minimum(self.margin, z[:, top - 1] - z[:, top])
        return relu2_moe(h, w, top)

    def forward(self, tokens, layer_outputs: list | None = None):
        """Logits [tokens, vocab] of one sequence from its first token."""
        tokens, eps, alpha = np.asarray(tokens), self.c["norm"]["eps"], self.c["postln_alpha"]
        x = self.embed(tokens)
        self.margin = np.full(len(tokens), np.inf)
        self.kv = {}

        def after(name, x, gate, y):
            y = y * sigmoid(linear(self.t[gate], x) + self.t[gate + ".b"])
            return unit_rms(alpha * x + y, eps) * self.t[name]

        for i, layer in enumerate(self.c["layers"]):
            l = f"l{i}."
            x = after(l + "norm1", x, l + "rg1", self.mixer(i, layer, x))
            if layer.get("mlp"):
                x = after(l + "norm2", x, l + "rg2", self.feed_forward(i, layer["mlp"], x))
            if layer_outputs is not None:
                layer_outputs.append(x.copy())
        return linear(self.t["embed"], unit_rms(x, eps) * self.t["final.norm"])
