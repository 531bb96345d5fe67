"""Small random checkpoints of the layered designs for the tests: configurations, tensors under the checkpoint's names
(values that bf16 represents exactly), the plain reference over them, and a writer for checkpoint folders."""
from __future__ import annotations

import json
import struct

import numpy as np

from paged_infer_b200.loader import LayeredConfig, bf16_bits_to_f32, f32_to_bf16_bits


def attention(heads=4, kv_heads=2, dim=16, vdim=32, window=24, rot=None, base=10000.0, diff=0.3, scale=None, ff=48):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": dim ** -0.5 if scale is None else scale,
                      "mask": {"size": window}, "rot": {"dims": dim if rot is None else rot, "base": base}}}


def gla(heads=3, dim=16, vdim=24, tau=8.0, ff=0):
    return {"type": "gla", "mlp": {"kind": "dense", "ff": ff} if ff else None, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def mlstm(heads=2, dim=24, vdim=40, cap=10.0, ff=0):
    return {"type": "mlstm", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def config(layers, width=64, vocab=96, eps=1e-5):
    return {"architecture": "Sumosun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# ---- Lilosun ------------------------------------------------------------------------------------------------------------------
YARN = {"factor": 8.0, "original": 96, "fast": 20.0, "slow": 2.0}


def latent(heads=3, dim=20, rot_dim=16, vdim=24, rank=48, window=28, base=10000.0, scaling=YARN, scale=None, mlp=None):
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = scaling
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": rot,
                      "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "mask": {"size": window} if window else None}}


def mamba2(heads=6, vdim=20, state=24, groups=2, norm_groups=3, conv=3, mlp=None):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=3, ff=40, limit=1.2, groups=(3, 2), shared=56, shared_limit=0.8):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared, "limit": shared_limit} if shared else None}


def lilosun(layers, width=88, vocab=400, eps=1e-5, logit_scale=1.5):
    return {"architecture": "Lilosun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": logit_scale}


# ---- Rubuvik ------------------------------------------------------------------------------------------------------------------
def biased(heads=6, kv_heads=2, dim=20, vdim=28, window=30, scale=None, v_mix=True, temp=(0.4, 9), mlp=None):
    """'attention': distance bias and query temperature."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "v_mix": v_mix,
         "mask": {"size": window} if window else None}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def sunk(heads=6, kv_heads=2, dim=20, vdim=28, window=30, scale=None, v_mix=True, mlp=None):
    """'attention_2': distance bias, biases, unit queries and keys, sink and gate per head."""
    return dict(biased(heads, kv_heads, dim, vdim, window, 3.0 * dim ** -0.5 if scale is None else scale, v_mix, None, mlp), type="attention_2")


def lightning(heads=4, dim=24, vdim=20, decay=(0.5, 0.83, 0.97, 0.998), mlp=None):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def softmax_moe(experts=12, top=3, ff=40, groups=(3, 2), shared=56, scale=1.7):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def rubuvik(layers, width=84, vocab=400, eps=1e-5, embed_scale=3.0, mult=0.6, side=12):
    return {"architecture": "Rubuvik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "embedding": {"scale": embed_scale},
            "residual_mult": mult, "token_side": {"dim": side} if side else None}


def rubuvik_tensors(cfg, seed):
    """As lilosun_tensors: no sublayer writes the channels the routers read."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    t = {}

    def put(name, shape, std=None, mean=0.0):
        x = rng.standard_normal(shape) * (1.0 / np.sqrt(shape[-1]) if std is None else std) + mean
        t[name] = bf16_bits_to_f32(f32_to_bf16_bits(np.asarray(x, np.float32))).reshape(shape)

    def gated(p, F):
        put(p + "gate", (F, W), 2.0 / np.sqrt(W))
        put(p + "up", (F, W), 1.5 / np.sqrt(W))
        put(p + "down", (W, F), 1.2 / np.sqrt(F))
        t[p + "down"][:CODE] = 0

    put("embed", (V, W), 0.5, 0.05)
    side = (cfg["token_side"] or {}).get("dim", 0)
    if side:
        put("side.embed", (V, side * len(cfg["layers"])), 1.0)
    for i, e in enumerate(cfg["layers"]):
        m, l = e["mixer"], f"l{i}."
        p = l + "mix."
        H, D, E = m["heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b"):
            put(l + n, (W,), 0.2)
        if e["type"] == "lightning":
            put(p + "q", (H * D, W), 1.5 / np.sqrt(W))
            put(p + "k", (H * D, W), 1.5 / np.sqrt(W))
            put(p + "v", (H * E, W), 1.5 / np.sqrt(W))
            put(p + "g", (H * E, W), 1.5 / np.sqrt(W))
            put(p + "norm", (H * E,), 0.2, 1.0)
        else:
            G = m["kv_heads"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * E)):
                put(p + n, (rows, W), 1.5 / np.sqrt(W))
                if e["type"] == "attention_2":
                    put(p + n + ".b", (rows,), 0.5)
            if e["type"] == "attention_2":
                put(p + "sink", (H,), 1.5, 0.5)
                put(p + "g", (H, W), 2.0 / np.sqrt(W))
            if m["v_mix"]:
                put(p + "vmix", (), 0.05, 0.4)
        put(p + "o", (W, H * E))
        t[p + "o"][:CODE] = 0
        f = e["mlp"]
        if f:
            for n in ("norm2", "norm2b"):
                put(l + n, (W,), 0.2)
            p = l + "mlp."
            if f["kind"] == "dense":
                gated(p, f["ff"])
            else:
                n = f["router"]["experts"]
                put(p + "router", (n, W), 0.45)
                t[p + "router"][:, CODE:] = 0
                put(p + "correction", (n,), 0.15, -0.1)
                for k in range(n):
                    gated(f"{p}e{k}.", f["expert"]["ff"])
                if f.get("shared"):
                    gated(p + "shared.", f["shared"]["ff"])
        if side:
            put(l + "side.gate", (side, W), 1.5 / np.sqrt(W))
            put(l + "side.proj", (W, side))
            t[l + "side.proj"][:CODE] = 0
            put(l + "side.norm", (W,), 0.2, 0.7)
    put("final.norm", (W,), 0.2)
    return t


# ---- Noresun ------------------------------------------------------------------------------------------------------------------
BANDS = {"factor": 6.0, "low": 1.5, "high": 5.0, "original": 160}


def sigmoid_attention(heads=6, kv_heads=2, dim=20, vdim=28, window=30, rot=12, base=10000.0, scaling=BANDS, scale=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
         "mask": {"size": window} if window else None}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if scaling:
            m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def mingru(width=44, mlp=None):
    return {"type": "mingru", "mlp": mlp, "mixer": {"width": width}}


def relu2_moe(experts=12, top=3, ff=40):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def noresun(layers, width=84, vocab=400, eps=1e-5, embed_scale=3.0, alpha=1.7, bigram=(211, 5, 3)):
    e = {"scale": embed_scale}
    if bigram:
        e["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Noresun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "embedding": e, "postln_alpha": alpha}


def noresun_tensors(cfg, seed):
    """As lilosun_tensors: no sublayer and no token pair writes the channels the routers read."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    t = {}

    def put(name, shape, std=None, mean=0.0):
        x = rng.standard_normal(shape) * (1.0 / np.sqrt(shape[-1]) if std is None else std) + mean
        t[name] = bf16_bits_to_f32(f32_to_bf16_bits(np.asarray(x, np.float32))).reshape(shape)

    def norm_and_gate(l, n):
        put(f"{l}norm{n}", (W,), 0.2, 1.0)
        t[f"{l}norm{n}"][:CODE] = 1.25
        put(f"{l}rg{n}", (W, W), 1.5 / np.sqrt(W))
        put(f"{l}rg{n}.b", (W,), 0.7, 0.3)

    put("embed", (V, W), 0.5, 0.05)
    t["embed"][:, :CODE] *= 1.5
    if cfg["embedding"].get("bigram"):
        put("bigram", (cfg["embedding"]["bigram"]["buckets"] + 1, W), 1.0)
        t["bigram"][:, :CODE] = 0
    for i, e in enumerate(cfg["layers"]):
        m, l = e["mixer"], f"l{i}."
        p = l + "mix."
        norm_and_gate(l, 1)
        if e["type"] == "mingru":
            inner = m["width"]
            for n in ("z", "x", "g"):
                put(p + n, (inner, W), 1.5 / np.sqrt(W))
            put(p + "z.b", (inner,), 1.5, -1.5)
            put(p + "x.b", (inner,), 0.7)
        else:
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            inner = H * E
            put(p + "q", (H * D, W), 1.5 / np.sqrt(W))
            put(p + "q.norm", (H * D,), 0.3, 1.2)
            put(p + "pb", (H,), 0.7, -1.5)
            if m.get("kv_from") is None:
                put(p + "k", (G * D, W), 1.5 / np.sqrt(W))
                put(p + "k.norm", (G * D,), 0.3, 1.2)
                put(p + "v", (G * E, W))
        put(p + "o", (W, inner), 1.0 / np.sqrt(inner))
        t[p + "o"][:CODE] = 0
        f = e["mlp"]
        if f:
            norm_and_gate(l, 2)
            p = l + "mlp."
            n, F = f["router"]["experts"], f["expert"]["ff"]
            put(p + "router", (n, W), 1.2)
            t[p + "router"][:, CODE:] = 0
            put(p + "router.b", (n,), 0.6)
            for k in range(n):
                put(f"{p}e{k}.up", (F, W), 1.3 / np.sqrt(W))
                put(f"{p}e{k}.down", (W, F), 1.0 / np.sqrt(F))
                t[f"{p}e{k}.down"][:CODE] = 0
    put("final.norm", (W,), 0.2, 1.0)
    return t


CODE = 16   # leading channels of the embedding that only the routers and norms see change: no sublayer writes them


def lilosun_tensors(cfg, seed):
    """Random tensors on the bf16 grid.  Routers read the leading channels, which carry a code per token that no sublayer touches, so
    that (for the tokens of ``clear_tokens``) no choice hangs on a rounding."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    t = {}

    def put(name, shape, std=None, mean=0.0):
        x = rng.standard_normal(shape) * (1.0 / np.sqrt(shape[-1]) if std is None else std) + mean
        t[name] = bf16_bits_to_f32(f32_to_bf16_bits(np.asarray(x, np.float32))).reshape(shape)

    def gated(p, F):
        put(p + "gate", (F, W), 2.0 / np.sqrt(W))
        put(p + "up", (F, W), 1.5 / np.sqrt(W))
        put(p + "down", (W, F), 1.2 / np.sqrt(F))
        t[p + "down"][:CODE] = 0

    put("embed", (V, W), 1.0, 0.1)
    t["embed"][:, :CODE] *= 1.5
    for i, e in enumerate(cfg["layers"]):
        m, l = e["mixer"], f"l{i}."
        p = l + "mix."
        put(l + "norm1", (W,), 0.2, 1.0)
        put(l + "ls1", (W,), 0.2, 0.5)
        H, E = m["heads"], m["vdim"]
        if e["type"] == "latent_attention":
            D, R, K = m["dim"], m["rot_dim"], m["kv_rank"]
            put(p + "q", (H * (D + R), W), 1.5 / np.sqrt(W))
            put(p + "dkv", (K + R, W), 1.5 / np.sqrt(W))
            put(p + "dkv.norm", (K,), 0.2, 1.0)
            put(p + "uk", (H * D, K))
            put(p + "uv", (H * E, K))
            put(p + "g", (H * E, W))
        else:
            N, G = m["state"], m["groups"]
            ch = H * E + 2 * G * N
            put(p + "in", (H * E + ch + H, W))
            put(p + "conv", (ch, m["conv"]), 0.6)
            put(p + "conv.b", (ch,), 0.3)
            put(p + "dt_bias", (H,), 1.0, -2.0)
            put(p + "A_log", (H,), 1.0)
            put(p + "D", (H,), 0.5, 0.5)
            put(p + "norm", (H * E,), 0.2, 1.0)
        put(p + "o", (W, H * E), 1.5 / np.sqrt(H * E))
        t[p + "o"][:CODE] = 0
        f = e["mlp"]
        if f:
            put(l + "norm2", (W,), 0.2, 1.0)
            put(l + "ls2", (W,), 0.2, 0.5)
            p = l + "mlp."
            if f["kind"] == "dense":
                gated(p, f["ff"])
            else:
                n = f["router"]["experts"]
                put(p + "router", (n, W), 0.9)
                t[p + "router"][:, CODE:] = 0
                put(p + "correction", (n,), 0.3, -0.2)
                for k in range(n):
                    gated(f"{p}e{k}.", f["expert"]["ff"])
                if f.get("shared"):
                    gated(p + "shared.", f["shared"]["ff"])
                    put(p + "shared.sg", (1, W), 1.0 / np.sqrt(W))
    put("final.norm", (W,), 0.2, 1.0)
    put("head", (V, W))
    return t


def clear_tokens(cfg, t, margin=0.05):
    """Token ids whose experts are chosen by a clear margin in every layer."""
    r = reference(cfg, t)
    r.forward(np.arange(cfg["vocab"]))
    ids = np.flatnonzero(r.margin > (2 * margin if cfg["architecture"] == "Noresun" else margin))
    assert len(ids) >= 12, len(ids)
    return ids


def draw(cfg, t, n, seed):
    """n random tokens, every choice of an expert clear where they stand."""
    rng, ids, r = np.random.default_rng(seed), clear_tokens(cfg, t), reference(cfg, t)
    toks = rng.choice(ids, n)
    for _ in range(60):
        r.forward(toks)
        close = np.flatnonzero(r.margin < (0.08 if cfg["architecture"] == "Noresun" else 0.02))   # logits there, scores elsewhere
        if not len(close):
            return toks.tolist()
        toks[close] = rng.choice(ids, len(close))
    raise AssertionError(f"{len(close)} close calls are left")


def tensors(cfg, seed, rank=5):
    """Random tensors (f32 values on the bf16 grid), scaled so that every part of the model moves the logits."""
    if cfg["architecture"] == "Lilosun":
        return lilosun_tensors(cfg, seed)
    if cfg["architecture"] == "Rubuvik":
        return rubuvik_tensors(cfg, seed)
    if cfg["architecture"] == "Noresun":
        return noresun_tensors(cfg, seed)
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    t = {}

    def put(name, shape, std=None, mean=0.0):
        x = rng.standard_normal(shape) * (1.0 / np.sqrt(shape[-1]) if std is None else std) + mean
        t[name] = bf16_bits_to_f32(f32_to_bf16_bits(np.asarray(x, np.float32))).reshape(shape)

    def norm(name, alpha):
        put(name, (W,), 0.2, 1.0)
        put(name + ".b", (W,), 0.1)
        put(name + ".alpha", (), 0.0, alpha)

    put("embed", (V, W), 1.0)
    for i, e in enumerate(cfg["layers"]):
        m, l = e["mixer"], f"l{i}"
        H, D, E = m["heads"], m["dim"], m["vdim"]
        norm(l + ".norm1", 0.7)
        norm(l + ".norm1b", 0.9)
        p = l + ".mix."
        if e["type"] == "attention":
            put(p + "q", (H * 2 * D, W), 1.5 / np.sqrt(W))
            put(p + "k", (m["kv_heads"] * 2 * D, W), 1.5 / np.sqrt(W))
            put(p + "v", (m["kv_heads"] * E, W))
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + n, (D,), 0.2)
        else:
            put(p + "q", (H * D, W))
            put(p + "k", (H * D, W))
            put(p + "v", (H * E, W))
            put(p + "g", (H * E, W))
            if e["type"] == "gla":
                put(p + "a1", (rank, W))
                put(p + "a2", (H * D, rank), 1.0)
                put(p + "a2.b", (H * D,), 1.5, 1.0)
                put(p + "norm", (E,), 0.2, 1.0)
            else:
                put(p + "i", (H, W))
                put(p + "i.b", (H,), 1.0)
                put(p + "f", (H, W))
                put(p + "f.b", (H,), 1.0, 3.0)
                put(p + "norm", (H * E,), 0.2, 1.0)
        put(p + "o", (W, H * E))
        if e["mlp"]:
            F = e["mlp"]["ff"]
            norm(l + ".norm2", 0.8)
            norm(l + ".norm2b", 1.1)
            put(l + ".mlp.gate", (F, W))
            put(l + ".mlp.up", (F, W))
            put(l + ".mlp.down", (W, F))
    norm("final.norm", 0.6)
    return t


def bits(t):
    return {k: f32_to_bf16_bits(np.asarray(v, np.float32)).reshape(np.shape(v)) for k, v in t.items()}


def write_checkpoint(folder, cfg, t):
    """config.json and model.safetensors as a user has them."""
    (folder / "config.json").write_text(json.dumps(cfg))
    header, blob = {}, b""
    for name, a in bits(t).items():
        raw = np.ascontiguousarray(a, "<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(t[name])), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    h = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + blob)
    return str(folder)


def reference(cfg, t):
    """The plain reference over the values the checkpoint holds."""
    from oracle import layers
    return getattr(layers, cfg["architecture"])(cfg, {k: bf16_bits_to_f32(v).reshape(np.shape(v)) for k, v in bits(t).items()})


def device_model(ctx, cfg, t, compute, max_rows=1024):
    from paged_infer_b200 import api
    return api.LayeredModel(ctx, layered_config(cfg), bits(t), compute, max_rows)


def layered_config(cfg):
    return getattr(LayeredConfig, "from_" + cfg["architecture"].lower())(cfg)


def distance(got, want):
    """Root mean square of the difference over the spread of the reference, per row (a common shift taken off)."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()


LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}


class Session:
    """Sequences over one pool and state pool, with block tables and slots the test chooses (scattered on purpose)."""

    def __init__(self, model, blocks=256, block_size=16, slots=6, seed=0):
        self.m, self.bs = model, block_size
        self.kv = model.kv_pool(blocks, block_size)
        self.state = model.state_pool(slots) if model.state_bytes() else None
        self.free = list(np.random.default_rng(seed).permutation(blocks))
        self.slots = list(range(slots))[::-1]
        self.seq = {}

    def open(self, name):
        self.seq[name] = [0, [], self.slots.pop()]

    def close(self, name):
        _, table, slot = self.seq.pop(name)
        self.free = table[::-1] + self.free      # used again at once
        self.slots.append(slot)

    def run(self, portions, every_row=True):
        """portions: [(name, tokens)] -> list of logits arrays, one per portion (every row, or the last)."""
        starts, tables, slots = [], [], []
        for name, toks in portions:
            if name not in self.seq:
                self.open(name)
            s = self.seq[name]
            starts.append(s[0])
            s[0] += len(toks)
            while len(s[1]) * self.bs < s[0]:
                s[1].append(int(self.free.pop(0)))
            tables.append(list(s[1]))
            slots.append(s[2])
        counts = [len(t) for _, t in portions]
        ends = np.cumsum(counts)
        rows = np.arange(ends[-1]) if every_row else ends - 1
        out = self.m.step([t for _, t in portions], starts, tables, self.kv, self.state, slots if self.state else None, rows)
        return np.split(out, ends[:-1]) if every_row else list(out[:, None])
