"""Host-side checkpoint reading: the counterpart of ``ModelLoader`` and
``LlamaConfig::from_hf_config`` (reference ``src/model.rs:65-103``, ``:388-455``).

Pure host code (numpy only): it parses a safetensors file holding bf16 tensors
under HuggingFace Llama names and returns raw bf16 bit arrays.  Widening,
quantisation and upload happen in the CUDA library.
"""
from __future__ import annotations

import json
import struct
from dataclasses import dataclass, field

import numpy as np

ROPE_NEOX = 0
ROPE_INTERLEAVED = 1

QUANT_F32 = "f32"    # reference Quantization::F32 (bf16 checkpoint widened exactly)
QUANT_INT8 = "int8"  # reference Quantization::Int8


@dataclass
class LlamaConfig:
    """Field-for-field ``LlamaConfig`` (reference ``src/model.rs:14-53``)."""

    hidden_size: int = 2048
    num_hidden_layers: int = 22
    num_attention_heads: int = 32
    num_key_value_heads: int = 4
    intermediate_size: int = 5632
    vocab_size: int = 32000
    rms_norm_eps: float = 1e-5
    rope_theta: float = 10000.0
    attention_window: int | None = None
    rope_style: int = ROPE_NEOX
    quantization: str = QUANT_F32

    @property
    def head_dim(self) -> int:
        return self.hidden_size // self.num_attention_heads

    @property
    def kv_group(self) -> int:
        return self.num_attention_heads // self.num_key_value_heads

    @property
    def kv_dim(self) -> int:
        return self.num_key_value_heads * self.head_dim

    @classmethod
    def from_hf_config(cls, path: str) -> "LlamaConfig":
        """Read the architecture from a HuggingFace ``config.json``; absent
        fields keep their defaults and ``num_key_value_heads`` falls back to the
        query head count (reference ``src/model.rs:65-96``)."""
        with open(path) as f:
            j = json.load(f)
        d = cls()
        heads = int(j.get("num_attention_heads", d.num_attention_heads))
        return cls(
            hidden_size=int(j.get("hidden_size", d.hidden_size)),
            num_hidden_layers=int(j.get("num_hidden_layers", d.num_hidden_layers)),
            num_attention_heads=heads,
            num_key_value_heads=int(j.get("num_key_value_heads", heads)),
            intermediate_size=int(j.get("intermediate_size", d.intermediate_size)),
            vocab_size=int(j.get("vocab_size", d.vocab_size)),
            rms_norm_eps=float(j.get("rms_norm_eps", d.rms_norm_eps)),
            rope_theta=float(j.get("rope_theta", d.rope_theta)),
        )

    def as_dict(self) -> dict:
        return {k: getattr(self, k) for k in (
            "hidden_size", "num_hidden_layers", "num_attention_heads", "num_key_value_heads",
            "intermediate_size", "vocab_size", "rms_norm_eps", "rope_theta", "attention_window", "rope_style")}


MIXER_ATTENTION, MIXER_GLA, MIXER_MLSTM, MIXER_LATENT, MIXER_SSD, MIXER_LIGHTNING, MIXER_MINGRU = 0, 1, 2, 3, 4, 5, 6
FF_GELU, FF_SILU, FF_EXPERTS = 0, 1, 2
UNIT_CLAMPED, UNIT_SILU, UNIT_RELU2 = 0, 1, 2
SCORE_SIGMOID, SCORE_SOFTMAX, SCORE_CHOSEN = 0, 1, 2
NORM_DYT, NORM_LAYER, NORM_RMS, NORM_SUM = 0, 1, 2, 3


@dataclass
class LayerConfig:
    """One layer of a layered design: a token mixer with its own sizes and, if ``ff``, a gated feed-forward.

    ``window`` None: everything before.  ``maps`` 2: differential attention (``diff`` its constant).  ``tau`` belongs to the
    gated linear recurrence, ``gate_cap`` to the matrix memory.  Latent attention: ``rank`` latent channels, ``dim`` unrotated and
    ``rot_dims`` rotated channels per head, rotation stretched by ``rot_factor`` and the three constants behind it.  State-space
    recurrence: ``dim`` state channels, heads in ``groups``, ``conv`` taps, ``norm_groups`` parts.  Routed experts: ``ff`` is one
    expert's size, ``shared_ff`` that of the expert every token meets (``shared_gate``: with a gate per token), ``unit`` their
    activation, ``score`` what the router makes of its logits; a group of experts is as good as its ``group_best`` best scores
    together; the chosen weights are brought to sum 1 if ``renorm`` and multiplied by ``route_scale``.  Attention with one map may
    have ``biases``, q and k of unit root mean square (``unit_qk``), a ``distance_bias``, a ``sink`` and a gate per head, queries
    that grow with the position (``q_temp_coef``, ``q_temp_every``; 0: not) and values mixed with those of the first layer that has
    ``v_mix``; or q and k normalised over the whole projection (``norm_qk``), ``sigmoid_weights`` that are not normalised over the
    keys, and the keys and values of the layer ``kv_from`` in place of its own.  ``rot_banded``: the rotation is stretched by
    wavelength.  ``decay``: the constant decay of every head of lightning attention.  The element-wise recurrence (minGRU) has one head
    of ``vdim`` channels.  ``router_bias``: of the router's logits, in place of a correction of the choice."""

    mixer: int
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0
    maps: int = 1
    window: int | None = None
    rot_dims: int = 0
    rot_base: float = 10000.0
    scale: float = 1.0
    diff: float = 0.0
    tau: float = 1.0
    gate_cap: float = 1.0
    ff: int = 0
    ff_kind: int = FF_GELU
    rank: int = 0
    rot_factor: float = 1.0
    rot_original: float = 1.0
    rot_fast: float = 32.0
    rot_slow: float = 1.0
    groups: int = 1
    norm_groups: int = 1
    conv: int = 1
    experts: int = 0
    top: int = 0
    expert_groups: int = 1
    keep_groups: int = 1
    shared_ff: int = 0
    limit: float = 0.0
    shared_limit: float = 0.0
    biases: bool = False
    unit_qk: bool = False
    distance_bias: bool = False
    sink: bool = False
    head_gate: bool = False
    v_mix: bool = False
    q_temp_coef: float = 0.0
    q_temp_every: float = 0.0
    decay: tuple | None = None
    unit: int = UNIT_CLAMPED
    score: int = SCORE_SIGMOID
    group_best: int = 2
    renorm: bool = True
    shared_gate: bool = True
    route_scale: float = 1.0
    router_bias: bool = False
    rot_banded: bool = False
    norm_qk: bool = False
    sigmoid_weights: bool = False
    kv_from: int | None = None


@dataclass
class LayeredConfig:
    """A design whose layers each name a mixer (``pi_layered_config``)."""

    width: int
    vocab_size: int
    norm_eps: float
    layers: list
    norm: int = NORM_DYT
    tied: bool = True
    logit_scale: float = 1.0
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    side_dim: int = 0
    residual_keep: float = 1.0
    sublayer_gate: bool = False
    pair_buckets: int = 0        # rows of the table of token pairs, but for the one of first tokens
    pair_prev: int = 0
    pair_cur: int = 0

    @property
    def has_state(self) -> bool:
        """Whether a sequence carries more than its cache: a recurrence, or the previous token."""
        return self.pair_buckets > 0 or any(l.mixer not in (MIXER_ATTENTION, MIXER_LATENT) for l in self.layers)

    @classmethod
    def from_sumosun(cls, j: dict) -> "LayeredConfig":
        """The Sumosun design's ``config.json``: differential attention, GLA and mLSTM layers in any order."""
        layers = []
        for i, e in enumerate(j["layers"]):
            m, mlp = e["mixer"], e.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            ff = int(mlp["ff"]) if mlp is not None else 0
            common = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), ff=ff)
            if e["type"] == "attention":
                mask, rot = m.get("mask"), m.get("rot")
                layers.append(LayerConfig(MIXER_ATTENTION, kv_heads=int(m["kv_heads"]), maps=2, window=int(mask["size"]) if mask else None,
                                          rot_dims=int(rot["dims"]) if rot else 0, rot_base=float(rot["base"]) if rot else 1.0,
                                          scale=float(m["scale"]), diff=float(m["diff"]), **common))
            elif e["type"] == "gla":
                layers.append(LayerConfig(MIXER_GLA, tau=float(m["tau"]), **common))
            elif e["type"] == "mlstm":
                layers.append(LayerConfig(MIXER_MLSTM, gate_cap=float(m["gate_cap"]), **common))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        return cls(width=int(j["width"]), vocab_size=int(j["vocab"]), norm_eps=float(j["norm"]["eps"]), layers=layers)

    @classmethod
    def from_lilosun(cls, j: dict) -> "LayeredConfig":
        """The Lilosun design's ``config.json``: latent attention and Mamba-2 layers in any order, each with a dense or a routed
        feed-forward or none."""
        layers = []
        for i, e in enumerate(j["layers"]):
            m = e["mixer"]
            kw = dict(heads=int(m["heads"]), vdim=int(m["vdim"]), **cls._lilosun_feed_forward(i, e.get("mlp")))
            if e["type"] == "latent_attention":
                mask, rot = m.get("mask"), m["rot"]
                if int(rot["dims"]) != int(m["rot_dim"]):
                    raise ValueError(f"layer {i}: {rot['dims']} rotated channels, the rotated part has {m['rot_dim']}")
                scaling = rot.get("scaling")
                if scaling:
                    kw.update(rot_factor=float(scaling["factor"]), rot_original=float(scaling["original"]), rot_fast=float(scaling["fast"]),
                              rot_slow=float(scaling["slow"]))
                layers.append(LayerConfig(MIXER_LATENT, dim=int(m["dim"]), rank=int(m["kv_rank"]), window=int(mask["size"]) if mask else None,
                                          rot_dims=int(m["rot_dim"]), rot_base=float(rot["base"]), scale=float(m["scale"]), **kw))
            elif e["type"] == "mamba2":
                layers.append(LayerConfig(MIXER_SSD, dim=int(m["state"]), groups=int(m["groups"]), norm_groups=int(m["norm_groups"]), conv=int(m["conv"]), **kw))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        return cls(width=int(j["width"]), vocab_size=int(j["vocab"]), norm_eps=float(j["norm"]["eps"]), layers=layers, norm=NORM_LAYER, tied=False,
                   logit_scale=float(j["logit_scale"]))

    @classmethod
    def _lilosun_feed_forward(cls, i: int, mlp: dict | None) -> dict:
        if mlp is None:
            return {}
        if mlp["kind"] == "dense":
            return dict(ff=int(mlp["ff"]), ff_kind=FF_SILU)
        if mlp["kind"] != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        kw = dict(limit=float(mlp["expert"]["limit"]), **cls._experts(mlp))
        if mlp.get("shared"):
            kw.update(shared_limit=float(mlp["shared"]["limit"]))
        return kw

    @staticmethod
    def _experts(mlp: dict) -> dict:
        r, groups, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
        kw = dict(ff=int(mlp["expert"]["ff"]), ff_kind=FF_EXPERTS, experts=int(r["experts"]), top=int(r["top"]))
        if groups:
            kw.update(expert_groups=int(groups["count"]), keep_groups=int(groups["keep"]))
        if shared:
            kw.update(shared_ff=int(shared["ff"]))
        return kw

    @classmethod
    def from_rubuvik(cls, j: dict) -> "LayeredConfig":
        """The Rubuvik design's ``config.json``: two kinds of attention with a distance bias and lightning attention in any order, each
        with a dense or a routed feed-forward or none, and a table of tokens beside the layers."""
        layers = []
        for i, e in enumerate(j["layers"]):
            m = e["mixer"]
            kw = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), **cls._rubuvik_feed_forward(i, e.get("mlp")))
            if e["type"] in ("attention", "attention_2"):
                mask, temp = m.get("mask"), m.get("q_temp")
                if e["type"] == "attention_2":
                    kw.update(biases=True, unit_qk=True, sink=True, head_gate=True)
                if temp:
                    kw.update(q_temp_coef=float(temp["coef"]), q_temp_every=float(temp["every"]))
                layers.append(LayerConfig(MIXER_ATTENTION, kv_heads=int(m["kv_heads"]), window=int(mask["size"]) if mask else None, scale=float(m["scale"]),
                                          distance_bias=True, v_mix=bool(m.get("v_mix", False)), **kw))
            elif e["type"] == "lightning":
                layers.append(LayerConfig(MIXER_LIGHTNING, decay=tuple(float(d) for d in m["decay"]), **kw))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        side = j.get("token_side")
        return cls(width=int(j["width"]), vocab_size=int(j["vocab"]), norm_eps=float(j["norm"]["eps"]), layers=layers, norm=NORM_RMS,
                   embed_scale=float(j["embedding"]["scale"]), residual_mult=float(j["residual_mult"]), side_dim=int(side["dim"]) if side else 0)

    @classmethod
    def _rubuvik_feed_forward(cls, i: int, mlp: dict | None) -> dict:
        if mlp is None:
            return {}
        if mlp["kind"] == "dense":
            return dict(ff=int(mlp["ff"]), ff_kind=FF_SILU)
        if mlp["kind"] != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        return dict(unit=UNIT_SILU, score=SCORE_SOFTMAX, group_best=1, renorm=False, shared_gate=False, route_scale=float(mlp["router"]["scale"]),
                    **cls._experts(mlp))

    @classmethod
    def from_noresun(cls, j: dict) -> "LayeredConfig":
        """The Noresun design's ``config.json``: attention with sigmoid weights, which may share the keys and values of an earlier layer,
        and minGRU layers in any order, each with routed experts or no feed-forward; gated sublayers, norms of the sum; a table of token
        pairs beside the embedding."""
        layers = []
        for i, e in enumerate(j["layers"]):
            m, mlp = e["mixer"], e.get("mlp")
            kw = {}
            if mlp is not None:
                if mlp["kind"] != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
                kw = dict(unit=UNIT_RELU2, score=SCORE_CHOSEN, shared_gate=False, router_bias=True, **cls._experts(mlp))
            if e["type"] == "attention":
                mask, rot, kv_from = m.get("mask"), m.get("rot"), m.get("kv_from")
                if rot:
                    kw.update(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]))
                    if rot.get("scaling"):
                        s = rot["scaling"]
                        kw.update(rot_banded=True, rot_factor=float(s["factor"]), rot_original=float(s["original"]), rot_fast=float(s["high"]),
                                  rot_slow=float(s["low"]))
                layers.append(LayerConfig(MIXER_ATTENTION, heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                          window=int(mask["size"]) if mask else None, scale=float(m["scale"]), norm_qk=True, sigmoid_weights=True,
                                          kv_from=None if kv_from is None else int(kv_from), **kw))
            elif e["type"] == "mingru":
                layers.append(LayerConfig(MIXER_MINGRU, heads=1, dim=1, vdim=int(m["width"]), **kw))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        pairs, kw = j["embedding"].get("bigram"), {}
        if pairs:
            n = int(pairs["buckets"])
            kw = dict(pair_buckets=n, pair_prev=int(pairs["mul_prev"]) % n, pair_cur=int(pairs["mul_cur"]) % n)
        return cls(width=int(j["width"]), vocab_size=int(j["vocab"]), norm_eps=float(j["norm"]["eps"]), layers=layers, norm=NORM_SUM,
                   embed_scale=float(j["embedding"]["scale"]), residual_keep=float(j["postln_alpha"]), sublayer_gate=True, **kw)


def read_safetensors(path: str) -> dict:
    """name -> array with the stored shape: bf16 tensors as uint16 bits, f32 and integer tables as they are."""
    dtypes = {"BF16": "<u2", "F32": "<f4", "I32": "<i4"}
    with open(path, "rb") as f:
        raw = f.read()
    (hlen,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + hlen])
    base = 8 + hlen
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in dtypes:
            raise ValueError(f"{name}: only BF16 checkpoints are supported, got {info['dtype']}")
        dt = np.dtype(dtypes[info["dtype"]])
        a, b = info["data_offsets"]
        if (base + a) % dt.itemsize:
            out[name] = np.frombuffer(raw[base + a:base + b], dtype=dt).reshape(info["shape"])
        else:
            out[name] = np.frombuffer(raw, dtype=dt, count=(b - a) // dt.itemsize, offset=base + a).reshape(info["shape"])
    return out


def bf16_bits_to_f32(bits: np.ndarray) -> np.ndarray:
    """Exact widening (reference ``pack_bf16_to_f32``, ``src/math.rs:66-71``)."""
    return (bits.astype(np.uint32) << np.uint32(16)).view(np.float32)


def f32_to_bf16_bits(x: np.ndarray) -> np.ndarray:
    """Round-to-nearest-even f32 -> bf16 bits."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    bias = np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))
    return ((u + bias) >> np.uint32(16)).astype(np.uint16)


@dataclass
class HostWeights:
    """What ``ModelLoader::load_weights`` collects (reference
    ``src/model.rs:398-446``), still as bf16 bits: the CUDA library decides the
    device representation per ``quantization``."""

    token_embeddings: np.ndarray            # [vocab, hidden] bf16 bits
    final_norm: np.ndarray                  # [hidden] f32
    attention_norm: list = field(default_factory=list)   # per layer [hidden] f32
    ffn_norm: list = field(default_factory=list)
    projections: list = field(default_factory=list)      # per layer dict wq..w3 -> bf16 bits [rows, cols]
    lm_head: np.ndarray | None = None       # bf16 bits [vocab, hidden]


def load_weights(path: str, cfg: LlamaConfig) -> HostWeights:
    t = read_safetensors(path)

    def need(name):
        if name not in t:
            raise KeyError(f"missing tensor: {name}")
        return t[name]

    embed = need("model.embed_tokens.weight")
    # Tied embeddings: fall back to the embedding matrix (reference :401-403).
    lm_head = t.get("lm_head.weight", embed)
    hw = HostWeights(token_embeddings=embed, final_norm=bf16_bits_to_f32(need("model.norm.weight")), lm_head=lm_head)
    for i in range(cfg.num_hidden_layers):
        p = f"model.layers.{i}"
        hw.attention_norm.append(bf16_bits_to_f32(need(f"{p}.input_layernorm.weight")))
        hw.ffn_norm.append(bf16_bits_to_f32(need(f"{p}.post_attention_layernorm.weight")))
        hw.projections.append({
            "wq": need(f"{p}.self_attn.q_proj.weight"),
            "wk": need(f"{p}.self_attn.k_proj.weight"),
            "wv": need(f"{p}.self_attn.v_proj.weight"),
            "wo": need(f"{p}.self_attn.o_proj.weight"),
            "w1": need(f"{p}.mlp.gate_proj.weight"),
            "w2": need(f"{p}.mlp.down_proj.weight"),
            "w3": need(f"{p}.mlp.up_proj.weight"),
        })
    return hw
