"""Noresun on the device against the plain reference: every mechanism alone, prefill against decoding, portions, mixed batches,
blocks and slots used again, window edges, shared keys, token pairs, long memories, routing, and generation through the engine.
Both number formats."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from layered_helpers import (BANDS, LIMIT, Session, device_model, distance, draw, mingru, noresun, reference, relu2_moe, sigmoid_attention, tensors,
                             write_checkpoint)
from test_gpu_layered import reference_greedy

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("compute", ["float32", "bfloat16"])


@pytest.fixture(scope="module")
def ctx():
    from paged_infer_b200 import api
    return api.Context(0)


# what one layer (or one and another that reads its keys) can be, in sizes that hit the kernels' special cases
ALONE = {
    "attention": [sigmoid_attention()],
    "attention_everything": [sigmoid_attention(window=None, heads=5, kv_heads=5)],
    "attention_window1": [sigmoid_attention(window=1, heads=2, kv_heads=1)],
    "attention_wide_window": [sigmoid_attention(window=1000, scale=0.05, base=300.0)],
    "attention_no_rotation": [sigmoid_attention(rot=0)],
    "attention_all_rotated": [sigmoid_attention(dim=24, rot=24, scaling=None)],
    "attention_odd": [sigmoid_attention(heads=3, kv_heads=3, dim=11, vdim=9, window=19, rot=6)],
    "attention_one_pair": [sigmoid_attention(heads=4, kv_heads=1, dim=14, vdim=18, rot=2)],
    "attention_17_per_group": [sigmoid_attention(heads=34, kv_heads=2, dim=16, vdim=16, window=90, rot=16)],
    "attention_one_head": [sigmoid_attention(heads=1, kv_heads=1, dim=80, vdim=32, window=65)],
    "attention_big_heads": [sigmoid_attention(heads=2, kv_heads=1, dim=200, vdim=150, window=50, rot=64)],
    "attention_wide_values": [sigmoid_attention(heads=4, kv_heads=2, dim=128, vdim=256, window=77, rot=128)],
    "attention_narrow_values": [sigmoid_attention(heads=4, kv_heads=2, dim=64, vdim=4, window=77)],
    "attention_huge_keys": [sigmoid_attention(heads=2, kv_heads=2, dim=300, vdim=20, window=40, scale=0.03)],
    "attention_many_heads": [sigmoid_attention(heads=48, kv_heads=6, dim=128, vdim=16, window=40)],          # norms over 6144 and 768 channels
    "attention_many_odd_heads": [sigmoid_attention(heads=36, kv_heads=12, dim=90, vdim=10, window=40, rot=30)],
    "shared": [sigmoid_attention(), sigmoid_attention(window=50, kv_from=0)],
    "shared_everything": [sigmoid_attention(window=9), sigmoid_attention(window=None, kv_from=0)],
    "shared_odd": [sigmoid_attention(heads=3, kv_heads=3, dim=11, vdim=9, rot=6), sigmoid_attention(heads=3, kv_heads=3, dim=11, vdim=9, rot=6, kv_from=0)],
    "shared_many_heads": [sigmoid_attention(heads=48, kv_heads=6, dim=128, vdim=16), sigmoid_attention(heads=48, kv_heads=6, dim=128, vdim=16, kv_from=0)],
    "shared_twice_and_apart": [sigmoid_attention(), mingru(), sigmoid_attention(heads=4, kv_heads=4, dim=16, rot=4), sigmoid_attention(window=7, kv_from=0),
                               sigmoid_attention(heads=4, kv_heads=4, dim=16, rot=4, kv_from=2), sigmoid_attention(kv_from=0, scale=0.4)],
    "mingru": [mingru()],
    "mingru_one": [mingru(1)],
    "mingru_odd": [mingru(37)],
    "mingru_large": [mingru(1030)],
    "moe": [mingru(mlp=relu2_moe())],
    "moe_top1": [sigmoid_attention(mlp=relu2_moe(experts=7, top=1, ff=24))],
    "moe_all": [mingru(mlp=relu2_moe(experts=4, top=4, ff=33))],
    "moe_one": [mingru(mlp=relu2_moe(experts=1, top=1, ff=50))],
    "moe_many": [sigmoid_attention(mlp=relu2_moe(experts=70, top=6, ff=17))],
    "moe_many_chosen": [mingru(mlp=relu2_moe(experts=50, top=41, ff=8))],
}
MIXED = noresun([sigmoid_attention(vdim=12), mingru(mlp=relu2_moe()), sigmoid_attention(vdim=12, window=44, kv_from=0, mlp=relu2_moe(experts=10, top=2)),
                 mingru(70, mlp=relu2_moe(experts=5, top=4, ff=30)), sigmoid_attention(window=None, heads=2, kv_heads=1, dim=32, rot=20, mlp=relu2_moe()),
                 sigmoid_attention(window=17, heads=6, vdim=12, kv_from=0), mingru()], vocab=500)


@pytest.fixture(scope="module")
def mixed():
    t = tensors(MIXED, 3)
    return t, reference(MIXED, t)


def check_alone(ctx, cfg, t, toks, compute):
    """Residual stream and logits of a model: a prompt in one step, then token by token."""
    layer = []
    want = reference(cfg, t).forward(toks, layer)
    n = len(toks) - 9
    m = device_model(ctx, cfg, t, compute)
    s = Session(m)
    m.trace_layers(True)
    got = s.run([("a", toks[:n])])[0]
    xs = [m.read_layer(i, n) for i in range(len(layer))]
    m.trace_layers(False)
    lim = LIMIT[compute]
    for x, l in zip(xs, layer):
        assert distance(x, l[:n]).max() < lim
    assert distance(got, want[:n]).max() < lim
    for i in range(n, len(toks)):
        assert distance(s.run([("a", [toks[i]])])[0], want[i:i + 1]).max() < 1.5 * lim


@BOTH
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(ctx, name, compute):
    cfg = noresun(ALONE[name], width=72, vocab=240)
    t = tensors(cfg, 11)
    check_alone(ctx, cfg, t, draw(cfg, t, 150, 5), compute)


@BOTH
@pytest.mark.parametrize("change", [dict(bigram=None), dict(bigram=(1, 1, 1)), dict(bigram=(997, 2000003, 31337), alpha=1.0), dict(embed_scale=1.0, alpha=5.0),
                                    dict(width=75), dict(width=1028), dict(width=2052), dict(width=4100), dict(eps=0.3), dict(alpha=0.25)], ids=str)
def test_sizes_and_constants_around_the_layers(ctx, change, compute):
    """Widths that leave the row kernel's registers, rows of odd length, no table of pairs, constants that are 1."""
    cfg = noresun([mingru(mlp=relu2_moe(experts=3, top=2, ff=40)), sigmoid_attention(), sigmoid_attention(kv_from=1, mlp=relu2_moe(experts=4, top=2, ff=24)), mingru(21)],
                  **{"vocab": 240, **change})
    t = tensors(cfg, 12)
    check_alone(ctx, cfg, t, draw(cfg, t, 80, 6), compute)


@BOTH
def test_decoding_equals_prefill(ctx, mixed, compute):
    t, ref = mixed
    toks = draw(MIXED, t, 100, 8)
    want = ref.forward(toks)
    s = Session(device_model(ctx, MIXED, t, compute), block_size=16)
    whole = s.run([("whole", toks)])[0]
    one = np.concatenate([s.run([("one", [x])])[0] for x in toks])
    assert distance(whole, want).max() < LIMIT[compute]
    assert distance(one, want).max() < LIMIT[compute]


@BOTH
@pytest.mark.parametrize("size", [2, 3, 7, 16, 63, 64, 65, 128, 129])
def test_portions(ctx, mixed, size, compute):
    t, ref = mixed
    toks = draw(MIXED, t, 200 if size > 7 else 70, 9)
    want = ref.forward(toks)
    s = Session(device_model(ctx, MIXED, t, compute), block_size=8)
    got = np.concatenate([s.run([("p", toks[i:i + size])])[0] for i in range(0, len(toks), size)])
    assert distance(got, want).max() < LIMIT[compute]


@BOTH
def test_uneven_batches_and_reuse(ctx, mixed, compute):
    """Portions beside single tokens, requests that pause, end and make room; freed blocks and slots are used at once."""
    t, ref = mixed
    s = Session(device_model(ctx, MIXED, t, compute), blocks=40, slots=3)
    rng = np.random.default_rng(1)
    live, got, done = {}, {}, 0
    for i in range(60):
        while len(live) < 3 and done + len(live) < 9:
            name = f"r{done + len(live)}.{i}"
            live[name] = draw(MIXED, t, int(rng.choice([1, 2, 19, 64, 150])), 100 + i + len(live))
            got[name] = []
        batch = []
        for name in list(live):
            if rng.random() < 0.2:
                continue    # pauses
            n = int(rng.choice([1, 1, 2, 5, 70, 90]))
            at = sum(len(x) for x in got[name])
            if live[name][at:at + n]:
                batch.append((name, live[name][at:at + n]))
        if not batch:
            continue
        for (name, _), out in zip(batch, s.run(batch)):
            got[name].append(out)
        for name in list(live):
            if sum(len(x) for x in got[name]) == len(live[name]):
                assert distance(np.concatenate(got[name]), ref.forward(live[name])).max() < LIMIT[compute], name
                s.close(name)
                del live[name]
                done += 1
    assert done == 9


@BOTH
def test_batch_does_not_change_a_row(ctx, mixed, compute):
    t, _ = mixed
    m = device_model(ctx, MIXED, t, compute)
    toks = {n: draw(MIXED, t, k, 40 + k) for n, k in (("a", 33), ("b", 70), ("c", 5), ("d", 101))}
    alone = {}
    for n in toks:
        s = Session(m, seed=1)
        alone[n] = [s.run([(n, toks[n][:-1])])[0], s.run([(n, toks[n][-1:])])[0]]
    s = Session(m, seed=2)
    first = s.run([(n, toks[n][:-1]) for n in toks])
    last = s.run([(n, toks[n][-1:]) for n in reversed(toks)])
    for i, n in enumerate(toks):
        assert distance(first[i], alone[n][0]).max() < LIMIT[compute] / 2
        assert distance(last[len(toks) - 1 - i], alone[n][1]).max() < LIMIT[compute] / 2


NEEDLE, SEEKER = 1, 2


def needle_model(window, shared, bias=-7.0):
    """An attention layer in which token SEEKER looks for token NEEDLE through one unrotated channel of every head, so that its weight is
    nearly 1 and every other key's is small.  ``shared``: the layer is the second one and reads the keys of the first, whose own
    window is one token wide."""
    heads, dim, rot = 4, 12, 6
    layer = sigmoid_attention(heads, 2, dim, 20, window, rot, scale=1.0, kv_from=0 if shared else None)
    layers = [sigmoid_attention(heads, 2, dim, 20, 1, rot, scale=1.0), layer] if shared else [layer]
    cfg = noresun(layers, width=64, vocab=96, embed_scale=1.0, alpha=2.0, bigram=None)
    t = tensors(cfg, 21)
    e = t["embed"]
    e[:, 40:42] = 0
    e[NEEDLE, 40] = e[SEEKER, 41] = 8.0
    for n in list(t):
        if n.endswith((".norm1", ".q.norm", ".k.norm")):
            t[n][:] = 1.0
        if n.endswith(".mix.o"):
            t[n][40:42] = 0                                              # the marks pass through a layer as they are
        if n.endswith(".pb"):
            t[n][:] = bias
        if n.endswith((".mix.q", ".mix.k")):
            t[n][:, 40:42] = 0
            t[n][dim - 1::dim] = 0
            t[n][dim - 1::dim, 41 if n.endswith("q") else 40] = 40.0     # behind the norm this channel is nearly all of q and k
        if n.endswith(".mix.v"):
            t[n][:, 40] *= 20                                            # and what is found there is large
    return cfg, t


@BOTH
@pytest.mark.parametrize("shared", [False, True], ids=["own_keys", "shared_keys"])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 47, 64, 65, 130])
def test_window_edge(ctx, window, shared, compute):
    """NEEDLE just inside and just outside the window of SEEKER, at block and tile borders, read in a prompt, in a portion of
    two and when decoded."""
    cfg, t = needle_model(window, shared)
    ref = reference(cfg, t)
    m = device_model(ctx, cfg, t, compute)
    fill = np.random.default_rng(3).integers(3, 96, 400).tolist()
    power = []
    for back in sorted({window - 1, window, window + 1} - {0}):
        for at in (back, back + 15, back + 16, back + 33, back + 63, back + 64):      # NEEDLE at at - back
            toks = fill[:at + 1]
            toks[at - back] = NEEDLE
            toks[at] = SEEKER
            want = ref.forward(toks)[-1:]
            other = list(toks)
            other[at - back] = 50
            power.append((back < window, distance(ref.forward(other)[-1:], want).max()))
            s = Session(m, block_size=16)
            assert distance(s.run([("whole", toks)], False)[0], want).max() < 2 * LIMIT[compute]
            s.run([("decode", toks[:-1])], False)
            assert distance(s.run([("decode", toks[-1:])], False)[0], want).max() < 2 * LIMIT[compute]
            if at > 2:
                s.run([("two", toks[:-2])], False)
                assert distance(s.run([("two", toks[-2:])], False)[0], want).max() < 2 * LIMIT[compute]
    # the test has teeth: inside, the needle matters a lot; outside, not at all
    assert all(p > 0.2 for inside, p in power if inside) and all(p < 1e-9 for inside, p in power if not inside)


@BOTH
@pytest.mark.parametrize("shared", [False, True], ids=["own_keys", "shared_keys"])
def test_far_key_without_a_window(ctx, shared, compute):
    """The first token among hundreds of keys, in a prompt, in portions and decoded far along (keys cut over a cluster)."""
    cfg, t = needle_model(None, shared, bias=-9.0)
    ref = reference(cfg, t)
    m = device_model(ctx, cfg, t, compute)
    toks = [NEEDLE] + np.random.default_rng(4).integers(3, 96, 700).tolist()
    for i in (1, 63, 64, 300, 517, 690, 699, 700):
        toks[i] = SEEKER
    want = ref.forward(toks)
    assert distance(ref.forward([50] + toks[1:])[-1:], want[-1:]).max() > 0.2
    for bs in (16, 12, 64):
        s = Session(m, block_size=bs)
        got = [s.run([("a", toks[:600])])[0], s.run([("a", toks[600:690])])[0]] + [s.run([("a", [x])])[0] for x in toks[690:]]
        assert distance(np.concatenate(got), want).max() < 2 * LIMIT[compute]


@BOTH
@pytest.mark.parametrize("bias", [-200.0, -6.0, 0.0, 90.0])
def test_weights_of_every_size(ctx, bias, compute):
    """Biases that shut every key out, and biases that let every key in with all its weight: hundreds of values added up."""
    cfg = noresun([sigmoid_attention(window=300, heads=6)], vocab=96)
    t = tensors(cfg, 22)
    t["l0.mix.pb"][:] = bias + np.arange(6)
    ref = reference(cfg, t)
    toks = np.random.default_rng(5).integers(0, 96, 400).tolist()
    want = ref.forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:380])])[0], s.run([("a", toks[380:383])])[0]] + [s.run([("a", [x])])[0] for x in toks[383:]]
    assert np.isfinite(np.concatenate(got)).all()
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_rotation_bands(ctx, compute):
    """Scores that hang on the rotation, at positions where the bands' frequencies have parted."""
    layer = lambda scaling: noresun([sigmoid_attention(heads=2, kv_heads=1, dim=16, rot=16, window=None, scale=0.8, base=200.0, scaling=scaling)], vocab=96)
    cfg = layer(BANDS)
    t = tensors(cfg, 23)
    toks = np.random.default_rng(6).integers(0, 96, 260).tolist()
    want = reference(cfg, t).forward(toks)
    for other in (None, dict(BANDS, low=1.6), dict(BANDS, high=4.8), dict(BANDS, factor=6.5), dict(BANDS, original=170)):
        assert distance(reference(layer(other), t).forward(toks), want).max() > 20 * LIMIT["float32"]
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:250])])[0]] + [s.run([("a", [x])])[0] for x in toks[250:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
@pytest.mark.parametrize("bigram", [(211, 5, 3), (65521, 65000, 64999), (1009, 2 ** 31 - 1, 2 ** 40 + 7)], ids=str)
def test_token_pairs_over_every_cut(ctx, bigram, compute):
    """The previous token across steps of all sizes, of several sequences at once and in slots used again; products beyond 32 bits."""
    cfg = noresun([mingru(24)], width=40, vocab=50000, bigram=bigram)
    t = tensors(cfg, 24)
    t["embed"][:, :16] *= 0.125                                      # the pair is most of what a token is
    t["bigram"] *= 4
    ref = reference(cfg, t)
    rng = np.random.default_rng(8)
    s = Session(device_model(ctx, cfg, t, compute, max_rows=128), slots=2)
    for _ in range(3):
        toks = {n: rng.integers(40000, 50000, 40).tolist() for n in "ab"}
        want = {n: ref.forward(v) for n, v in toks.items()}
        swapped = toks["a"][:]
        swapped[4] = 3
        assert distance(ref.forward(swapped)[5:6], want["a"][5:6]).max() > 0.05      # another token before it
        at, got = dict.fromkeys(toks, 0), {n: [] for n in toks}
        for sizes in ({"a": 1}, {"b": 2}, {"a": 1, "b": 1}, {"a": 3}, {"b": 5, "a": 2}, {"a": 1, "b": 1}, {"a": 30}, {"b": 30}, {"b": 1, "a": 1}, {"a": 1}):
            for (n, k), out in zip(sizes.items(), s.run([(n, toks[n][at[n]:at[n] + k]) for n, k in sizes.items()])):
                got[n].append(out)
                at[n] += k
        assert at == {"a": 40, "b": 40}
        for n in toks:
            assert distance(np.concatenate(got[n]), want[n]).max() < LIMIT[compute]
            s.close(n)


@BOTH
def test_first_token_is_remembered(ctx, compute):
    """Gates that are nearly shut: the first token still moves the logits a thousand tokens on, through portions and decoding."""
    cfg = noresun([mingru(40)], vocab=96, bigram=None)
    t = tensors(cfg, 31)
    t["l0.mix.z"] *= np.float32(0.05)
    t["l0.mix.z.b"][:] = np.linspace(-9, -6, 40)
    t["l0.mix.x"] *= np.float32(0.2)
    for n in ("z", "x"):                                             # what only token 7 has opens the gate and is large
        t[f"l0.mix.{n}"][:, 50] = 3.0
    t["embed"][:, 50] = 0
    t["embed"][7, 50] = 4.0
    toks = [7] + np.random.default_rng(5).integers(8, 96, 1199).tolist()
    ref = reference(cfg, t)
    want = ref.forward(toks)
    assert distance(ref.forward([8] + toks[1:])[-1:], want[-1:]).max() > 0.1
    s = Session(device_model(ctx, cfg, t, compute, max_rows=1200))
    got = [s.run([("a", toks[:1100])])[0], s.run([("a", toks[1100:1180])])[0]] + [s.run([("a", [x])])[0] for x in toks[1180:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_gates_and_candidates_of_every_size(ctx, compute):
    """Gates wide open and shut, candidates far below and far above zero, and exactly at it."""
    cfg = noresun([mingru(48)], vocab=96)
    t = tensors(cfg, 32)
    t["l0.mix.z.b"][:] = np.tile([-120.0, -25.0, -4.0, 0.0, 25.0, 120.0], 8)
    t["l0.mix.x.b"][:] = np.repeat([-120.0, -20.0, -1.0, 0.0, 0.0, 1.0, 20.0, 120.0], 6)
    t["l0.mix.x"][18:24] = 0                                         # u is exactly 0
    t["l0.mix.o"][CODE_END:, 36:] *= 0.05
    toks = np.random.default_rng(6).integers(0, 96, 150).tolist()
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:70])])[0], s.run([("a", toks[70:140])])[0]] + [s.run([("a", [x])])[0] for x in toks[140:]]
    assert np.isfinite(np.concatenate(got)).all()
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


CODE_END = 16


@pytest.mark.parametrize("width", [7, 40, 130, 520])
def test_chunks_equal_token_by_token(ctx, width):
    """The cluster kernel against the scan on the same projections (both in the bf16 mode), around every length at which it cuts
    time differently: far tighter than bf16 itself."""
    cfg = noresun([mingru(width)], width=48, vocab=96)
    t = tensors(cfg, 41)
    t["l0.mix.z.b"] -= np.float32(2.0)
    m = device_model(ctx, cfg, t, "bfloat16", max_rows=2200)
    toks = np.random.default_rng(42).integers(0, 96, 2200).tolist()
    s = Session(m)
    scan = np.concatenate([s.run([("a", toks[i:i + 63])])[0] for i in range(0, len(toks), 63)])
    for sizes in ((2200,), (64, 65, 127, 128, 129, 1023), (1024, 1025), (700, 5, 1, 1300)):
        s, at = Session(m), 0
        for n in sizes:
            out = s.run([("a", toks[at:at + n])])[0]
            assert np.isfinite(out).all() and distance(out, scan[at:at + n]).max() < 6e-3
            at += n
    assert distance(scan[:300], reference(cfg, t).forward(toks[:300])).max() < LIMIT["bfloat16"]


@BOTH
def test_long_decoding(ctx, mixed, compute):
    t, ref = mixed
    m = device_model(ctx, MIXED, t, compute)
    a, b = draw(MIXED, t, 300, 13), draw(MIXED, t, 300, 14)
    s = Session(m)
    got = [s.run([("a", [x]), ("b", [y])]) for x, y in zip(a, b)]
    for i, toks in enumerate((a, b)):
        assert distance(np.concatenate([g[i] for g in got]), ref.forward(toks)).max() < LIMIT[compute]


def test_wide_model_many_rows(ctx):
    """Sizes that fill the tensor-core tiles, up to several hundred rows; expert tiles of every height."""
    attn = dict(heads=8, kv_heads=2, dim=64, vdim=96, rot=32)
    cfg = noresun([sigmoid_attention(window=100, mlp=relu2_moe(experts=16, top=2, ff=136), **attn), mingru(600, mlp=relu2_moe(experts=5, top=3, ff=300)),
                   sigmoid_attention(window=200, kv_from=0, mlp=relu2_moe(experts=40, top=5, ff=64), **attn)], width=520, vocab=1000)
    t = tensors(cfg, 14)
    toks = draw(cfg, t, 600, 15)
    want = reference(cfg, t).forward(toks)
    m = device_model(ctx, cfg, t, "bfloat16")
    for rows in ((600,), (350, 130, 120), (20, 40, 5, 1, 33, 501)):
        s = Session(m)
        got, at = [], 0
        for n in rows:
            got.append(s.run([("a", toks[at:at + n])])[0])
            at += n
        assert distance(np.concatenate(got), want).max() < LIMIT["bfloat16"]


@BOTH
@pytest.mark.parametrize("shift", [-80.0, 0.0, 80.0])
def test_routing_with_large_biases(ctx, shift, compute):
    """Logits all far below or above zero, and two experts that are always chosen with a weight each that differs by e^6."""
    cfg = noresun([mingru(mlp=relu2_moe(experts=12, top=4)), sigmoid_attention(mlp=relu2_moe(experts=9, top=5))])
    t = tensors(cfg, 51)
    for i in (0, 1):
        t[f"l{i}.mlp.router.b"] += np.float32(shift)
        t[f"l{i}.mlp.router.b"][1:3] += [4.0, 10.0]
    toks = draw(cfg, t, 90, 52)
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:80])])[0]] + [s.run([("a", [x])])[0] for x in toks[80:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_one_expert_takes_every_token(ctx, compute):
    cfg = noresun([mingru(mlp=relu2_moe(experts=6, top=1))])
    t = tensors(cfg, 53)
    t["l0.mlp.router.b"][:] = [0, 0, 0, 0, 40.0, 0]
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 160).tolist()
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:150])])[0]] + [s.run([("a", [x])])[0] for x in toks[150:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@pytest.mark.parametrize("in_batches", [True, False], ids=["mixed_batches", "prefill_at_admission"])
def test_generation_through_the_engine(ctx, tmp_path, mixed, in_batches):
    """registry -> engine: more requests than state slots, a pool that makes them wait, greedy tokens of every request."""
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    t, ref = mixed
    m = registry.load(ctx, write_checkpoint(tmp_path, MIXED, t), "float32", max_rows=48)
    prompts = [draw(MIXED, t, n, 60 + n) for n in (3, 40, 17, 80, 1, 29, 64)]
    e = Engine(ctx, m, num_blocks=20, block_size=16, prefill_chunk=19, mixed_batches=in_batches, state_slots=3)
    got = e.generate(prompts, 8)
    for p, out in zip(prompts, got):
        want, margin = reference_greedy(ref, p, 8)
        assert margin > 1e-4 and out == want
    assert e.stats()["free_blocks"] == 20 and e.stats()["free_state_slots"] == 3
    assert e.generate([prompts[1]], 4) == [got[1][:4]]


@pytest.mark.parametrize("layers", [MIXED["layers"], [sigmoid_attention(), sigmoid_attention(kv_from=0)]], ids=["mixed", "attention_alone"])
def test_samples_copy_the_state(ctx, tmp_path, layers):
    """A fork takes the recurrent state and the previous token with it (the only state of a model of attention layers)."""
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    cfg = {**MIXED, "layers": layers}
    t = tensors(cfg, 3)
    m = registry.load(ctx, write_checkpoint(tmp_path, cfg, t), "float32", max_rows=48)
    e = Engine(ctx, m, num_blocks=20, state_slots=4)
    p = draw(cfg, t, 37, 61)
    e.add_request(5, p, 8, samples=3)
    while e.step():
        pass
    want, margin = reference_greedy(reference(cfg, t), p, 8)
    assert margin > 1e-4 and [(i, x) for i, x, _ in e.finished()] == [(5, want)] * 3


@pytest.mark.parametrize("bigram", [None, (31, 3, 2)], ids=["no_pairs", "pairs"])
def test_prompts_that_begin_alike(ctx, tmp_path, bigram):
    """Attention alone, without token pairs, carries nothing but its cache: a prompt that begins like an earlier one resumes from its
    blocks.  With token pairs it does not, since the blocks lack the previous token."""
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    cfg = noresun([sigmoid_attention(), sigmoid_attention(kv_from=0, mlp=relu2_moe()), sigmoid_attention(window=12)], vocab=96, bigram=bigram)
    t = tensors(cfg, 25)
    ref = reference(cfg, t)
    m = registry.load(ctx, write_checkpoint(tmp_path, cfg, t), "float32", max_rows=64)
    e = Engine(ctx, m, num_blocks=40, block_size=16, prefix_cache=True)
    p = np.random.default_rng(7).integers(0, 96, 53).tolist()
    for prompt in (p, p, p[:40] + [1, 2, 3]):
        want, margin = reference_greedy(ref, prompt, 6)
        assert margin > 1e-4 and e.generate([prompt], 6) == [want]
    s = e.stats()
    assert (s["prompt_tokens_prefilled"] < s["prompt_tokens"]) == (bigram is None)


@BOTH
@pytest.mark.parametrize("n_seqs", [3, 7])
def test_steps_on_the_device_equal_single_steps(ctx, mixed, compute, n_seqs):
    """Greedy steps without returning to the host (one captured graph) choose what single steps choose."""
    t, _ = mixed
    m = device_model(ctx, MIXED, t, compute)
    names = "abcdefg"[:n_seqs]
    prompts = [draw(MIXED, t, n, n) for n in (30, 7, 55, 12, 3, 21, 44)[:n_seqs]]
    s = Session(m, slots=8)
    first = [int(np.argmax(x)) for x in s.run(list(zip(names, prompts)), False)]
    for n in names:   # room for what is to come
        while len(s.seq[n][1]) * s.bs < s.seq[n][0] + 12:
            s.seq[n][1].append(int(s.free.pop(0)))
    out = m.step_multi(first, [s.seq[n][0] for n in names], [s.seq[n][1] for n in names], s.kv, 10, s.state, [s.seq[n][2] for n in names])
    s2 = Session(m, slots=8, seed=3)
    s2.run(list(zip(names, prompts)), False)
    cur, want = first, []
    for _ in range(10):
        cur = [int(np.argmax(x)) for x in s2.run([(n, [c]) for n, c in zip(names, cur)], False)]
        want.append(cur)
    assert out.tolist() == want


def test_replay_and_command_line(tmp_path, mixed):
    """bin/trace_run and the command line as a user calls them."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    t, ref = mixed
    folder = write_checkpoint(tmp_path, MIXED, t)
    a, b = draw(MIXED, t, 70, 1), draw(MIXED, t, 20, 2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:67], "want": []}, {"id": "y", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": b[19:], "want": [0]}, {"id": "x", "tokens": a[67:], "want": [1, 2]}], "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": b, "want": [19]}], "end": ["z"]}]
    la, lb = ref.forward(a), ref.forward(b)
    want = {0: la[[0, 65]], 1: lb[[18]], 2: np.stack([lb[19], la[68], la[69]]), 3: lb[[19]]}
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(4)]
        for i, w in want.items():
            assert distance(np.fromfile(out / f"{i}.f32", "<f4").reshape(w.shape), w).max() < LIMIT[dtype]
    r = subprocess.run([sys.executable, "-m", "paged_infer_b200", "generate", "--model", folder, "--dtype", "float32", "--tokens",
                        ",".join(map(str, b)), "--tokens", "5,6", "--max-tokens", "6"], capture_output=True, text=True, cwd=root, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, reference_greedy(ref, p, 6)[0])) for p in (b, [5, 6])]


def test_wrong_configurations_are_errors(ctx):
    from paged_infer_b200.api import PiError
    for layers, why in (([sigmoid_attention(heads=5, kv_heads=2)], "share"), ([sigmoid_attention(rot=22)], "rotary"),
                        ([mingru(), sigmoid_attention(kv_from=0)], "no keys and values to share"), ([sigmoid_attention(kv_from=0)], "no keys and values to share"),
                        ([sigmoid_attention(), sigmoid_attention(kv_from=0), sigmoid_attention(kv_from=1)], "no keys and values to share"),
                        ([sigmoid_attention(), sigmoid_attention(vdim=12, kv_from=0)], "heads differ"),
                        ([mingru(mlp=relu2_moe(experts=3, top=4))], "experts per token")):
        cfg = noresun(layers)
        with pytest.raises(PiError, match=why):
            device_model(ctx, cfg, tensors(cfg, 1), "float32")
    cfg = noresun([sigmoid_attention(mlp=relu2_moe()), mingru()])
    t = tensors(cfg, 4)
    for missing in ("l0.mlp.e11.down", "l0.mlp.router.b", "l0.rg2", "l0.rg1.b", "bigram", "l0.norm2", "l0.mix.pb", "l0.mix.q.norm", "l1.mix.x.b"):
        with pytest.raises(PiError, match=f"missing tensor: {missing}"):
            device_model(ctx, cfg, {k: v for k, v in t.items() if k != missing}, "float32")
