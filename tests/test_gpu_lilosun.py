"""Lilosun on the device against the plain reference: every mechanism alone, prefill against decoding, portions, mixed batches,
blocks and slots used again, window edges, routing, and generation through the engine.  Both number formats."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from layered_helpers import (LIMIT, Session, dense, device_model, distance, draw, latent, lilosun, mamba2, moe, reference, tensors,
                             write_checkpoint)
from test_gpu_layered import reference_greedy

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("compute", ["float32", "bfloat16"])


@pytest.fixture(scope="module")
def ctx():
    from paged_infer_b200 import api
    return api.Context(0)


# what one layer can be, in sizes that hit the kernels' special cases
ALONE = {
    "latent": latent(),
    "latent_plain_rotation": latent(scaling=None, heads=2, dim=8, rot_dim=4, vdim=12, rank=16),
    "latent_everything": latent(window=None, heads=5, rank=40),
    "latent_window1": latent(window=1, heads=2),
    "latent_wide_window": latent(window=1000, scale=0.05),
    "latent_odd": latent(heads=3, dim=11, rot_dim=6, vdim=9, rank=33, window=19),
    "latent_odd_rank": latent(heads=1, dim=10, rot_dim=2, vdim=7, rank=21, window=70),
    "latent_17_heads": latent(heads=17, dim=16, rot_dim=16, vdim=16, rank=80, window=90),
    "latent_rank200": latent(heads=4, dim=40, rot_dim=24, vdim=72, rank=200, window=77),
    "latent_rank512": latent(heads=2, dim=128, rot_dim=64, vdim=128, rank=512, window=100, scale=0.1),
    "latent_big_heads": latent(heads=2, dim=200, rot_dim=40, vdim=150, rank=64, window=50),
    "latent_huge_keys": latent(heads=1, dim=280, rot_dim=16, vdim=20, rank=300, window=40),
    "yarn_steep": latent(scaling={"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}, rot_dim=64, window=60, base=500.0),
    "yarn_one_pair": latent(scaling={"factor": 2.5, "original": 64, "fast": 3.0, "slow": 2.9}, rot_dim=10, window=None),
    "mamba2": mamba2(),
    "mamba2_one_group": mamba2(heads=8, vdim=16, state=16, groups=1, norm_groups=1, conv=4),
    "mamba2_group_per_head": mamba2(heads=5, vdim=8, state=12, groups=5, norm_groups=5, conv=2),
    "mamba2_no_memory_conv": mamba2(heads=2, vdim=32, state=8, groups=1, norm_groups=2, conv=1),
    "mamba2_long_conv": mamba2(heads=4, vdim=12, state=20, groups=2, norm_groups=4, conv=7),
    "mamba2_odd": mamba2(heads=3, vdim=7, state=5, groups=3, norm_groups=7, conv=3),
    "mamba2_large": mamba2(heads=8, vdim=64, state=128, groups=1, norm_groups=1, conv=4),
    "mamba2_wide_value": mamba2(heads=2, vdim=200, state=40, groups=1, norm_groups=2, conv=4),
    "mamba2_wide_state": mamba2(heads=2, vdim=36, state=250, groups=2, norm_groups=1, conv=4),
    "mamba2_state_in_memory": mamba2(heads=1, vdim=128, state=300, groups=1, norm_groups=1, conv=4),
    "dense": mamba2(mlp=dense(50)),
    "dense_odd": latent(heads=1, mlp=dense(13)),
    "moe": mamba2(mlp=moe()),
    "moe_top1": latent(mlp=moe(experts=8, top=1, ff=24, groups=(2, 1))),
    "moe_all": mamba2(mlp=moe(experts=4, top=4, ff=33, groups=None)),
    "moe_no_shared": mamba2(mlp=moe(experts=10, top=2, ff=48, groups=(5, 3), shared=None)),
    "moe_groups_of_one": latent(mlp=moe(experts=6, top=2, ff=20, groups=(6, 4), limit=0.5)),
    "moe_keeps_all_groups": mamba2(mlp=moe(experts=6, top=2, ff=20, groups=(2, 2), limit=7.0, shared_limit=3.0)),
    "moe_many": mamba2(mlp=moe(experts=70, top=6, ff=17, groups=(7, 3), shared=31)),
}
MIXED = lilosun([latent(mlp=moe()), mamba2(mlp=dense()), mamba2(mlp=moe(experts=10, groups=None, top=2)), latent(window=40, heads=5, rank=33, dim=14, mlp=moe(shared=None)),
                 mamba2(heads=4, vdim=24, state=16, groups=1, norm_groups=2, conv=4), latent(window=None, scaling=None, heads=2, mlp=dense(31))], vocab=500)


@pytest.fixture(scope="module")
def mixed():
    t = tensors(MIXED, 3)
    return t, reference(MIXED, t)


@BOTH
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(ctx, name, compute):
    """Residual stream and logits of a one-layer model: a prompt in one step, then token by token."""
    cfg = lilosun([ALONE[name]], width=72, vocab=240)
    t = tensors(cfg, 11)
    toks = draw(cfg, t, 150, 5)
    layer = []
    want = reference(cfg, t).forward(toks, layer)
    m = device_model(ctx, cfg, t, compute)
    s = Session(m)
    m.trace_layers(True)
    got = s.run([("a", toks[:141])])[0]
    x = m.read_layer(0, 141)
    m.trace_layers(False)
    lim = LIMIT[compute]
    assert distance(x, layer[0][:141]).max() < lim
    assert distance(got, want[:141]).max() < lim
    for i in range(141, 150):
        assert distance(s.run([("a", [toks[i]])])[0], want[i:i + 1]).max() < 1.5 * lim


@BOTH
def test_decoding_equals_prefill(ctx, mixed, compute):
    t, ref = mixed
    toks = draw(MIXED, t, 100, 8)
    want = ref.forward(toks)
    m = device_model(ctx, MIXED, t, compute)
    s = Session(m, block_size=16)
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
    m = device_model(ctx, MIXED, t, compute)
    s = Session(m, blocks=40, slots=3)
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


def needle_model(window):
    """One latent attention layer in which token SEEKER looks for token NEEDLE through an unrotated channel of every head, fed by
    a latent channel that only NEEDLE fills: one score stands far above all others."""
    heads, dim, rot = 3, 12, 8
    cfg = lilosun([latent(heads, dim, rot, 20, 24, window, scale=1.0)], width=64, vocab=96)
    t = tensors(cfg, 21)
    e = t["embed"]
    e[:, 40:42] = 0
    e[NEEDLE, 40] = 10.0
    e[SEEKER, 41] = 10.0
    t["l0.norm1"][:] = 1.0
    t["l0.ls1"][:] = 2.0
    t["l0.mix.dkv"][0, :] = 0
    t["l0.mix.dkv"][0, 40] = 2.0
    t["l0.mix.dkv.norm"][0] = 1.0
    t["l0.mix.q"][:, 40:42] = 0
    for h in range(heads):
        t["l0.mix.uk"][h * dim] = 0
        t["l0.mix.uk"][h * dim, 0] = 2.0
        q = t["l0.mix.q"][h * (dim + rot)]
        q[:] = 0
        q[41] = 1.0
    return cfg, t


@BOTH
@pytest.mark.parametrize("window", [1, 2, 16, 17, 47, 64, 65, 130])
def test_window_edge(ctx, window, compute):
    """NEEDLE just inside and just outside the window of SEEKER, at block and tile borders, read in a prompt, in a portion of
    two and when decoded."""
    cfg, t = needle_model(window)
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
def test_far_key_without_a_window(ctx, compute):
    """The first token among hundreds of keys, in a prompt, in portions and decoded far along (keys cut over a cluster)."""
    cfg, t = needle_model(None)
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
def test_first_token_is_remembered(ctx, compute):
    """A slow decay: the first token still moves the logits hundreds of tokens on, through portions and decoding."""
    cfg = lilosun([mamba2(conv=4)], vocab=96)
    t = tensors(cfg, 31)
    t["l0.mix.A_log"][:] = -9.0
    t["l0.mix.dt_bias"][:] = 0.0
    t["embed"][7] *= 4
    toks = [7] + np.random.default_rng(5).integers(8, 96, 320).tolist()
    ref = reference(cfg, t)
    want = ref.forward(toks)
    assert distance(ref.forward([8] + toks[1:])[-1:], want[-1:]).max() > 50 * LIMIT["float32"]
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:200])])[0], s.run([("a", toks[200:270])])[0]] + [s.run([("a", [x])])[0] for x in toks[270:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_convolution_over_the_cut(ctx, compute):
    """A long convolution whose earliest tap is by far the strongest: portions shorter than it, of its length and longer, from
    slots that held another sequence."""
    cfg = lilosun([mamba2(heads=2, vdim=16, state=8, groups=1, norm_groups=1, conv=6)], vocab=96)
    t = tensors(cfg, 33)
    t["l0.mix.conv"][:, 0] *= 6
    m = device_model(ctx, cfg, t, compute)
    ref = reference(cfg, t)
    s = Session(m, slots=1)
    rng = np.random.default_rng(0)
    for n, size in enumerate((1, 2, 3, 4, 5, 6, 7, 64, 67)):
        toks = rng.integers(0, 96, 40 if size < 60 else 150).tolist()
        got = np.concatenate([s.run([(n, toks[i:i + size])])[0] for i in range(0, len(toks), size)])
        assert distance(got, ref.forward(toks)).max() < LIMIT[compute], size
        s.close(n)


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
    cfg = lilosun([latent(heads=8, dim=64, rot_dim=32, vdim=64, rank=128, window=100, mlp=moe(experts=16, top=2, ff=136, groups=(4, 2), shared=200)),
                   mamba2(heads=12, vdim=32, state=64, groups=2, norm_groups=2, conv=4, mlp=moe(experts=5, top=3, ff=300, groups=None, shared=None)),
                   mamba2(heads=4, vdim=64, state=128, groups=1, norm_groups=1, conv=4, mlp=dense(1000))], width=520, vocab=1000)
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
@pytest.mark.parametrize("shift", [-3.0, 0.0, 3.0])
def test_routing_with_large_corrections(ctx, shift, compute):
    """Choice scores all negative or all far above 1: what is masked counts as minus infinity, and the correction leaves the
    weights alone."""
    cfg = lilosun([mamba2(mlp=moe(experts=12, top=4, groups=(4, 2), shared=None)), latent(mlp=moe(experts=9, top=5, groups=(3, 2)))])
    t = tensors(cfg, 51)
    for i in (0, 1):
        t[f"l{i}.mlp.correction"] += np.float32(shift)
    toks = draw(cfg, t, 90, 52)
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:80])])[0]] + [s.run([("a", [x])])[0] for x in toks[80:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_all_tokens_on_one_expert(ctx, compute):
    """The most uneven load: every token chooses the same experts, the others get none."""
    cfg = lilosun([mamba2(mlp=moe(experts=20, top=2, groups=None, ff=24))])
    t = tensors(cfg, 61)
    t["l0.mlp.correction"][:] = -1.0
    t["l0.mlp.correction"][[3, 17]] = 4.0
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 300).tolist()
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:290])])[0], s.run([("a", toks[290:])])[0]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@pytest.mark.parametrize("layer", [mamba2(heads=4, vdim=64, state=128, groups=1, norm_groups=1, conv=4), mamba2(heads=6, vdim=20, state=24, groups=2), mamba2(heads=3, vdim=7, state=5, groups=1, norm_groups=1),
                                   mamba2(heads=2, vdim=150, state=40, groups=1, norm_groups=1)], ids=lambda l: f"{l['mixer']['state']}-{l['mixer']['vdim']}")
@pytest.mark.parametrize("gates", ["plain", "extreme"])
def test_chunks_equal_token_by_token(ctx, layer, gates):
    """The chunked kernels against the scan on the same projections (both in the bf16 mode): far tighter than bf16 itself."""
    cfg = lilosun([layer], width=48, vocab=96)
    t = tensors(cfg, 41)
    if gates == "extreme":    # heads that empty their state within a token beside heads that never forget
        t["l0.mix.A_log"][::2], t["l0.mix.A_log"][1::2] = 5.0, -8.0
        t["l0.mix.dt_bias"][:] = 2.0
    m = device_model(ctx, cfg, t, "bfloat16")
    toks = np.random.default_rng(42).integers(0, 96, 64 * 3 + 21).tolist()
    outs = []
    for size in (len(toks), 63, 64 + 37):    # all chunks; scan only; both, with the state handed over
        s = Session(m)
        outs.append(np.concatenate([s.run([("a", toks[i:i + size])])[0] for i in range(0, len(toks), size)]))
    assert np.isfinite(outs[0]).all()
    assert distance(outs[0], outs[1]).max() < 6e-3 and distance(outs[2], outs[1]).max() < 6e-3
    want = reference(cfg, t).forward(toks)
    assert distance(outs[0], want).max() < LIMIT["bfloat16"]
    exact = Session(device_model(ctx, cfg, t, "float32")).run([("a", toks)])[0]
    assert distance(exact, want).max() < LIMIT["float32"]


def test_expanded_equals_absorbed(ctx):
    """Long portions with keys and values spelled out against short ones over the latents: the same projections, two ways."""
    cfg = lilosun([latent(heads=6, dim=24, rot_dim=16, vdim=40, rank=64, window=90)], vocab=96)
    t = tensors(cfg, 43)
    m = device_model(ctx, cfg, t, "bfloat16")
    toks = np.random.default_rng(44).integers(0, 96, 330).tolist()
    outs = []
    for size in (330, 63, 100):
        s = Session(m, block_size=12)
        outs.append(np.concatenate([s.run([("a", toks[i:i + size])])[0] for i in range(0, len(toks), size)]))
    assert distance(outs[0], outs[1]).max() < 1e-2 and distance(outs[2], outs[1]).max() < 1e-2


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


def test_samples_copy_the_state(ctx, tmp_path, mixed):
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    t, ref = mixed
    m = registry.load(ctx, write_checkpoint(tmp_path, MIXED, t), "float32", max_rows=48)
    e = Engine(ctx, m, num_blocks=20, state_slots=4)
    p = draw(MIXED, t, 37, 61)
    e.add_request(5, p, 8, samples=3)
    while e.step():
        pass
    want, _ = reference_greedy(ref, p, 8)
    assert [(i, x) for i, x, _ in e.finished()] == [(5, want)] * 3


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
    for layer, why in ((mamba2(heads=6, groups=4), "groups"), (mamba2(norm_groups=7), "parts"), (mamba2(mlp=moe(experts=12, groups=(5, 2))), "groups"),
                       (mamba2(mlp=moe(experts=12, top=5, groups=(3, 1))), "experts per token"), (latent(rot_dim=7), "rotary"),
                       (latent(scaling={"factor": 2.0, "original": 0, "fast": 1.0, "slow": 1.0}), "rotary scaling")):
        cfg = lilosun([layer])
        with pytest.raises(PiError, match=why):
            device_model(ctx, cfg, {"embed": np.zeros((cfg["vocab"], 88), np.float32), "head": np.zeros((cfg["vocab"], 88), np.float32),
                                    "final.norm": np.zeros(88, np.float32)}, "float32")
    cfg = lilosun([mamba2(mlp=moe())])
    t = tensors(cfg, 4)
    with pytest.raises(PiError, match="missing tensor: l0.mlp.e11.down"):
        device_model(ctx, cfg, {k: v for k, v in t.items() if k != "l0.mlp.e11.down"}, "float32")
