"""Layered designs on the device against the plain reference: every mechanism alone, prefill against decoding, portions,
mixed batches, blocks and slots used again, window edges, and generation through the engine.  Both number formats."""
import numpy as np
import pytest

from layered_helpers import (LIMIT, Session, attention, config, device_model, distance, gla, mlstm, reference, tensors, write_checkpoint)

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("compute", ["float32", "bfloat16"])


@pytest.fixture(scope="module")
def ctx():
    from paged_infer_b200 import api
    return api.Context(0)


def tokens(n, seed, vocab=96):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


# what one layer can be, in sizes that hit the kernels' special cases: channels that are no multiple of a tile, one head,
# one key/value head per query head, groups of 1..8 heads, partial and no rotation, windows of 1, of odd size, and beyond any prompt
ALONE = {
    "attention": attention(),
    "attention_gqa8": attention(heads=8, kv_heads=1, dim=32, vdim=64, window=40, ff=0),
    "attention_group3": attention(heads=6, kv_heads=2, dim=24, vdim=20, window=33, rot=8, diff=0.7),
    "attention_mha": attention(heads=3, kv_heads=3, dim=64, vdim=128, window=100, rot=32, base=500.0, ff=0),
    "attention_wide": attention(heads=2, kv_heads=1, dim=128, vdim=256, window=1000, scale=0.2, ff=0),
    "attention_window1": attention(heads=2, kv_heads=1, dim=6, vdim=10, window=1, ff=0),
    "attention_odd_dim": attention(heads=4, kv_heads=2, dim=11, vdim=9, window=19, rot=4, ff=0),
    "attention_no_rotation": attention(heads=5, kv_heads=1, dim=18, vdim=34, window=17, rot=0, ff=31),
    "attention_group12": attention(heads=12, kv_heads=1, dim=16, vdim=16, window=50, ff=0),
    "gla": gla(),
    "gla_ff": gla(heads=2, dim=32, vdim=64, tau=16.0, ff=40),
    "gla_fast_decay": gla(heads=1, dim=20, vdim=36, tau=0.5),
    "gla_tau1": gla(heads=4, dim=64, vdim=128, tau=1.0),
    "gla_odd": gla(heads=3, dim=13, vdim=23, tau=4.0),
    "gla_wide": gla(heads=1, dim=48, vdim=272, tau=8.0),
    "mlstm": mlstm(),
    "mlstm_ff": mlstm(heads=4, dim=32, vdim=32, cap=15.0, ff=72),
    "mlstm_tight_cap": mlstm(heads=3, dim=64, vdim=128, cap=1.0),
    "mlstm_odd": mlstm(heads=1, dim=11, vdim=19, cap=3.0),
    "mlstm_wide": mlstm(heads=2, dim=80, vdim=160, cap=20.0),
    "mlstm_wide_key": mlstm(heads=1, dim=288, vdim=64, cap=8.0),
}
MIXED = config([attention(window=20), gla(ff=40), mlstm(), attention(heads=6, kv_heads=3, dim=24, vdim=40, window=37, rot=16, diff=0.5, ff=0),
                mlstm(heads=3, dim=16, vdim=16, cap=4.0, ff=33), gla(heads=2, dim=40, vdim=72, tau=2.0)], width=72, vocab=120)


@BOTH
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(ctx, name, compute):
    """Residual stream and logits of a one-layer model: a prompt in one step, then token by token."""
    cfg = config([ALONE[name]], width=56, vocab=88, eps=1e-5)
    t = tensors(cfg, 11)
    toks = tokens(150, 5, 88)
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
def test_decoding_equals_prefill(ctx, compute):
    t = tensors(MIXED, 2)
    toks = tokens(90, 8, MIXED["vocab"])
    want = reference(MIXED, t).forward(toks)
    m = device_model(ctx, MIXED, t, compute)
    s = Session(m, block_size=16)
    whole = s.run([("whole", toks)])[0]
    one = np.concatenate([s.run([("one", [x])])[0] for x in toks])
    assert distance(whole, want).max() < LIMIT[compute]
    assert distance(one, want).max() < LIMIT[compute]


@BOTH
@pytest.mark.parametrize("size", [2, 3, 7, 16, 63, 64, 65, 128, 129])
def test_portions(ctx, size, compute):
    t = tensors(MIXED, 3)
    toks = tokens(200 if size > 7 else 70, 9, MIXED["vocab"])
    want = reference(MIXED, t).forward(toks)
    m = device_model(ctx, MIXED, t, compute)
    s = Session(m, block_size=8)
    got = np.concatenate([s.run([("p", toks[i:i + size])])[0] for i in range(0, len(toks), size)])
    assert distance(got, want).max() < LIMIT[compute]


@BOTH
def test_uneven_batches_and_reuse(ctx, compute):
    """Portions beside single tokens, requests that pause, end and make room; freed blocks and slots are used at once."""
    t = tensors(MIXED, 4)
    m = device_model(ctx, MIXED, t, compute)
    ref = reference(MIXED, t)
    s = Session(m, blocks=40, slots=3)
    rng = np.random.default_rng(1)
    live, got, done = {}, {}, 0
    for i in range(60):
        while len(live) < 3 and done + len(live) < 9:
            name = f"r{done + len(live)}.{i}"
            live[name] = tokens(int(rng.choice([1, 2, 19, 64, 150])), 100 + i + len(live), MIXED["vocab"])
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
                want = ref.forward(live[name])
                assert distance(np.concatenate(got[name]), want).max() < LIMIT[compute], name
                s.close(name)
                del live[name]
                done += 1
    assert done == 9


@BOTH
def test_batch_does_not_change_a_row(ctx, compute):
    t = tensors(MIXED, 6)
    m = device_model(ctx, MIXED, t, compute)
    toks = {n: tokens(k, 40 + k, MIXED["vocab"]) for n, k in (("a", 33), ("b", 70), ("c", 5), ("d", 101))}
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


def needle_model(window, heads=4, kv_heads=2, dim=16, vdim=32):
    """One attention layer in which token SEEKER looks for token NEEDLE: one score stands far above all others, so a key
    that is lost or wrongly seen shows.  Scores come from a channel that is not rotated."""
    cfg = config([attention(heads, kv_heads, dim, vdim, window, rot=8, diff=0.3, scale=1.0, ff=0)], width=64, vocab=96)
    t = tensors(cfg, 21)
    e = t["embed"]
    e[:, :2] = 0
    e[NEEDLE, 0] = 8.0
    e[SEEKER, 1] = 8.0
    t["l0.norm1"][:] = 1.0
    t["l0.norm1.b"][:] = 0.0
    for name, channel, n in (("q", 1, heads), ("k", 0, kv_heads)):
        w = t["l0.mix." + name]
        w[:, :2] = 0
        for h in range(n):
            w[h * 2 * dim + dim - 1, :] = 0          # last channel of map 1: the marker alone
            w[h * 2 * dim + dim - 1, channel] = 4.0
    return cfg, t


@BOTH
@pytest.mark.parametrize("window", [1, 2, 16, 17, 47, 64, 130])
def test_window_edge(ctx, window, compute):
    """NEEDLE just inside and just outside the window of SEEKER, at block borders, read in a prompt, in a portion of two and
    when decoded."""
    cfg, t = needle_model(window)
    ref = reference(cfg, t)
    m = device_model(ctx, cfg, t, compute)
    fill = [x + 3 for x in tokens(400, 3, 90)]
    power = []
    for back in sorted({window - 1, window, window + 1} - {0}):
        for at in (back, back + 15, back + 16, back + 33):      # SEEKER's position; NEEDLE at at - back: 0, 15, 16, 33
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
@pytest.mark.parametrize("layer", [gla(tau=64.0), mlstm(cap=15.0)], ids=["gla", "mlstm"])
def test_first_token_is_remembered(ctx, layer, compute):
    """A slow decay: the first token still moves the logits hundreds of tokens on, through portions and decoding."""
    cfg = config([layer])
    t = tensors(cfg, 31)
    if layer["type"] == "gla":
        t["l0.mix.a2.b"][:] = 6.0
    else:
        t["l0.mix.f.b"][:] = 9.0
    t["embed"][7] *= 4
    t["l0.norm1.alpha"] = np.float32(0.25)
    toks = [7] + [x + 8 for x in tokens(320, 5, 80)]
    ref = reference(cfg, t)
    want = ref.forward(toks)
    assert distance(ref.forward([8] + toks[1:])[-1:], want[-1:]).max() > 10 * LIMIT["float32"]
    m = device_model(ctx, cfg, t, compute)
    s = Session(m)
    got = [s.run([("a", toks[:200])])[0], s.run([("a", toks[200:270])])[0]] + [s.run([("a", [x])])[0] for x in toks[270:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_long_decoding(ctx, compute):
    t = tensors(MIXED, 12)
    m = device_model(ctx, MIXED, t, compute)
    toks = tokens(300, 13, MIXED["vocab"])
    want = reference(MIXED, t).forward(toks)
    s = Session(m)
    got = np.concatenate([s.run([("a", [x]), ("b", [y])])[0] for x, y in zip(toks, reversed(toks))])
    assert distance(got, want).max() < LIMIT[compute]


def test_wide_model_many_rows(ctx):
    """Sizes that fill the tensor-core tiles and cut K over clusters, up to several hundred rows."""
    cfg = config([attention(heads=8, kv_heads=2, dim=64, vdim=128, window=100, ff=1000), gla(heads=4, dim=64, vdim=128, tau=16.0),
                  mlstm(heads=4, dim=64, vdim=128)], width=520, vocab=1000)
    t = tensors(cfg, 14, rank=16)
    toks = tokens(330, 15, 1000)
    want = reference(cfg, t).forward(toks)
    m = device_model(ctx, cfg, t, "bfloat16")
    for rows in ((330,), (200, 130), (20, 40, 5, 1, 264)):
        s = Session(m)
        got, at = [], 0
        for n in rows:
            got.append(s.run([("a", toks[at:at + n])])[0])
            at += n
        assert distance(np.concatenate(got), want).max() < LIMIT["bfloat16"]


@BOTH
def test_sizes_that_are_multiples_of_nothing(ctx, compute):
    cfg = config([attention(heads=3, kv_heads=1, dim=10, vdim=7, window=21, rot=6, ff=13), gla(heads=1, dim=5, vdim=3, ff=1),
                  mlstm(heads=1, dim=3, vdim=6), mlstm(heads=3, dim=9, vdim=131), gla(heads=2, dim=31, vdim=65, tau=1.5)], width=37, vocab=41)
    t = tensors(cfg, 71, rank=3)
    toks = tokens(160, 72, 41)
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute), block_size=5)
    got = [s.run([("a", toks[:139])])[0], s.run([("a", toks[139:150])])[0]] + [s.run([("a", [c])])[0] for c in toks[150:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute] * 1.5


def reference_greedy(ref, prompt, n):
    toks, margin = list(prompt), np.inf
    for _ in range(n):
        l = ref.forward(toks)[-1]
        top = np.sort(l)[-2:]
        margin = min(margin, top[1] - top[0])
        toks.append(int(np.argmax(l)))
    return toks[len(prompt):], margin


@pytest.mark.parametrize("mixed", [True, False], ids=["mixed_batches", "prefill_at_admission"])
def test_generation_through_the_engine(ctx, tmp_path, mixed):
    """registry -> engine: more requests than state slots, a pool that makes them wait, greedy tokens of every request."""
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    t = tensors(MIXED, 17)
    m = registry.load(ctx, write_checkpoint(tmp_path, MIXED, t), "float32", max_rows=48)
    prompts = [tokens(n, 60 + n, MIXED["vocab"]) for n in (3, 40, 17, 80, 1, 29, 64)]
    e = Engine(ctx, m, num_blocks=20, block_size=16, prefill_chunk=19, mixed_batches=mixed, state_slots=3)
    got = e.generate(prompts, 12)
    ref = reference(MIXED, t)
    for p, out in zip(prompts, got):
        want, margin = reference_greedy(ref, p, 12)
        assert margin > 1e-4 and out == want
    assert e.stats()["free_blocks"] == 20 and e.stats()["free_state_slots"] == 3
    assert e.generate([prompts[1]], 4) == [got[1][:4]]


def test_samples_copy_the_state(ctx, tmp_path):
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    t = tensors(MIXED, 17)
    m = registry.load(ctx, write_checkpoint(tmp_path, MIXED, t), "float32", max_rows=48)
    e = Engine(ctx, m, num_blocks=20, state_slots=4)
    p = tokens(37, 61, MIXED["vocab"])
    e.add_request(5, p, 8, samples=3)
    while e.step():
        pass
    want, _ = reference_greedy(reference(MIXED, t), p, 8)
    assert [(i, x) for i, x, _ in e.finished()] == [(5, want)] * 3


@BOTH
def test_steps_on_the_device_equal_single_steps(ctx, compute):
    """Greedy steps without returning to the host (one captured graph) choose what single steps choose."""
    t = tensors(MIXED, 18)
    m = device_model(ctx, MIXED, t, compute)
    prompts = [tokens(n, n, MIXED["vocab"]) for n in (30, 7, 55)]
    s = Session(m)
    first = [int(np.argmax(x)) for x in s.run(list(zip("abc", prompts)), False)]
    for n in "abc":   # room for what is to come
        while len(s.seq[n][1]) * s.bs < s.seq[n][0] + 12:
            s.seq[n][1].append(int(s.free.pop(0)))
    out = m.step_multi(first, [s.seq[n][0] for n in "abc"], [s.seq[n][1] for n in "abc"], s.kv, 10, s.state, [s.seq[n][2] for n in "abc"])
    s2 = Session(m, seed=3)
    s2.run(list(zip("abc", prompts)), False)
    cur, want = first, []
    for _ in range(10):
        cur = [int(np.argmax(x)) for x in s2.run([(n, [c]) for n, c in zip("abc", cur)], False)]
        want.append(cur)
    assert out.tolist() == want


def test_replay_and_command_line(ctx, tmp_path):
    """bin/trace_run and the command line as a user calls them."""
    import json
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    t = tensors(MIXED, 19)
    folder = write_checkpoint(tmp_path, MIXED, t)
    a, b = tokens(70, 1, MIXED["vocab"]), tokens(20, 2, MIXED["vocab"])
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:67], "want": []}, {"id": "y", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": b[19:], "want": [0]}, {"id": "x", "tokens": a[67:], "want": [1, 2]}], "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": b, "want": [19]}], "end": ["z"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "192"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(4)]
    ref = reference(MIXED, t)
    la, lb = ref.forward(a), ref.forward(b)
    want = {0: la[[0, 65]], 1: lb[[18]], 2: np.stack([lb[19], la[68], la[69]]), 3: lb[[19]]}
    for i, w in want.items():
        got = np.fromfile(out / f"{i}.f32", "<f4").reshape(w.shape)
        assert distance(got, w).max() < LIMIT["float32"]
    r = subprocess.run([sys.executable, "-m", "paged_infer_b200", "generate", "--model", folder, "--dtype", "float32", "--tokens",
                        ",".join(map(str, b)), "--tokens", "5,6", "--max-tokens", "6"], capture_output=True, text=True, cwd=root, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, reference_greedy(ref, p, 6)[0])) for p in (b, [5, 6])]


def test_wrong_arguments_are_errors(ctx):
    from paged_infer_b200.api import PiError
    t = tensors(MIXED, 4)
    m = device_model(ctx, MIXED, t, "float32", max_rows=8)
    kv, st = m.kv_pool(4, 16), m.state_pool(2)
    for kw in (dict(slots=[2]), dict(slots=None), dict(slots=[-1])):
        with pytest.raises(PiError):
            m.step([[1]], [0], [[0]], kv, st, **kw)
    with pytest.raises(PiError, match="share state slot"):
        m.step([[1], [2]], [0, 0], [[0], [1]], kv, st, [1, 1])
    with pytest.raises(PiError, match="rows"):
        m.step([list(range(9))], [0], [[0]], kv, st, [0])
    with pytest.raises(PiError, match="physical id"):
        m.step([[1]], [0], [[4]], kv, st, [0])
    with pytest.raises(PiError, match="missing tensor: l1.mix.a1"):
        device_model(ctx, MIXED, {k: v for k, v in t.items() if k != "l1.mix.a1"}, "float32")


def test_ragged_step_of_a_llama(ctx):
    """The same step call on the uniform models: portions and single tokens in one batch, rows picked from it."""
    from helpers import load_golden
    from paged_infer_b200 import api
    cfg, toks, golden, hw = load_golden()
    m = api.LlamaWeights(ctx, cfg, hw, max_batch=64)
    kv = m.kv_pool(8, 16)
    ta, tb = [3, 1, 5], [0, 7, 2]
    m.step([toks[:9].tolist()], [0], [ta], kv)
    got = m.step([toks[:20].tolist(), toks[9:10].tolist()], [0, 9], [tb, ta], kv, out_rows=[4, 19, 20])
    assert np.abs(got - golden[[4, 19, 9]]).max() < 5e-4
    got, ids = m.step([toks[10:11].tolist(), toks[20:21].tolist()], [10, 20], [ta, tb], kv, want_argmax=True)
    assert np.abs(got - golden[[10, 20]]).max() < 5e-4 and ids.tolist() == golden[[10, 20]].argmax(-1).tolist()


@pytest.mark.parametrize("n,k", [(33, 100), (128, 64), (600, 1000), (2048, 512), (20, 8), (4100, 2056), (130, 4096)])
def test_bf16_projection(ctx, n, k):
    """Every tile width, K split over clusters and not, sizes that are no multiple of anything, against f32 on the host."""
    import torch
    from paged_infer_b200 import api
    from paged_infer_b200.loader import bf16_bits_to_f32, f32_to_bf16_bits
    rng = np.random.default_rng(n)
    w = f32_to_bf16_bits(rng.standard_normal((n, k)).astype(np.float32))
    lin = api.Projection.f32(ctx, w)
    ld = (k + 7) // 8 * 8
    for m in (1, 5, 16, 17, 32, 40, 64, 100, 128, 129, 300, 700):
        x = f32_to_bf16_bits(rng.standard_normal((m, ld)).astype(np.float32))   # what lies behind k is garbage
        xd = torch.from_numpy(x.view(np.int16)).cuda()
        out = torch.full((m, n), 7.0, device="cuda")
        lin.apply_device_bf16(xd, ld, out, m)
        ctx.synchronize()
        want = bf16_bits_to_f32(x)[:, :k].astype(np.float64) @ bf16_bits_to_f32(w).T.astype(np.float64)
        assert np.abs(out.cpu().numpy() - want).max() < 3e-5 * np.sqrt(k), (m, n, k)


def extreme(t, kind):
    """Gates far out: GLA decays that empty the state within a few tokens next to channels that never forget; mLSTM input
    gates that jump over tens of units."""
    if kind == "gla":
        b = t["l0.mix.a2.b"]
        b[::3], b[1::3], b[2::3] = -40.0, 12.0, 0.0
    elif kind == "mlstm":
        t["l0.mix.i"] *= 16
        t["l0.mix.f"] *= 16
    return t


@pytest.mark.parametrize("layer", [gla(heads=2, dim=64, vdim=128, tau=0.5), gla(heads=3, dim=40, vdim=72, tau=16.0), gla(heads=1, dim=128, vdim=256, tau=2.0),
                                   gla(heads=2, dim=13, vdim=19, tau=1.0), mlstm(heads=2, dim=128, vdim=256, cap=30.0), mlstm(heads=3, dim=24, vdim=40, cap=15.0),
                                   mlstm(heads=1, dim=17, vdim=150, cap=60.0)], ids=lambda l: f"{l['type']}-{l['mixer']['dim']}-{l['mixer']['vdim']}")
@pytest.mark.parametrize("gates", ["plain", "extreme"])
def test_chunks_equal_token_by_token(ctx, layer, gates):
    """The chunked kernels against the scan on the same projections (both in the bf16 mode): far tighter than bf16 itself."""
    cfg = config([layer], width=48)
    t = tensors(cfg, 41)
    if gates == "extreme":
        t = extreme(t, layer["type"])
    m = device_model(ctx, cfg, t, "bfloat16")
    toks = tokens(64 * 3 + 21, 42)
    outs = []
    for size in (len(toks), 63, 64 + 37):    # all chunks; scan only; both, with the state handed over
        s = Session(m)
        outs.append(np.concatenate([s.run([("a", toks[i:i + size])])[0] for i in range(0, len(toks), size)]))
    assert np.isfinite(outs[0]).all()
    assert distance(outs[0], outs[1]).max() < 6e-3 and distance(outs[2], outs[1]).max() < 6e-3
    # steep gates turn the rounding of the bf16 input into a wider error; the f32 mode has none of it
    want = reference(cfg, t).forward(toks)
    assert distance(outs[0], want).max() < (LIMIT["bfloat16"] if gates == "plain" else 0.2)
    exact = Session(device_model(ctx, cfg, t, "float32")).run([("a", toks)])[0]
    assert distance(exact, want).max() < 5 * LIMIT["float32"]


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_one_softmax_map(ctx, compute):
    """Plain grouped attention (one map) is the same mechanism with its constants: against the reference's window softmax."""
    from oracle import layers as L
    from layered_helpers import bits
    from paged_infer_b200 import api, loader
    H, G, D, E, W, T = 20, 1, 24, 40, 48, 130
    two = config([attention(H, G, D, E, 50, ff=0)], width=W)
    t = tensors(two, 51)
    t["l0.mix.q"] = t["l0.mix.q"].reshape(H, 2, D, W)[:, 0].reshape(H * D, W).copy()
    t["l0.mix.k"] = t["l0.mix.k"].reshape(G, 2, D, W)[:, 0].reshape(G * D, W).copy()
    cfg = loader.LayeredConfig(W, 96, 1e-5, [loader.LayerConfig(loader.MIXER_ATTENTION, heads=H, kv_heads=G, dim=D, vdim=E, maps=1, window=None,
                                                               rot_dims=10, rot_base=300.0, scale=0.3)])
    m = api.LayeredModel(ctx, cfg, bits(t), compute, 256)
    toks = tokens(T, 52)
    f = {k: np.asarray(v, np.float64) for k, v in t.items()}
    x = f["embed"][toks]
    h = L.dyt_norm(x, f["l0.norm1.alpha"], f["l0.norm1"], f["l0.norm1.b"])
    q = L.rotate_interleaved((h @ f["l0.mix.q"].T).reshape(T, H, D), np.arange(T), 10, 300.0)
    k = L.rotate_interleaved((h @ f["l0.mix.k"].T).reshape(T, G, D), np.arange(T), 10, 300.0)
    v = (h @ f["l0.mix.v"].T).reshape(T, G, E)
    a = np.stack([L.window_softmax(q[:, n], k[:, 0], v[:, 0], 0.3, None) for n in range(H)], 1)
    x = x + L.dyt_norm(a.reshape(T, H * E) @ f["l0.mix.o"].T, f["l0.norm1b.alpha"], f["l0.norm1b"], f["l0.norm1b.b"])
    want = L.dyt_norm(x, f["final.norm.alpha"], f["final.norm"], f["final.norm.b"]) @ f["embed"].T
    s = Session(m)
    got = np.concatenate([s.run([("a", toks[:100])])[0]] + [s.run([("a", [c])])[0] for c in toks[100:]])
    assert distance(got, want).max() < LIMIT[compute]


@pytest.mark.parametrize("window", [300, 2000])
def test_long_context_decoding_splits_keys(ctx, window):
    """One sequence far along: its keys are cut over a cluster of CTAs; a block size that tiles straddle, and one they do not."""
    cfg = config([attention(heads=4, kv_heads=1, dim=32, vdim=64, window=window, ff=0)], width=64)
    t = tensors(cfg, 61)
    toks = tokens(901, 62)
    want = reference(cfg, t).forward(toks)
    m = device_model(ctx, cfg, t, "bfloat16")
    for bs in (16, 12, 64):
        s = Session(m, block_size=bs)
        s.run([("a", toks[:895])], False)
        for i in range(895, 901):
            assert distance(s.run([("a", [toks[i]])])[0], want[i:i + 1]).max() < LIMIT["bfloat16"]
