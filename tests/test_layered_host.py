"""Configuration, registry and checkpoint reading of the layered designs (host code, no GPU)."""
import json

import numpy as np
import pytest

from layered_helpers import attention, bits, config, gla, mlstm, tensors, write_checkpoint
from paged_infer_b200 import loader, registry


def test_config_fields_reach_the_layers():
    c = loader.LayeredConfig.from_sumosun(config([attention(heads=6, kv_heads=3, dim=10, vdim=14, window=9, rot=4, base=77.0, diff=0.25, scale=0.5, ff=21),
                                                  gla(heads=2, dim=5, vdim=7, tau=3.0), mlstm(heads=4, dim=6, vdim=8, cap=2.5, ff=11)],
                                                 width=30, vocab=50, eps=1e-4))
    a, g, x = c.layers
    assert (c.width, c.vocab_size, c.norm_eps, c.has_state) == (30, 50, 1e-4, True)
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.maps, a.window, a.rot_dims, a.rot_base, a.scale, a.diff, a.ff) == \
        (loader.MIXER_ATTENTION, 6, 3, 10, 14, 2, 9, 4, 77.0, 0.5, 0.25, 21)
    assert (g.mixer, g.heads, g.dim, g.vdim, g.tau, g.ff) == (loader.MIXER_GLA, 2, 5, 7, 3.0, 0)
    assert (x.mixer, x.heads, x.dim, x.vdim, x.gate_cap, x.ff) == (loader.MIXER_MLSTM, 4, 6, 8, 2.5, 11)
    assert not loader.LayeredConfig.from_sumosun(config([attention()])).has_state


def test_unknown_parts_are_refused():
    bad = config([attention()])
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        loader.LayeredConfig.from_sumosun(bad)
    bad = config([attention()])
    bad["layers"][0]["mlp"]["kind"] = "routed"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        loader.LayeredConfig.from_sumosun(bad)


def test_registry_names():
    assert registry.family_of({"architecture": "Sumosun"}) == "Sumosun"
    assert registry.family_of({"architectures": ["LlamaForCausalLM"]}) == "Llama"
    assert registry.family_of({"hidden_size": 64}) == "Llama"
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.family_of({"architecture": "Elsewhere"})
    with pytest.raises(registry.UnsupportedDtype):
        registry.load(None, _folder({"hidden_size": 64}), "bfloat16")


def _folder(cfg):
    import pathlib
    import tempfile
    d = pathlib.Path(tempfile.mkdtemp())
    (d / "config.json").write_text(json.dumps(cfg))
    return str(d)


def test_checkpoint_round_trip(tmp_path):
    cfg = config([attention(), gla(), mlstm()])
    t = tensors(cfg, 1)
    folder = write_checkpoint(tmp_path, cfg, t)
    assert registry.family_of(registry.read_config(folder)) == "Sumosun"
    got = loader.read_safetensors(folder + "/model.safetensors")
    assert set(got) == set(t) and got["l0.norm1.alpha"].shape == ()
    for k, v in bits(t).items():
        assert np.array_equal(got[k], v)


def test_safetensors_with_integer_and_f32_tables(tmp_path):
    import struct
    a, b = np.arange(3, dtype="<i4"), np.array([[1.5]], "<f4")
    h = json.dumps({"x": {"dtype": "I32", "shape": [3], "data_offsets": [0, 12]}, "y": {"dtype": "F32", "shape": [1, 1], "data_offsets": [12, 16]}}).encode()
    p = tmp_path / "t.safetensors"
    p.write_bytes(struct.pack("<Q", len(h)) + h + a.tobytes() + b.tobytes())
    got = loader.read_safetensors(str(p))
    assert np.array_equal(got["x"], a) and np.array_equal(got["y"], b)
