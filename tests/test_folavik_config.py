"""The Folavik configuration reader on the CPU: what it builds from config.json, what it refuses, and the two frequency
scalings against the plain implementation."""
import copy
import math

import numpy as np
import pytest

import plain_folavik as pf
from aien_sovereign_core_mv_b200 import ConfigError, model_spec_for
from aien_sovereign_core_mv_b200.models.decoder import Decoder
from aien_sovereign_core_mv_b200.parts.rotary import inverse_frequencies, yarn_frequencies

DIFF = {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 14, "scale": 0.3, "softcap": 7.0, "diff": 0.35, "mask": {"size": 21},
        "rot": {"base": 900.0, "dims": 6, "scaling": {"factor": 3.0, "original": 64, "fast": 5.0, "slow": 0.5}}}
CHUNK = {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 18, "scale": 0.2, "mask": {"size": 33},
         "rot": {"base": 7000.0, "dims": 8, "scaling": {"factor": 5.0, "low": 2.0, "high": 6.0, "original": 100}}}
LATENT = {"heads": 3, "dim": 9, "vdim": 11, "kv_rank": 26, "scale": 0.4}
CONFIG = {"architecture": "Folavik", "vocab": 77, "width": 42, "norm": {"eps": 2e-5}, "logit_scale": 0.6, "logit_softcap": 9.0, "layers": [
    {"type": "latent_attention", "mixer": LATENT, "mlp": {"kind": "dense", "ff": 50}},
    {"type": "attention_2", "mixer": DIFF, "mlp": None},
    {"type": "attention", "mixer": CHUNK, "mlp": {"kind": "dense", "ff": 34}},
    {"type": "attention_2", "mixer": dict(DIFF, heads=2, kv_heads=2, mask={"size": 5}), "mlp": {"kind": "dense", "ff": 22}}]}


def test_spec_parts_and_tensor_names():
    cfg, spec = model_spec_for(CONFIG)
    assert cfg.num_hidden_layers == 4 and (cfg.norm_eps, cfg.logit_scale, cfg.logit_softcap) == (2e-5, 0.6, 9.0)
    assert [l.block for l in spec.layers] == ["prenorm", "prenorm_mixer", "prenorm", "prenorm"]
    assert [l.mixer.kind for l in spec.layers] == ["latent_attention", "differential_attention", "value_attention", "differential_attention"]
    assert all(l.norm.kind == "layernorm" and l.norm.params["eps"] == 2e-5 for l in spec.layers) and spec.final_norm.kind == "layernorm"
    assert spec.embedding.kind == "table_normed" and spec.embedding.params["norm"]["kind"] == "layernorm"
    assert (spec.head.params["scale"], spec.head.params["softcap"], spec.head.params["tied"]) == (0.6, 9.0, False)
    assert spec.layers[0].feed_forward.params["act"] == "gelu_tanh" and spec.layers[1].feed_forward is None
    p = spec.layers[1].mixer.params
    assert (p["window"], p["softcap"], p["diff"], p["bias"], p["norm_eps"], p["value_dim"]) == (21, 7.0, 0.35, True, 2e-5, 14) and "chunk" not in p
    assert spec.layers[1].position.params["yarn"] == {"factor": 3.0, "original": 64.0, "fast": 5.0, "slow": 0.5}
    p = spec.layers[2].mixer.params
    assert (p["chunk"], p["scale"], p["value_dim"]) == (33, 0.2, 18) and "window" not in p and "bias" not in p
    assert spec.layers[2].position.params["rotary_dim"] == 8 and "yarn" not in spec.layers[2].position.params
    p = spec.layers[0].mixer.params
    assert (p["q_rank"], p["rot_dim"], p["out_gate"], p["kv_rank"], p["norm_eps"]) == (0, 0, True, 26, 2e-5)
    model = Decoder(spec)
    cat = {k: v[0] for k, v in model.catalog().items()}
    assert not model.tied and cat["head"] == (77, 42) and cat["embed"] == (77, 42) and cat["embed.norm"] == (42,) and cat["final.norm"] == (42,)
    assert cat["l0.mix.q"] == (27, 42) and cat["l0.mix.dkv"] == (26, 42) and cat["l0.mix.dkv.norm"] == (26,) and cat["l0.mix.uk"] == (27, 26)
    assert cat["l0.mix.uv"] == (33, 26) and cat["l0.mix.g"] == (33, 42) and cat["l0.mix.o"] == (42, 33) and cat["l0.mlp.gate"] == (50, 42)
    assert cat["l1.mix.q"] == (120, 42) and cat["l1.mix.q.b"] == (120,) and cat["l1.mix.k"] == (60, 42) and cat["l1.mix.k.b"] == (60,)
    assert cat["l1.mix.v"] == (42, 42) and cat["l1.mix.v.b"] == (42,) and cat["l1.mix.o"] == (42, 84) and cat["l1.mix.lq1"] == (10,)
    assert {f"l1.mix.{n}" for n in ("lq1", "lk1", "lq2", "lk2")} <= set(cat) and "l1.norm2" not in cat and "l1.mlp.up" not in cat
    assert cat["l2.mix.q"] == (48, 42) and cat["l2.mix.k"] == (24, 42) and cat["l2.mix.v"] == (36, 42) and cat["l2.mix.o"] == (42, 72)
    assert not [k for k in cat if k.startswith("l2.") and k.endswith(".b")] and cat["l3.norm2"] == (42,) and cat["l2.mlp.down"] == (42, 34)
    assert [(n.kind, n.window, dict(n.planes)) for n in model.group_needs] == [
        ("full", 0, {"latent": (26,)}), ("window", 21, {"k": (6, 10), "v": (3, 14)}), ("chunk", 33, {"k": (2, 12), "v": (2, 18)}),
        ("window", 5, {"k": (4, 10), "v": (2, 14)})]


def test_key_value_heads_and_value_sizes_default():
    c = copy.deepcopy(CONFIG)
    del c["layers"][2]["mixer"]["kv_heads"], c["layers"][2]["mixer"]["vdim"]
    p = model_spec_for(c)[1].layers[2].mixer.params
    assert (p["num_kv_heads"], p["value_dim"]) == (4, 12)


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "mamba", "type"), (("layers", 1, "mixer", "kv_heads"), 4, "multiple"), (("layers", 1, "mixer", "rot", "dims"), 5, "even"),
    (("layers", 2, "mixer", "rot", "dims"), 14, "dims"), (("layers", 2, "mixer", "scale"), None, "scale"), (("layers", 1, "mixer", "diff"), None, "diff"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), 0, "factor"), (("layers", 2, "mixer", "rot", "scaling", "low"), None, "low"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"), (("layers", 0, "mlp", "ff"), 0, "ff"), (("norm", "eps"), None, "eps"), (("width",), -3, "width"),
    (("layers", 0, "mixer", "kv_rank"), "x", "kv_rank"), (("layers",), [], "layers"), (("logit_scale",), "big", "logit_scale")])
def test_refusals_name_the_key(path, value, word):
    c = copy.deepcopy(CONFIG)
    o = c
    for k in path[:-1]:
        o = o[k]
    o[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        Decoder(model_spec_for(c)[1])
    assert word in str(e.value)


@pytest.mark.parametrize("base,dims,factor,original,fast,slow", [
    (10000.0, 64, 4.0, 2048, 32.0, 1.0), (500.0, 10, 2.5, 100, 8.0, 2.0), (1e6, 128, 40.0, 4096, 32.0, 1.0),
    (100.0, 4, 8.0, 16, 300.0, 0.001),                      # both ends clamped
    (10000.0, 32, 3.0, 512, 4.0, 4.0)])                     # both ends name the same turns
def test_yarn_frequencies(base, dims, factor, original, fast, slow):
    want, mult = pf.yarn_frequencies({"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}})
    got, m = yarn_frequencies(dims, base, factor, original, fast, slow)
    assert m == pytest.approx(mult, rel=1e-14) and m == pytest.approx(1.0 + math.log(factor) / 10.0)
    np.testing.assert_allclose(got, want, rtol=1e-13)


@pytest.mark.parametrize("base,dims,factor,low,high,original", [(10000.0, 64, 8.0, 1.0, 4.0, 8192), (500.0, 12, 3.0, 0.5, 2.0, 50), (1e6, 128, 16.0, 2.0, 3.0, 1000)])
def test_smoothed_frequencies(base, dims, factor, low, high, original):
    rot = {"base": base, "dims": dims, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}
    want, plain = pf.smoothed_frequencies(rot), pf.frequencies(rot)
    got = inverse_frequencies(dims, base, {"factor": factor, "low_freq_factor": low, "high_freq_factor": high, "original_max_position_embeddings": original},
                              dims, False)
    np.testing.assert_allclose(got, want, rtol=1e-13)
    ratio = plain / want
    assert ratio.min() == pytest.approx(1.0) and ratio.max() == pytest.approx(factor) and ((ratio > 1.001) & (ratio < factor * 0.999)).any()
