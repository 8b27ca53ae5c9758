"""The Kuvidra configuration reader on the CPU: what it builds from config.json, and what it refuses."""
import copy

import pytest

from aien_sovereign_core_mv_b200 import ConfigError, model_spec_for
from aien_sovereign_core_mv_b200.models.decoder import Decoder

LATENT = {"heads": 3, "dim": 10, "vdim": 14, "kv_rank": 18, "q_rank": 22, "scale": 0.3}
CONFIG = {"architecture": "Kuvidra", "vocab": 91, "width": 40, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 3},
          "layers": [
              {"type": "latent_attention", "mixer": LATENT, "mlp": {"kind": "dense", "ff": 52}},
              {"type": "mlstm", "mixer": {"heads": 2, "dim": 6, "vdim": 9, "gate_cap": 7.0},
               "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 4, "top": 2}, "shared": {"ff": 26}}},
              {"type": "latent_attention", "mixer": dict(LATENT, heads=5), "mlp": None},
              {"type": "mlstm", "mixer": {"heads": 1, "dim": 8, "vdim": 4, "gate_cap": 20}, "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 3, "top": 1}}}]}


def test_spec_parts_run_list_and_tensor_names():
    cfg, spec = model_spec_for(CONFIG)
    assert cfg.num_hidden_layers == 4 and cfg.loop == (1, 3, 3) and cfg.norm_eps == 1e-5
    assert [l.block for l in spec.layers] == ["parallel"] * 4
    assert [l.mixer.kind for l in spec.layers] == ["latent_attention", "matrix_memory"] * 2
    # layers 1 and 2 run three times; every run has a cache of its own; the first run of every pass opens it, also the first
    assert [(r.layer, r.cache, r.enter) for r in spec.run_list] == [(0, 0, -1), (1, 1, 0), (2, 2, -1), (1, 3, 1), (2, 4, -1), (1, 5, 2), (2, 6, -1), (3, 7, -1)]
    assert all(r.writes_cache for r in spec.run_list) and spec.pass_input.kind == "step_projection" and spec.pass_input.params["times"] == 3
    p = spec.layers[0].mixer.params
    assert (p["rot_dim"], p["head_gate"], p["scale"], p["value_dim"], p["norm_eps"]) == (0, True, 0.3, 14, 1e-5)
    assert spec.layers[1].mixer.params["gate_cap"] == 7.0 and spec.layers[3].mixer.params["gate_cap"] == 20.0
    f = spec.layers[1].feed_forward.params
    assert (f["num_experts"], f["top"], f["act"], f["score"], f["weight_on_input"], f["shared_ff"], f["shared_gate"]) == (4, 2, "swiglu", "sigmoid", True, 26, True)
    assert (spec.layers[3].feed_forward.params["shared_ff"], spec.layers[3].feed_forward.params["shared_gate"]) == (0, False)
    assert spec.layers[0].feed_forward.params["act"] == "gelu" and spec.layers[2].feed_forward is None
    model = Decoder(spec)
    cat = {k: v[0] for k, v in model.catalog().items()}
    assert model.tied and "head" not in cat and cat["embed"] == (91, 40) and cat["final.norm"] == (40,)
    assert cat["loop.in"] == (40, 80) and cat["loop.step"] == (3, 40)
    assert cat["l0.mix.dq"] == (22, 40) and cat["l0.mix.dq.norm"] == (22,) and cat["l0.mix.uq"] == (30, 22) and cat["l0.mix.dkv"] == (18, 40)
    assert cat["l0.mix.dkv.norm"] == (18,) and cat["l0.mix.uk"] == (30, 18) and cat["l0.mix.uv"] == (42, 18) and cat["l0.mix.g"] == (3, 40)
    assert cat["l0.mix.o"] == (40, 42) and cat["l0.mlp.up"] == (52, 40) and cat["l0.mlp.down"] == (40, 52) and cat["l0.norm1"] == (40,)
    assert cat["l1.mix.q"] == (12, 40) and cat["l1.mix.v"] == (18, 40) and cat["l1.mix.g"] == (18, 40) and cat["l1.mix.i"] == (2, 40)
    assert cat["l1.mix.i.b"] == (2,) and cat["l1.mix.f"] == (2, 40) and cat["l1.mix.f.b"] == (2,) and cat["l1.mix.norm"] == (18,)
    assert cat["l1.mlp.router"] == (4, 40) and cat["l1.mlp.e3.gate"] == (12, 40) and cat["l1.mlp.e3.down"] == (40, 12) and "l1.mlp.e4.up" not in cat
    assert cat["l1.mlp.shared.sg"] == (1, 40) and cat["l1.mlp.shared.gate"] == (26, 40) and cat["l1.mlp.shared.down"] == (40, 26)
    assert not [k for k in cat if "norm2" in k or k.startswith("l2.mlp") or k.startswith("l3.mlp.shared")]
    # pages for the attention of four runs; state slots for the memories: three runs of layer 1, one of layer 3
    assert [s for n, s in zip(model.group_needs, model.group_slots) if n.kind == "full"] == [4]
    states = sorted((n.state_shape[0], s) for n, s in zip(model.group_needs, model.group_slots) if n.kind == "state")
    assert states == sorted([(2 * (54 + 6 + 1) + 2, 3), (32 + 8 + 1 + 3, 1)])        # S, n, m, filled up to whole groups of four


def test_without_a_loop_there_is_no_pass_input():
    c = copy.deepcopy(CONFIG)
    c["loop"] = None
    _, spec = model_spec_for(c)
    assert spec.pass_input is None and [r.enter for r in spec.run_list] == [-1] * 4
    assert not [k for k in Decoder(spec).catalog() if k.startswith("loop")]


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "conv", "mixers"),
    (("layers", 0, "mixer", "kv_rank"), 0, "kv_rank"),
    (("layers", 0, "mixer", "scale"), None, "scale"),
    (("layers", 0, "mixer", "rot_dim"), 8, "rotated"),
    (("layers", 1, "mixer", "gate_cap"), 0.0, "gate_cap"),
    (("layers", 1, "mlp", "router", "top"), 5, "top"),
    (("layers", 1, "mlp", "shared"), {"size": 3}, "ff"),
    (("layers", 0, "mlp", "kind"), "glu", "feed-forwards"),
    (("loop", "stop"), 5, "loop"),
    (("loop", "times"), 0, "times"),
    (("norm", "eps"), None, "eps"),
    (("layers",), [], "layers"),
])
def test_refusals(path, value, word):
    c = copy.deepcopy(CONFIG)
    at = c
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        model_spec_for(c)
    assert word in str(e.value)
