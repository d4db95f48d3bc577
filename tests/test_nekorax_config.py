"""Nekorax configuration and spec on the CPU: keys, defaults, errors that name the key, the tensor list, the plain
implementation's own consistency."""
from __future__ import annotations

import copy

import pytest
import torch

import nekorax_tiny as V
import plain_nekorax as P
from cpi_b200.config.common import ConfigError
from cpi_b200.config.nekorax import NekoraxConfig
from cpi_b200.config.registry import architecture_of
from cpi_b200.config.spec import PartSpec
from cpi_b200.engine.model import tensor_requirements
from cpi_b200.parts.base import build_part

F64 = torch.float64


@pytest.mark.parametrize("cfg", [V.MIXED_A, V.MIXED_B, V.MIXED_C] + [V.draw_config(s) for s in range(1, 13)])
def test_the_tensor_list_is_the_drawn_weights(cfg):
    arch = architecture_of(cfg)
    assert arch.name == "Nekorax"
    spec = arch.build_spec(arch.parse_config(cfg))
    spec.validate()
    need = {r.name: tuple(r.shape) for r in tensor_requirements(spec)}
    have = {k: tuple(v.shape) for k, v in V.draw_weights(cfg, 1).items()}
    assert need == have


def test_defaults_and_parts():
    cfg = NekoraxConfig.from_json_dict(V.MIXED_C)
    spec = architecture_of(V.MIXED_C).build_spec(cfg)
    assert cfg.logit_softcap is None and cfg.loop is None and cfg.embedding_scale == 1.0 and spec.junctions == ()
    assert [l.block.kind for l in spec.layers] == ["sandwich_norm"] * 5
    assert spec.layers[0].mixer["conv"] is None and spec.layers[0].mixer["output_gate"] == "elementwise"
    assert spec.layers[1].mixer["window"] == {"kind": "sliding", "size": 1} and spec.layers[3].mixer["window"] == {"kind": "full"}
    assert spec.layers[2].feed_forward is None and spec.layers[2].feed_forward_post_norm is None
    ff = spec.layers[4].feed_forward
    assert ff["num_experts"] == 4 and ff["identity_experts"] == 4 and ff["router_rule"]["groups"] == 8
    assert spec.layers[3].feed_forward["router_rule"]["groups"] == 1
    a = architecture_of(V.MIXED_A).build_spec(NekoraxConfig.from_json_dict(V.MIXED_A))
    assert [e.layer for e in a.run_order] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [e.before for e in a.run_order] == [None, "pass0", None, "pass1", None, "pass2", None, None]
    assert dict(a.junctions)["pass2"]["pass_index"] == 2 and a.embedding["scale"] == 0.7
    rope = a.layers[0].mixer["position"]
    assert rope["pairing"] == "interleaved" and rope["scaling"]["rope_type"] == "yarn"
    assert a.layers[1].mixer["position"]["pairing"] == "half_split" and a.layers[1].mixer["value_rotation"] == {"theta": 300.0}


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["layers"][0].update(type="other"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=7), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(mask={"size": 4}), "mask"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=2), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=2), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].pop("start"), "start"),
    (lambda c: c.update(logit_softcap=0.0), "logit_softcap"),
    (lambda c: c.update(embedding=2.0), "embedding"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_errors_name_the_key(change, word):
    cfg = copy.deepcopy(V.MIXED_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        NekoraxConfig.from_json_dict(cfg)
    assert word in str(e.value)


@pytest.mark.parametrize("family,kind,params", [
    ("mixer", "attention", {"value_dim": 7}), ("mixer", "attention", {"output_gate": "half"}),
    ("mixer", "attention", {"differential": {"lambda_init": 0.3}}), ("mixer", "attention", {"value_mix": {"role": "first"}}),
    ("feed_forward", "moe_swiglu", {"activation": "swish_clamped"}), ("feed_forward", "moe_swiglu", {"router_gate": "sigmoid_input"}),
    ("feed_forward", "moe_swiglu", {"router_rule": {"score": "tanh"}}), ("feed_forward", "moe_swiglu", {"router_rule": {"groups": 5, "keep": 1}}),
])
def test_parts_refuse_what_they_cannot_do(family, kind, params):
    base = {"attention": {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "value_dim": 8, "softmax_scale": 1.0,
                          "position": PartSpec("none", {}), "value_rotation": {"theta": 10.0}, "output_gate": "elementwise"},
            "moe_swiglu": {"hidden_size": 16, "num_experts": 4, "identity_experts": 2, "top_k": 2, "expert_size": 8,
                           "activation": "silu", "router_gate": "scored"}}[kind]
    build_part(family, PartSpec(kind, base))
    with pytest.raises(ValueError):
        build_part(family, PartSpec(kind, {**base, **params}))


def test_plain_implementation_is_causal_and_its_mechanisms_do_what_they_say():
    """A prefix's logits do not depend on what follows; values turned by their positions and turned back reach a query
    turned by the distance alone; the sink takes its share; an expert without tensors returns its input."""
    cfg = V.MIXED_A
    W = V.draw_weights(cfg, 3)
    toks = V.tokens(40, cfg["vocab"], 1)
    whole = P.forward(cfg, W, toks)
    assert (P.forward(cfg, W, toks[:23]) - whole[:23]).abs().max() < 1e-9
    f, _ = P.frequencies(6, 30.0)
    v = torch.randn(9, 1, 6, dtype=F64)
    pos = torch.arange(9)
    out = P.turn(P.turn(v, pos, f)[3:4].expand(9, 1, 6), pos, f, sign=-1.0)      # position 3's value as every query gets it
    assert (out[7, 0] - P.turn(v[3:4], torch.tensor([-4]), f)[0, 0]).abs().max() < 1e-12
    q = k = torch.zeros(1, 1, 2, dtype=F64)
    one = torch.ones(1, 1, 3, dtype=F64)
    assert abs(float(P.weighted_values(q, k, one, 1.0, P.visible(1), True)[0, 0, 0]) - 0.5) < 1e-12
    r = {"experts": 1, "identity": 3, "top": 2, "groups": {"count": 2, "keep": 1}}
    mlp = {"expert": {"ff": 2, "limit": 1.0}, "router": r}
    Wf = {"router": torch.zeros(4, 5), "correction": torch.tensor([-5.0, -5.0, -1.0, -2.0]), "e0.gate": torch.ones(2, 5),
          "e0.up": torch.ones(2, 5), "e0.down": torch.ones(5, 2)}
    h = torch.randn(3, 5, dtype=F64)
    assert (P.routed_ff(h, Wf, "", mlp) - 0.5 * h).abs().max() < 1e-9               # both chosen are the identity: 1/4 + 1/4
    assert [i for i, t in P.run_order(V.MIXED_B)] == [0, 1, 0, 1, 2, 3]
