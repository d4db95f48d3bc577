"""Delilorn configuration and spec on the CPU: keys, defaults, errors that name the key, the tensor list, the cache that
layers share, the plain implementation's own consistency."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import delilorn_tiny as V
import plain_delilorn as P
from cpi_b200.config.common import ConfigError
from cpi_b200.config.delilorn import DelilornConfig
from cpi_b200.config.registry import architecture_of
from cpi_b200.config.spec import PartSpec
from cpi_b200.engine.model import DecoderModel, tensor_requirements
from cpi_b200.parts.base import build_part
from cpi_b200.parts.positions import llama3_frequencies_f64

F64 = torch.float64


@pytest.mark.parametrize("cfg", [V.MIXED_A, V.MIXED_B, V.MIXED_C] + [V.draw_config(s) for s in range(1, 13)])
def test_the_tensor_list_is_the_drawn_weights(cfg):
    arch = architecture_of(cfg)
    assert arch.name == "Delilorn"
    spec = arch.build_spec(arch.parse_config(cfg))
    spec.validate()
    need = {r.name: tuple(r.shape) for r in tensor_requirements(spec)}
    have = {k: tuple(v.shape) for k, v in V.draw_weights(cfg, 1).items()}
    assert need == have


def test_defaults_and_parts():
    cfg = DelilornConfig.from_json_dict(V.MIXED_C)
    spec = architecture_of(V.MIXED_C).build_spec(cfg)
    assert all(l.block.kind == "sandwich_norm" and l.mixer_post_norm["weight_offset"] == 1.0 for l in spec.layers)
    assert spec.head["weight"] == spec.embedding["weight"] == "embed"
    assert spec.layers[1].mixer["window"]["kind"] == "full" and spec.layers[1].mixer["position"].kind == "none"
    assert spec.layers[3].mixer["window"] == {"kind": "sliding", "size": 1, "keep_first": 0}
    assert spec.layers[3].feed_forward is None and spec.layers[3].feed_forward_post_norm is None
    assert spec.layers[0].mixer["decay"] == (1.0,) and spec.layers[0].feed_forward.kind == "moe_mlp"
    a = architecture_of(V.MIXED_A).build_spec(DelilornConfig.from_json_dict(V.MIXED_A))
    assert [e.cache_of for e in a.run_order] == [None, 0, None, None, 0, None]
    assert a.layers[3].mixer["window"] == {"kind": "sliding", "size": 19, "keep_first": 3}
    assert a.layers[3].mixer["position"]["scaling"]["rope_type"] == "llama3"
    assert a.layers[0].mixer["output_gate"] and a.layers[0].mixer["sink"]


def test_layers_that_read_another_s_latent_keep_nothing():
    """Cache and state belong to the layers that write them; a reading layer has neither pages nor a latent's matrices."""
    m = DecoderModel(architecture_of(V.MIXED_B).build_spec(DelilornConfig.from_json_dict(V.MIXED_B)), torch.float32, "cpu")
    kv, state = m.cache_requirements()
    assert sorted(kv) == [0, 1, 4, 6] and sorted(state) == [2, 7]
    assert kv[1].streams == (("latent", 1, 112),) and kv[0].keep_first == 4 and kv[6].keep_first == 65
    assert state[7][0].shape == (2, 64, 128) and state[7][0].dtype == torch.float32
    names = {r.name for r in m.layers[3].mixer.requirements()}
    assert "l3.mix.dkv" not in names and "l3.mix.g" in names


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["layers"][0].update(type="other"), "type"),
    (lambda c: c["layers"][3]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(dims=12), "dims"),
    (lambda c: c["layers"][3]["mixer"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][3]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][3]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][3]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=2), "dims"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=4), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=True), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_rank=12), "kv_rank"),
    (lambda c: c["layers"][4]["mixer"]["rot"].update(base=301.0), "rot"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 0.6]), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 0.6, 1.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(heads=2), "decay"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_errors_name_the_key(change, word):
    cfg = copy.deepcopy(V.MIXED_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        DelilornConfig.from_json_dict(cfg)
    assert word in str(e.value)


@pytest.mark.parametrize("kind,params", [
    ("lightning", {"decay": (0.5,)}), ("lightning", {"decay": (0.5, 1.1)}), ("lightning", {"key_dim": 2000}),
    ("moe_mlp", {"activation": "silu"}), ("moe_mlp", {"expert_layout": "stacked"}), ("moe_mlp", {"top_k": 9}),
    ("moe_mlp", {"expert_names": {"gate": "g{e}", "up": "u{e}", "down": "d{e}"}}),
])
def test_parts_refuse_what_they_cannot_do(kind, params):
    family, base = {
        "lightning": ("mixer", {"hidden_size": 16, "heads": 2, "key_dim": 8, "value_dim": 4, "decay": (0.5, 1.0), "norm_eps": 1e-5}),
        "moe_mlp": ("feed_forward", {"hidden_size": 16, "num_experts": 4, "top_k": 2, "expert_size": 8, "router_gate": "scored",
                                     "expert_layout": "per_expert", "expert_names": {"up": "u{e}", "down": "d{e}"}})}[kind]
    build_part(family, PartSpec(kind, base))
    with pytest.raises(ValueError):
        build_part(family, PartSpec(kind, {**base, **params}))


def test_the_two_statements_of_the_frequency_rule_agree():
    for sc in (None, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}, {"factor": 8.0, "low": 0.5, "high": 2.0, "original": 1000}):
        lib = None if sc is None else {"factor": sc["factor"], "low_freq_factor": sc["low"], "high_freq_factor": sc["high"],
                                       "original_max_position_embeddings": sc["original"]}
        got, want = llama3_frequencies_f64(48, 700.0, lib), P.frequencies(48, 700.0, sc)
        assert (torch.from_numpy(got).double() / want - 1.0).abs().max() < 1e-6
        if sc:                          # all three cases occur
            ratio = (want / P.frequencies(48, 700.0)).tolist()
            assert any(r == 1.0 for r in ratio) and any(abs(r * sc["factor"] - 1.0) < 1e-12 for r in ratio)
            assert any(1.001 / sc["factor"] < r < 0.999 for r in ratio)


def test_plain_implementation_is_causal_and_its_mechanisms_do_what_they_say():
    cfg = V.MIXED_A
    W = V.draw_weights(cfg, 3)
    toks = V.tokens(40, cfg["vocab"], 1)
    whole = P.forward(cfg, W, toks)
    assert (P.forward(cfg, W, toks[:23]) - whole[:23]).abs().max() < 1e-9
    ok = P.visible(9, 3, 2)
    assert ok[7].nonzero().flatten().tolist() == [0, 1, 5, 6, 7] and ok[1].nonzero().flatten().tolist() == [0, 1]
    q = k = torch.zeros(1, 1, 2, dtype=F64)
    one = torch.ones(1, 1, 3, dtype=F64)
    got = float(P.weighted_values(q, k, one, 1.0, P.visible(1), torch.tensor([math.log(3.0)]))[0, 0, 0])
    assert abs(got - 0.25) < 1e-6                                                    # 1 / (1 + 3)
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(6, 2, n, generator=g, dtype=F64) for n in (3, 3, 5))
    a = torch.tensor([0.7, 0.2], dtype=F64)
    o, S = P.decayed_sum(q, k, v, a)
    for t in range(6):
        for h in range(2):
            want = sum(a[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert (o[t, h] - want).abs().max() < 1e-12
    first, mid = P.decayed_sum(q[:4], k[:4], v[:4], a)
    assert (P.decayed_sum(q[4:], k[4:], v[4:], a, mid)[1] - S).abs().max() < 1e-12
