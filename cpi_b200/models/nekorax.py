"""Nekorax as a `ModelSpec`: every layer is a `sandwich_norm` block whose four norms (and the model's last) are
`dynamic_tanh`.  The mixer is `attention` with a short convolution over q, k and v, a rotation of pairs (i, i + dims / 2)
over part of each head, values that turn with their positions (`value_rotation`), a constant sink of score 0 and an
elementwise output gate; or `latent_attention` with a sliding window and an interleaved rotation under the yarn rule.  The
feed-forward is `moe_swiglu` with clamped experts, identity experts and a choice by softmax scores plus a correction among
the best groups.  A range of layers may run several times, every pass with its own cache and state, entered through a
matrix over [residual ; embedding output] and a vector of the pass (junctions `concat_linear`).

Tensor names: `embed`, `loop.in`, `loop.step`, `final.norm`, `head`; layer i under `l<i>.`: `norm1`, `norm1b`, `norm2`,
`norm2b` (a norm's `.alpha` and `.b` beside it), `mix.{q,k,v,q.conv,k.conv,v.conv,g,o}` or
`mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}`, `mlp.{router,correction,e<n>.{gate,up,down}}`.
"""
from __future__ import annotations

from ..config.nekorax import NekoraxConfig
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def _position(rot, head_dim, pairing) -> PartSpec:
    sc = rot["scaling"]
    scaling = None if sc is None else {
        "rope_type": "yarn", "factor": sc["factor"], "original_max_position_embeddings": sc["original"],
        "beta_fast": sc["fast"], "beta_slow": sc["slow"]}
    return PartSpec("rope", {"head_dim": head_dim, "theta": rot["base"], "pairing": pairing, "rotary_dims": rot["dims"],
                             "scaling": scaling, "frequency_math": "float64"})


def _mixer_spec(cfg: NekoraxConfig, layer) -> PartSpec:
    m, W = layer.mixer, cfg.width
    if layer.type == "attention":
        return PartSpec("attention", {
            "hidden_size": W, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "value_dim": m["vdim"], "softmax_scale": m["scale"], "position": _position(m["rot"], m["dim"], "half_split"),
            "qk_norm": False, "window": {"kind": "full", "size": 0}, "query_temperature": None, "conv": m["conv"],
            "value_rotation": {"theta": m["rot"]["base"]}, "sink": {"constant": 0.0}, "output_gate": "elementwise",
            "tensor_names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "q_conv": "mix.q.conv",
                             "k_conv": "mix.k.conv", "v_conv": "mix.v.conv", "g": "mix.g"}})
    window = {"kind": "full"} if m["mask"] is None else {"kind": "sliding", "size": m["mask"]["size"]}
    return PartSpec("latent_attention", {
        "hidden_size": W, "heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "value_dim": m["vdim"],
        "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "softmax_scale": m["scale"], "norm_eps": cfg.eps,
        "position": _position(m["rot"], m["rot_dim"], "interleaved"), "window": window,
        "tensor_names": {"dq": "mix.dq", "dq_norm": "mix.dq.norm", "uq": "mix.uq", "dkv": "mix.dkv",
                         "dkv_norm": "mix.dkv.norm", "uk": "mix.uk", "uv": "mix.uv", "o": "mix.o"}})


def _ff_spec(cfg: NekoraxConfig, mlp) -> PartSpec:
    return PartSpec("moe_swiglu", {
        "hidden_size": cfg.width, "num_experts": mlp["experts"], "identity_experts": mlp["identity"], "top_k": mlp["top"],
        "expert_size": mlp["ff"], "activation": "swish_clamped", "limit": mlp["limit"], "router_gate": "scored",
        "router_name": "mlp.router",
        "router_rule": {"score": "softmax", "choice_bias": "mlp.correction", "groups": mlp["groups"], "keep": mlp["keep"],
                        "group_score": "max", "normalise": False},
        "expert_layout": "per_expert",
        "expert_names": {"gate": "mlp.e{e}.gate", "up": "mlp.e{e}.up", "down": "mlp.e{e}.down"}})


def build_spec(cfg: NekoraxConfig) -> ModelSpec:
    W = cfg.width

    def norm(name) -> PartSpec:
        return PartSpec("dynamic_tanh", {"size": W, "weight": name, "alpha": name + ".alpha", "offset": name + ".b"})

    layers = []
    for i, L in enumerate(cfg.layers):
        has_ff = L.mlp is not None
        layers.append(LayerSpec(
            prefix=f"l{i}.", block=PartSpec("sandwich_norm", {}), mixer=_mixer_spec(cfg, L),
            feed_forward=_ff_spec(cfg, L.mlp) if has_ff else None, mixer_norm=norm("norm1"),
            feed_forward_norm=norm("norm2") if has_ff else None, mixer_post_norm=norm("norm1b"),
            feed_forward_post_norm=norm("norm2b") if has_ff else None))
    times = 0 if cfg.loop is None else cfg.loop[2]
    head = {"weight": "head", "vocab_size": cfg.vocab, "hidden_size": W}
    if cfg.logit_softcap is not None:
        head["logit_softcap"] = cfg.logit_softcap
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=W, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"weight": "embed", "vocab_size": cfg.vocab, "hidden_size": W,
                                               "scale": cfg.embedding_scale}),
        layers=tuple(layers),
        # every pass of a repeated layer owns its cache and state; a pass is entered through its junction
        run_order=tuple(RunEntry(i, before=None if t is None else f"pass{t}") for i, t in cfg.run_order()),
        final_norm=norm("final.norm"), head=PartSpec("linear_head", head), initializer_range=cfg.initializer_range,
        junctions=tuple((f"pass{t}", PartSpec("concat_linear", {
            "hidden_size": W, "weight": "loop.in", "step": "loop.step", "pass_index": t, "passes": times,
            "products": "single_cta"})) for t in range(times)),
        # norms that a folder stores around a feed-forward that a layer does not have are not read
        ignored_tensor_prefixes=tuple(f"l{i}.norm2" for i, L in enumerate(cfg.layers) if L.mlp is None))


register_architecture(Architecture("Nekorax", NekoraxConfig.from_json_dict, build_spec))
