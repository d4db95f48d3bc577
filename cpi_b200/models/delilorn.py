"""Delilorn as a `ModelSpec`: every layer is a `sandwich_norm` block whose four norms (and the model's last) are RMS norms
with weights stored around zero.  The mixer is `lightning` (linear attention, a constant decay per head); or
`latent_attention` with a sink, an elementwise output gate and a half-split rotation, some of whose layers have no latent
of their own and read an earlier run entry's cache; or `attention` with a rotation of part of each head (the llama3
frequency rule) under a sliding window that keeps the sequence's first tokens.  The feed-forward is `moe_mlp`: experts of
two matrices with a squared relu, weighted by their softmax scores as they are.  The head is the embedding table.

Tensor names: `embed`, `final.norm`; layer i under `l<i>.`: `norm1`, `norm1b`, `norm2`, `norm2b`,
`mix.{q,k,v,g,o,norm}`, `mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,g,o}` or `mix.{q,k,v,o}`,
`mlp.{router,e<n>.{up,down}}`.
"""
from __future__ import annotations

from ..config.delilorn import DelilornConfig
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def _position(rot, head_dim) -> PartSpec:
    if rot is None:
        return PartSpec("none", {})
    sc = rot["scaling"]
    scaling = None if sc is None else {
        "rope_type": "llama3", "factor": sc["factor"], "low_freq_factor": sc["low"], "high_freq_factor": sc["high"],
        "original_max_position_embeddings": sc["original"]}
    return PartSpec("rope", {"head_dim": head_dim, "theta": rot["base"], "pairing": "half_split",
                             "rotary_dims": rot["dims"], "scaling": scaling, "frequency_math": "float64"})


def _mixer_spec(cfg: DelilornConfig, layer) -> PartSpec:
    m, W = layer.mixer, cfg.width
    if layer.type == "lightning":
        return PartSpec("lightning", {
            "hidden_size": W, "heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"], "decay": m["decay"],
            "norm_eps": cfg.eps,
            "tensor_names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "g": "mix.g", "o": "mix.o", "norm": "mix.norm"}})
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", {
            "hidden_size": W, "heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "value_dim": m["vdim"],
            "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "softmax_scale": m["scale"], "norm_eps": cfg.eps,
            "position": _position(m["rot"], m["rot_dim"]), "sink": True, "output_gate": True,
            "tensor_names": {"dq": "mix.dq", "dq_norm": "mix.dq.norm", "uq": "mix.uq", "dkv": "mix.dkv",
                             "dkv_norm": "mix.dkv.norm", "uk": "mix.uk", "uv": "mix.uv", "o": "mix.o", "sink": "mix.sink",
                             "g": "mix.g"}})
    window = {"kind": "full", "size": 0} if m["mask"] is None else {"kind": "sliding", **m["mask"]}
    return PartSpec("attention", {
        "hidden_size": W, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
        "value_dim": m["vdim"], "softmax_scale": m["scale"], "position": _position(m["rot"], m["dim"]), "qk_norm": False,
        "window": window, "query_temperature": None,
        "tensor_names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o"}})


def _ff_spec(cfg: DelilornConfig, mlp) -> PartSpec:
    return PartSpec("moe_mlp", {
        "hidden_size": cfg.width, "num_experts": mlp["experts"], "top_k": mlp["top"], "expert_size": mlp["ff"],
        "activation": "relu_squared", "router_gate": "scored", "router_name": "mlp.router",
        "router_rule": {"score": "softmax", "normalise": False}, "expert_layout": "per_expert",
        "expert_names": {"up": "mlp.e{e}.up", "down": "mlp.e{e}.down"}})


def build_spec(cfg: DelilornConfig) -> ModelSpec:
    W = cfg.width

    def norm(name) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": cfg.eps, "weight": name, "weight_offset": 1.0})

    layers = []
    for i, L in enumerate(cfg.layers):
        has_ff = L.mlp is not None
        layers.append(LayerSpec(
            prefix=f"l{i}.", block=PartSpec("sandwich_norm", {}), mixer=_mixer_spec(cfg, L),
            feed_forward=_ff_spec(cfg, L.mlp) if has_ff else None, mixer_norm=norm("norm1"),
            feed_forward_norm=norm("norm2") if has_ff else None, mixer_post_norm=norm("norm1b"),
            feed_forward_post_norm=norm("norm2b") if has_ff else None))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=W, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"weight": "embed", "vocab_size": cfg.vocab, "hidden_size": W}),
        layers=tuple(layers),
        # every layer runs once, so the run entry that a layer reads has the number of its layer
        run_order=tuple(RunEntry(i, cache_of=L.mixer.get("kv_from")) for i, L in enumerate(cfg.layers)),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"weight": "embed", "vocab_size": cfg.vocab, "hidden_size": W}),
        initializer_range=cfg.initializer_range,
        # norms that a folder stores around a feed-forward that a layer does not have are not read
        ignored_tensor_prefixes=tuple(f"l{i}.norm2" for i, L in enumerate(cfg.layers) if L.mlp is None))


register_architecture(Architecture("Delilorn", DelilornConfig.from_json_dict, build_spec))
