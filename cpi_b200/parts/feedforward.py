"""Feed-forward parts: a dense SwiGLU MLP, and routed experts with a shared expert.

Reference (src/engine/llama4_cpu_engine.cpp:252-291): router logits, the best expert, its
gate_up [H, 2I] and down [I, H] matrices applied as x @ W with a = silu(gate) * up, plus a shared
expert with ordinary [out, in] matrices, both added to the residual.  The reference takes one expert
and no gate value; top-k and the sigmoid gate (on the expert's input or output) are parameters here.

dense_swiglu  params: hidden_size, intermediate_size, activation ("silu" by default, or "gelu_tanh": the gate's
              activation; down(act(gate h) * (up h)); or "swish_clamped" with `limit`: g = min(gate h, limit),
              u = clamp(up h, -limit, limit), down(g sigmoid(1.702 g) (u + 1))), tensor_names (gate, up, down under
              the prefix), token_gate (a tensor name [1, H] or None: the output of a token is multiplied by
              sigmoid(token_gate . h))
              tensors: feed_forward.{gate,up,down}_proj.weight
moe_swiglu    params: hidden_size, num_experts, top_k, expert_size, shared_size (0 = no shared expert),
              router_gate ("sigmoid_input" | "sigmoid_output" | "none" | "softmax_chosen": the chosen experts'
              outputs weighted by the softmax over their logits | "sigmoid_normed": with s = sigmoid(logits) the choice is
              made on s + choice bias (`router_rule` {"choice_bias": a tensor name [E] or None, "groups": n, "keep": m,
              "scale": c}; only experts of the m best of n equal groups of neighbours can be chosen, a group's score
              being the sum of its two largest choice scores), and the chosen experts' outputs are weighted by their s
              divided by the chosen s' sum, times c | "scored": the same with the choices in `router_rule`: "score"
              ("sigmoid", or "softmax" over all of a token's logits), "group_score" ("top2_sum" or "max"), "normalise" (the
              division by the chosen scores' sum)), router_bias (a tensor name [E] added to the logits,
              or None), expert_layout ("stacked", below, or "per_expert": `expert_names` {"gate", "up", "down"} with
              "{e}" for the expert's number, each [out, in]), router_name, shared (None or the params of a
              dense_swiglu part that runs for every token beside the routed experts, instead of shared_size),
              activation ("silu", "gelu_tanh" or "swish_clamped" with `limit`, as above), identity_experts (n: the router
              knows n more experts, after the others, whose output is the input h itself; they have no tensors)
              tensors: feed_forward.router.weight [E, H], feed_forward.experts.gate_up_proj [E, H, 2I],
              feed_forward.experts.down_proj [E, I, H], feed_forward.shared_expert.{gate,up,down}_proj.weight

moe_mlp       the same with experts that have no gate: down(act(up h)), activation "relu_squared" or "gelu_tanh" as in
              dense_mlp; expert_names {"up", "down"} in the "per_expert" layout (the only one).  Identity experts, the
              router's gates and rules, and a shared expert are those of moe_swiglu.

dense_mlp     params: hidden_size, intermediate_size, activation ("relu_squared": max(z, 0)^2, or "gelu_tanh"), tensor_names (up, down):
              down(act(up h)), no gate.  The activation acts on the float32 accumulator of the first product, so its
              input is rounded once, after it.
              tensors: feed_forward.{up,down}_proj.weight

On load gate and up are stacked into one [2I, H] matrix, and the expert matrices are transposed to
[E, 2I, H] and [E, H, I], so that every contraction reads its weights along the reduction axis.
"""
from __future__ import annotations

import torch

from ..csrc import lib as K
from ..phases import active as phases_active, phase
from ..weights.store import TensorReq
from .base import ExpertSum, FeedForward, register_feed_forward
from .linear import (MODE_ADD, MODE_CLAMPED_GLU, MODE_GEGLU, MODE_STORE, MODE_STORE_GELU, MODE_STORE_RELU2, MODE_SWIGLU,
                     project)


def _stack(a, b):
    dt = torch.float32 if (a.dtype == torch.float32 or b.dtype == torch.float32) else torch.bfloat16
    return torch.cat([a.to(dt), b.to(dt)], dim=0).contiguous()


def _turned(t):
    """[E, in, out] as stored -> [E, out, in], contiguous (the library's transposing kernel on a GPU)."""
    if t.is_cuda and t.element_size() in (2, 4):
        return K.transpose_last2(t.contiguous())
    return t.transpose(1, 2).contiguous()


@register_feed_forward("dense_swiglu")
class DenseSwiGLU(FeedForward):
    graph_safe = True
    def __init__(self, spec, prefix="", workspace=None, names=("feed_forward.gate_proj.weight",
                                                                "feed_forward.up_proj.weight",
                                                                "feed_forward.down_proj.weight")):
        super().__init__(spec, prefix)
        self.hidden, self.inter = int(spec["hidden_size"]), int(spec["intermediate_size"])
        self.activation = spec.get("activation", "silu")
        if self.activation not in K.GATE_ACTS:
            raise ValueError(f"dense_swiglu: unknown activation '{self.activation}'; known: {sorted(K.GATE_ACTS)}")
        self.limit = float(spec.get("limit") or 0.0)
        if self.activation == "swish_clamped" and not self.limit > 0:
            raise ValueError("dense_swiglu: the clamped activation needs a positive limit")
        tn = spec.get("tensor_names")
        if tn:
            names = (tn["gate"], tn["up"], tn["down"])
        self.names = tuple(prefix + n for n in names)
        self.token_gate_name = None if spec.get("token_gate") is None else prefix + spec["token_gate"]
        self.ws = workspace
        self.w_gate_up = self.w_down = self.w_token_gate = None

    def requirements(self):
        g, u, d = self.names
        reqs = [TensorReq(g, (self.inter, self.hidden)), TensorReq(u, (self.inter, self.hidden)),
                TensorReq(d, (self.hidden, self.inter))]
        if self.token_gate_name is not None:
            reqs.append(TensorReq(self.token_gate_name, (1, self.hidden)))
        return reqs

    def load(self, source, device):
        g, u, d = self.names
        self.w_gate_up = _stack(source.get(g, device), source.get(u, device))
        self.w_down = source.get(d, device).contiguous()
        if self.token_gate_name is not None:
            self.w_token_gate = source.get(self.token_gate_name, device).contiguous()

    can_store = True          # forward(..., add=False) stores the output (float32) instead of adding it

    def forward(self, h, residual, batch, add=True):
        T = h.shape[0]
        a = self.ws.get("ffn_act", (T, self.inter), h.dtype)
        with phase("mlp"):
            scale = None
            if self.w_token_gate is not None:
                # one number per token, sigmoid(w . h) in float32: the router's dot-product kernel with a single row
                scale = self.ws.get("ffn_token_gate", (T, 1), torch.float32)
                K.row_gates(h, self.w_token_gate, scale)
            # the gate's activation (its clamps too) and the product with `up` happen in the epilogue of the first product
            if self.activation == "swish_clamped":
                project(h, self.w_gate_up, a, MODE_CLAMPED_GLU, gate_limit=self.limit)
            else:
                project(h, self.w_gate_up, a, MODE_SWIGLU if self.activation == "silu" else MODE_GEGLU)
            project(a, self.w_down, residual, MODE_ADD if add else MODE_STORE, row_scale=scale)


UNGATED_ACTIVATIONS = {"relu_squared": MODE_STORE_RELU2, "gelu_tanh": MODE_STORE_GELU}


@register_feed_forward("dense_mlp")
class DenseMLP(FeedForward):
    graph_safe = True
    can_store = True
    ACTIVATIONS = UNGATED_ACTIVATIONS

    def __init__(self, spec, prefix="", workspace=None):
        super().__init__(spec, prefix)
        self.hidden, self.inter = int(spec["hidden_size"]), int(spec["intermediate_size"])
        self.activation = spec.get("activation", "relu_squared")
        if self.activation not in self.ACTIVATIONS:
            raise ValueError(f"dense_mlp: unknown activation '{self.activation}'; known: {list(self.ACTIVATIONS)}")
        tn = {"up": "feed_forward.up_proj.weight", "down": "feed_forward.down_proj.weight"}
        tn.update(spec.get("tensor_names") or {})
        self.names = (prefix + tn["up"], prefix + tn["down"])
        self.ws = workspace
        self.w_up = self.w_down = None

    def requirements(self):
        return [TensorReq(self.names[0], (self.inter, self.hidden)), TensorReq(self.names[1], (self.hidden, self.inter))]

    def load(self, source, device):
        self.w_up = source.get(self.names[0], device).contiguous()
        self.w_down = source.get(self.names[1], device).contiguous()

    def forward(self, h, residual, batch, add=True):
        T = h.shape[0]
        with phase("mlp"):
            a = self.ws.get("mlp_act", (T, self.inter), h.dtype)
            project(h, self.w_up, a, self.ACTIVATIONS[self.activation])      # the activation in the product's epilogue
            project(a, self.w_down, residual, MODE_ADD if add else MODE_STORE)


@register_feed_forward("moe_swiglu")
class MoESwiGLU(FeedForward):
    graph_safe = True
    gated = True
    DEFAULT_ACTIVATION = "silu"
    # the first product's mode, by activation (the activation is part of its epilogue)
    ACTIVATIONS = {"silu": MODE_SWIGLU, "gelu_tanh": MODE_GEGLU, "swish_clamped": MODE_CLAMPED_GLU}

    def __init__(self, spec, prefix="", workspace=None):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden, self.n_experts, self.top_k = int(p["hidden_size"]), int(p["num_experts"]), int(p["top_k"])
        self.inter, self.shared_inter = int(p["expert_size"]), int(p.get("shared_size", 0))
        self.gate_mode = p.get("router_gate", "sigmoid_input")
        if self.gate_mode not in ("sigmoid_input", "sigmoid_output", "none", "softmax_chosen", "sigmoid_normed", "scored"):
            raise ValueError(f"moe_swiglu: unknown router_gate '{self.gate_mode}'")
        self.activation, self.limit = p.get("activation", self.DEFAULT_ACTIVATION), float(p.get("limit") or 0.0)
        if self.activation not in self.ACTIVATIONS:
            raise ValueError(f"{spec.kind}: unknown activation '{self.activation}'; known: {sorted(self.ACTIVATIONS)}")
        if self.activation == "swish_clamped" and not self.limit > 0:
            raise ValueError("moe_swiglu: the clamped activation needs a positive limit")
        self.n_identity = int(p.get("identity_experts") or 0)
        self.n_routed = self.n_experts + self.n_identity           # what the router chooses from
        if self.n_identity < 0 or (self.n_identity and self.gate_mode in ("sigmoid_input", "none")):
            raise ValueError("moe_swiglu: identity experts go with a gate on the experts' outputs")
        rule = dict(p.get("router_rule") or {})
        self.rule = None
        self.n_choice_bias = None
        if self.gate_mode in ("sigmoid_normed", "scored"):
            groups, keep = int(rule.get("groups", 1)), int(rule.get("keep", 1))
            if not (1 <= keep <= groups <= 64) or self.n_routed % groups:
                raise ValueError(f"moe_swiglu: {self.n_routed} experts in {groups} groups of which {keep} are kept")
            if int(p["top_k"]) > keep * (self.n_routed // groups):
                raise ValueError(f"moe_swiglu: top_k {p['top_k']} exceeds the experts of the {keep} kept groups")
            self.rule = {"choice_bias": None, "groups": groups, "keep": keep, "scale": float(rule.get("scale", 1.0))}
            if self.gate_mode == "scored":
                self.rule.update(score=rule.get("score", "sigmoid"), group_score=rule.get("group_score", "top2_sum"),
                                 normalise=bool(rule.get("normalise", True)))
                if self.rule["score"] not in ("sigmoid", "softmax") or self.rule["group_score"] not in ("top2_sum", "max"):
                    raise ValueError(f"moe_swiglu: unknown score '{self.rule['score']}' or group_score "
                                     f"'{self.rule['group_score']}'")
            if rule.get("choice_bias") is not None:
                self.n_choice_bias = prefix + rule["choice_bias"]
        elif rule:
            raise ValueError("moe_swiglu: router_rule belongs to the gates 'sigmoid_normed' and 'scored'")
        if not 1 <= self.top_k <= self.n_routed:
            raise ValueError(f"moe_swiglu: top_k {self.top_k} of {self.n_routed} experts")
        if self.n_routed > 256:
            raise ValueError(f"moe_swiglu: {self.n_routed} experts (supported: up to 256)")
        self.ws = workspace
        f = prefix + "feed_forward."
        self.n_router, self.n_gate_up, self.n_down = f + "router.weight", f + "experts.gate_up_proj", f + "experts.down_proj"
        if p.get("router_name"):
            self.n_router = prefix + p["router_name"]
        self.n_router_bias = None if p.get("router_bias") is None else prefix + p["router_bias"]
        self.layout = p.get("expert_layout", "stacked")
        if self.layout not in ("stacked", "per_expert"):
            raise ValueError(f"moe_swiglu: unknown expert_layout '{self.layout}'")
        self.expert_names = {k: prefix + v for k, v in (p.get("expert_names") or {}).items()}
        # what the first product reads, stacked into one matrix per expert
        self.inputs = ("gate", "up") if self.gated else ("up",)
        if self.layout == "per_expert" and set(self.expert_names) != {*self.inputs, "down"}:
            raise ValueError(f"{spec.kind}: the per_expert layout needs expert_names for {', '.join(self.inputs)} and down")
        if self.layout == "stacked" and not self.gated:
            raise ValueError(f"{spec.kind}: experts without a gate are stored one by one (expert_layout 'per_expert')")
        self.b_router = None
        self.shared = None
        if p.get("shared") is not None:
            from ..config.spec import PartSpec
            self.shared = DenseSwiGLU(PartSpec("dense_swiglu", {"hidden_size": self.hidden, **p["shared"]}), prefix, workspace)
            self.shared_inter = self.shared.inter
        elif self.shared_inter > 0:
            from ..config.spec import PartSpec
            self.shared = DenseSwiGLU(
                PartSpec("dense_swiglu", {"hidden_size": self.hidden, "intermediate_size": self.shared_inter}),
                prefix, workspace, names=("feed_forward.shared_expert.gate_proj.weight",
                                          "feed_forward.shared_expert.up_proj.weight",
                                          "feed_forward.shared_expert.down_proj.weight"))
        self.w_router = self.w_gate_up = self.w_down = None
        # The shared expert does not depend on the routing, so it runs on a second stream beside the routed
        # experts (fork after the norm).  The two must not add into the same residual rows at the same time:
        # either the routed outputs are stored and combined after the join, or (one expert per token, a step of
        # `join_early_tokens` tokens or more) the join comes before the routed down projection, which then adds
        # into the residual itself (measured at 2,048 tokens: 2.5 % of the step).
        self.overlap_shared = True
        self.join_early_tokens = 256
        self._side_stream = None
        self.capture = None        # a list: every forward appends a copy of its expert choices [T, k]

    def requirements(self):
        reqs = [TensorReq(self.n_router, (self.n_routed, self.hidden))]
        if self.n_router_bias is not None:
            reqs.append(TensorReq(self.n_router_bias, (self.n_routed,)))
        if self.n_choice_bias is not None:
            reqs.append(TensorReq(self.n_choice_bias, (self.n_routed,)))
        if self.layout == "per_expert":
            for e in range(self.n_experts):
                reqs += [TensorReq(self.expert_names[n].format(e=e), (self.inter, self.hidden)) for n in self.inputs]
                reqs.append(TensorReq(self.expert_names["down"].format(e=e), (self.hidden, self.inter)))
        else:
            reqs += [TensorReq(self.n_gate_up, (self.n_experts, self.hidden, 2 * self.inter)),
                     TensorReq(self.n_down, (self.n_experts, self.inter, self.hidden))]
        if self.shared is not None:
            reqs += self.shared.requirements()
        return reqs

    def load(self, source, device):
        self.w_router = source.get(self.n_router, device).contiguous()
        if self.n_router_bias is not None:
            self.b_router = source.get(self.n_router_bias, device).to(torch.float32).contiguous()
        if self.n_choice_bias is not None:
            self.rule["choice_bias"] = source.get(self.n_choice_bias, device).to(torch.float32).contiguous()
        if self.layout == "per_expert":                                       # stored [out, in] already
            n = self.expert_names
            get = lambda name, e: source.get(n[name].format(e=e), device)
            self.w_gate_up = torch.stack([_stack(get("gate", e), get("up", e)) if self.gated else get("up", e)
                                          for e in range(self.n_experts)]).contiguous()             # [E, 2I (or I), H]
            self.w_down = torch.stack([source.get(n["down"].format(e=e), device)
                                       for e in range(self.n_experts)]).contiguous()                # [E, H, I]
        else:
            self.w_gate_up = _turned(source.get(self.n_gate_up, device))          # [E, 2I, H]
            self.w_down = _turned(source.get(self.n_down, device))                # [E, H, I]
        if self.shared is not None:
            self.shared.load(source, device)

    def expert_sum(self, h, batch):
        """The routed experts' outputs before they are added up (see ExpertSum), for a block that does more with the sum
        than add it to the residual; None when a shared expert adds to it as well."""
        return None if self.shared is not None else self._run(h, None, batch, defer=True)

    def forward(self, h, residual, batch):
        self._run(h, residual, batch)

    def _run(self, h, residual, batch, defer=False):
        T, E, R, Kk = h.shape[0], self.n_experts, self.n_routed, self.top_k
        ws, i32, f32 = self.ws, torch.int32, torch.float32
        forked = None
        if self.shared is not None and self.overlap_shared and h.is_cuda and phases_active() is None:
            if self._side_stream is None:
                self._side_stream = torch.cuda.Stream(device=h.device)
            fork = torch.cuda.Event()
            fork.record(torch.cuda.current_stream())
            self._side_stream.wait_event(fork)
            with torch.cuda.stream(self._side_stream):
                self.shared.forward(h, residual, batch)
                forked = torch.cuda.Event()
                forked.record(self._side_stream)
        idx = ws.get("moe_topk_idx", (T, Kk), i32)
        gate = ws.get("moe_topk_gate", (T, Kk), f32)
        logits = ws.get("moe_router_logits", (T, R), f32)
        offsets = ws.get("moe_offsets", (R + 1,), i32)
        row_token = ws.get("moe_row_token", (T * Kk,), i32)
        row_scale = ws.get("moe_row_scale", (T * Kk,), f32)
        row_of_slot = ws.get("moe_row_of_slot", (T * Kk,), i32)
        M = T * Kk
        # rows sorted by expert, so that each expert reads a contiguous block (when rows are 16-byte multiples)
        sortable = (h.shape[1] * h.element_size()) % 16 == 0 and h.stride(0) * h.element_size() % 16 == 0
        sorted_h = ws.get("moe_in", (M, self.hidden), h.dtype) if sortable else None
        with phase("moe_router"):
            gathered = K.moe_route(h, self.w_router, idx, gate, logits, offsets, row_token, row_scale, row_of_slot,
                                   top_k=Kk, sorted_h=sorted_h, bias=self.b_router,
                                   sigmoid_gate=self.gate_mode if self.gate_mode in ("softmax_chosen", "sigmoid_normed", "scored")
                                   else self.gate_mode != "none", rule=self.rule)
        if self.capture is not None:
            self.capture.append(idx.clone())
        # identity experts come after the others, so their rows are the last ones and lie outside the products' E groups
        hint = max(1, -(-M // R))
        offsets = offsets[:E + 1]
        act_mode = self.ACTIVATIONS[self.activation]
        act = ws.get("moe_act", (M, self.inter), h.dtype)
        in_scale = row_scale if self.gate_mode == "sigmoid_input" else None
        with phase("moe_expert"):
            if sortable:
                if not gathered:
                    K.gather_rows(h, row_token, sorted_h)
                project(sorted_h, self.w_gate_up, act, act_mode, m_rows=M, row_scale=in_scale, gate_limit=self.limit,
                        group_offsets=offsets, n_groups=E, rows_per_group_hint=hint)
            else:
                project(h, self.w_gate_up, act, act_mode, m_rows=M, a_rows=row_token, row_scale=in_scale,
                        gate_limit=self.limit, group_offsets=offsets, n_groups=E, rows_per_group_hint=hint)
            out_scale = row_scale if self.gate_mode in ("sigmoid_output", "softmax_chosen", "sigmoid_normed", "scored") else None
            # One expert per token: the down projection can add straight into the residual rows.  Beside a shared
            # expert on the second stream that needs an order (two kernels adding into the same rows at once would
            # sum in whatever order they meet): in a step with many tokens the join comes before the down
            # projection (each product fills the GPU by itself, so nothing is lost by the wait, and the stored
            # outputs and the combine kernel go); in a step with few tokens the two chains run side by side to the
            # end and the combine adds the routed outputs after the join.
            join_early = forked is not None and Kk == 1 and T >= self.join_early_tokens and not self.n_identity
            if join_early:
                torch.cuda.current_stream().wait_event(forked)
            direct = Kk == 1 and (forked is None or join_early) and not defer and not self.n_identity
            if direct:
                project(act, self.w_down, residual, MODE_ADD, m_rows=M, out_rows=row_token, row_scale=out_scale,
                        group_offsets=offsets, n_groups=E, rows_per_group_hint=hint)
            else:
                y = ws.get("moe_y", (M, self.hidden), f32)
                project(act, self.w_down, y, MODE_STORE, m_rows=M, row_scale=out_scale,
                        group_offsets=offsets, n_groups=E, rows_per_group_hint=hint)
        if defer:
            return ExpertSum(y, row_of_slot, idx, gate, h, E)
        if not direct:
            if forked is not None:
                torch.cuda.current_stream().wait_event(forked)
            with phase("moe_merge"):
                if self.n_identity:
                    ExpertSum(y, row_of_slot, idx, gate, h, E).add_to(residual)
                else:
                    K.moe_combine(residual, y, row_of_slot, top_k=Kk)
        if forked is not None:
            return
        if self.shared is not None:
            self.shared.forward(h, residual, batch)


@register_feed_forward("moe_mlp")
class MoEMLP(MoESwiGLU):
    """Routed experts of two matrices: the first product's epilogue applies the activation to its float32 sums."""
    gated = False
    DEFAULT_ACTIVATION = "relu_squared"
    ACTIVATIONS = UNGATED_ACTIVATIONS
