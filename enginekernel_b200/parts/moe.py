"""Routed experts: every token goes through ``top`` of E small feed-forwards.

    z = W_router h (32-bit);   s = softmax(z) over all experts
    experts form ``groups`` equal groups of neighbours; a group's score is its best expert's; only
    experts of the ``keep`` best groups can be chosen; the ``top`` largest scores among those are;
    weight = chosen score / (sum of the chosen scores + 1e-20) * ``scale``
    out = sum over the chosen experts of weight * W_down,e act(W_up,e h)

With ``weights="softmax_of_chosen"`` the ``top`` largest logits (of the kept groups) are chosen and the
weights are the softmax over those chosen logits alone, times ``scale``.  With ``gated`` an expert is
W_down,e (act(W_gate,e h) * (W_up,e h)) (tensors ``gate_<e>`` [I, hidden] beside ``up_<e>``; gate and up rows
are interleaved at load, so that one product gives both and its epilogue their 32-bit product).

With ``weights="sigmoid"`` the scores are the logits' sigmoids, each for itself, and the weights are the chosen scores
times ``scale``, not divided by their sum.  With ``weigh="input"`` the weight multiplies the expert's input instead of
its output: out = sum over the chosen experts of W_down,e act(W_up,e (weight h)); the product is linear, so the
weight joins it in the 32-bit sums.  ``shared``, a feed-forward PartSpec, runs for every token and is added.

With ``weights="softmax"`` the weights are the chosen scores of the softmax over all experts, times ``scale`` and not
divided by their sum; with ``corrected`` a learned number per expert (tensor ``correction`` [E + identity], any sign)
joins the scores for the choice, not for the weights.  ``identity`` more experts without tensors stand behind the others
in the router: such an expert's output is the input itself.

Experts have no biases; ``activation`` is ``"relu2"`` (the square of relu), ``"silu"``,
``"gelu_tanh"``, ``"none"`` or, for gated experts, ``"clamped"`` with a ``limit`` (``parts/mlp.py``).  The choice is made and used on the device: a kernel sorts the (token,
choice) pairs by expert and cuts every expert's stretch into row tiles, and the two expert products
walk those tiles, so nothing here waits for the device and the step can be captured in a graph.

Parameters: ``hidden_size``, ``intermediate_size`` (of one expert), ``experts``, ``top``, ``groups``
(default 1), ``keep`` (default: all groups), ``scale``, ``activation``, ``gated`` (default False), ``weights``
(``"scores_of_chosen"``, the default, ``"softmax_of_chosen"``, ``"sigmoid"`` or ``"softmax"``), ``weigh`` (``"output"``, the default, or
``"input"``), ``limit``, ``shared``, ``corrected``, ``identity`` (default 0).  Tensors: ``router`` [E + identity, hidden]
and per expert ``up_<e>`` [I, hidden], ``down_<e>`` [hidden, I].
"""

from __future__ import annotations

import torch

from ..ops import kernels
from ..ops.linear import linear
from ..registry import lookup_part, register_part
from .base import FeedForward
from .spec import TensorSpec


@register_part("feed_forward", "routed_experts")
class RoutedExperts(FeedForward):
    @classmethod
    def tensors(cls, spec):
        p, w = spec.params, spec.weights
        h, i, n = p["hidden_size"], p["intermediate_size"], p["experts"]
        out = [TensorSpec(w["router"], (n + int(p.get("identity") or 0), h))]
        if p.get("corrected"):
            out.append(TensorSpec(w["correction"], (n + int(p.get("identity") or 0),), "around_zero"))
        for e in range(n):
            if p.get("gated"):
                out.append(TensorSpec(w[f"gate_{e}"], (i, h)))
            out += [TensorSpec(w[f"up_{e}"], (i, h)), TensorSpec(w[f"down_{e}"], (h, i))]
        shared = p.get("shared")
        if shared is not None:
            out += lookup_part("feed_forward", shared.kind).tensors(shared)
        return out

    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        g = lambda n: int(self.param(n))
        self.hidden, self.inter, self.experts, self.top = g("hidden_size"), g("intermediate_size"), g("experts"), g("top")
        self.groups = int(spec.params.get("groups") or 1)
        self.keep = int(spec.params.get("keep") or self.groups)
        self.scale = float(spec.params.get("scale", 1.0))
        self.activation = spec.params.get("activation", "relu2")
        self.gated = bool(spec.params.get("gated"))
        self.weights = spec.params.get("weights", "scores_of_chosen")
        self.weigh_input = spec.params.get("weigh", "output") == "input"
        self.limit = float(spec.params.get("limit") or 0.0)
        self.identity = int(spec.params.get("identity") or 0)
        self.corrected = bool(spec.params.get("corrected"))
        self.routed = self.experts + self.identity           # what the router chooses among
        shared = spec.params.get("shared")
        self.shared = None if shared is None else lookup_part("feed_forward", shared.kind)(shared, dtype, device)
        if spec.params.get("weigh", "output") not in ("output", "input"):
            raise ValueError("routed_experts: the weight joins the expert's input or its output")
        if self.activation == "clamped" and not (self.gated and self.limit > 0):
            raise ValueError("routed_experts: the clamped gate needs gated experts and a positive limit")
        if self.weights not in kernels.ROUTE_WEIGHTS:
            raise ValueError(f"routed_experts has no weights {self.weights!r}")
        if self.activation not in kernels.EXPERT_ACTIVATIONS:
            raise ValueError(f"routed_experts has no activation {self.activation!r}")
        if self.routed % self.groups or not 1 <= self.keep <= self.groups:
            raise ValueError("routed_experts: groups must divide experts, 1 <= keep <= groups")
        if not 1 <= self.top <= self.keep * (self.routed // self.groups):
            raise ValueError("routed_experts: top exceeds the experts of the kept groups")
        if self.corrected and self.weights != "softmax":
            raise ValueError("routed_experts: a correction of the choice goes with the weights 'softmax'")
        if self.identity < 0 or (self.identity and self.weigh_input):
            raise ValueError("routed_experts: identity experts are counted from 0 and are weighed on their output")
        self.correction = None
        self.w_router = self.w_up = self.w_down = None

    def load(self, tensors):
        w = self.spec.weights
        if self.shared is not None:
            self.shared.load(tensors)
        router = tensors[w["router"]]           # (zero rows up to a multiple of 16: the library is slow on a ragged few)
        self.w_router = torch.cat([router, router.new_zeros((-self.routed % 16, self.hidden))], 0).to(self.dtype).contiguous()
        if self.corrected:
            self.correction = tensors[w["correction"]].to(torch.float32).contiguous()
        ups = [tensors[w[f"up_{e}"]] for e in range(self.experts)]
        if self.gated:               # rows gate_0, up_0, gate_1, up_1, ... of every expert
            ups = [torch.stack([tensors[w[f"gate_{e}"]], up], 1).reshape(2 * self.inter, self.hidden)
                   for e, up in enumerate(ups)]
        self.w_up = torch.stack(ups).to(self.dtype).contiguous()
        self.w_down = torch.stack([tensors[w[f"down_{e}"]] for e in range(self.experts)]).to(self.dtype).contiguous()

    def bytes_read_per_step(self, n_tokens):
        """The router and the experts that ``n_tokens`` tokens can reach at most."""
        touched = min(self.experts, n_tokens * self.top)
        per_expert = (self.w_up[0].numel() + self.w_down[0].numel()) * self.w_up.element_size()
        shared = self.shared.bytes_read_per_step(n_tokens) if self.shared is not None else 0
        return self.w_router.numel() * self.w_router.element_size() + touched * per_expert + shared

    def forward(self, x, ctx):
        t, ws, top = ctx.n_tokens, ctx.workspace, self.top
        pairs = t * top
        logits = linear(x, self.w_router, ctx, "router_logits", n_rows=t, out_dtype=torch.float32, wide_f32="library")
        chosen = ws.get("moe_chosen", (t, top), torch.int32)
        weight = ws.get("moe_weight", (t, top), torch.float32)
        kernels.moe_route(chosen, weight, logits[:, :self.routed], t, self.groups, self.keep, top, self.scale,
                          weights=self.weights, correction=self.correction)
        sorted_pair = ws.get("moe_sorted", (pairs,), torch.int32)
        tiles = ws.get("moe_tiles", (kernels.moe_max_tiles(pairs, self.experts), 3), torch.int32)
        n_tiles = ws.get("moe_n_tiles", (1,), torch.int32)
        kernels.moe_plan(sorted_pair, tiles, n_tiles, chosen, pairs, self.experts)
        act = ws.get("moe_act", (pairs, self.inter), self.dtype)
        kernels.moe_expert_up(act, x, self.w_up, tiles, n_tiles, sorted_pair, pairs, top, self.activation,
                              gated=self.gated, limit=self.limit, input_weight=weight if self.weigh_input else None)
        pair_out = ws.get("moe_pair_out", (pairs, self.hidden), torch.float32)
        kernels.moe_expert_down(pair_out, act, self.w_down, tiles, n_tiles, sorted_pair,
                                None if self.weigh_input else weight, pairs)
        add = None
        if self.shared is not None:
            self.shared.product_image = self.product_image
            add = self.shared.forward(x, ctx)
        out = ws.get("moe_out", (t, self.hidden), self.dtype)
        kernels.moe_combine(out, pair_out, t, top, add=add,
                            identity=(chosen, weight, x, self.experts) if self.identity else None)
        return out
