"""A feed-forward of many small gated experts, of which every token uses a few.

Expert ``e``: ``W_down[e] (silu(W_gate[e] x) * (W_up[e] x))``, no biases.  Router: ``z = W_r x`` in 32-bit, scores
``s = sigmoid(z)``; the choice goes by ``s + correction`` (a stored vector), the weights by ``s`` alone.  The experts form
``n_groups`` equal groups of neighbours; a group's score is the sum of its two largest choice scores, and only experts of
the best ``keep_groups`` groups can be chosen (the others count as minus infinity).  The ``top`` largest choice scores are
chosen; a chosen expert's output is weighted by ``s * route_scale`` (not renormalised) and the weighted outputs are added.

Tensors: ``e<i>.gate``, ``e<i>.up`` ``[ff, hidden]``, ``e<i>.down`` ``[hidden, ff]``, ``router`` ``[experts, hidden]``,
``correction`` ``[experts]``; stacked at load into ``[E, 2, ff, hidden]`` and ``[E, hidden, ff]``.

With ``logit_weights`` the router is plainer: scores are the logits plus a stored bias, ``s = z + b`` (the bias tensor's
name is the builder's, ``bias_name``), the ``top`` largest are chosen, and the chosen experts' weights are the softmax
over the chosen scores alone (times ``route_scale``).

Further rules, each a parameter: ``scores="softmax"``: ``s`` is the softmax of the logits over all experts;
``group_rule="best"``: a group's score is its largest choice score; ``renormalise``: the chosen experts' ``s`` are divided
by their sum (plus 1e-20) before ``route_scale``; ``shared_size``: one more expert of that inner size, of the same form
(tensors ``shared.gate``, ``shared.up``, ``shared.down``), runs for every token and is added with weight one, or with
``shared_gate`` with the sigmoid of one number per token, ``W_s x`` in 32-bit (tensor ``shared.sg`` ``[1, hidden]``).  That number
is formed with the router's; a gated shared expert of the experts' own inner size runs as one more expert that every token
has chosen.  ``bias_name`` None: no stored vector on the scores.

The result is 32-bit (it goes into the residual stream); ``forward_added`` folds another branch's output into the
same sum, for blocks whose branches read one norm.
"""

from __future__ import annotations

import torch

from ..ops import functional as F
from ..ops.linear import grouped_product_ok, linear, linear_grouped
from .base import FeedForward, StepContext, TensorSpec, register_part


class RoutedExperts(FeedForward):
    graph_safe = True

    def __init__(self, hidden_size: int, expert_size: int, n_experts: int, top: int, route_scale: float = 1.0,
                 n_groups: int = 1, keep_groups: int = 1, logit_weights: bool = False, bias_name: str | None = "correction",
                 scores: str = "sigmoid", group_rule: str = "two_best", renormalise: bool = False, shared_size: int | None = None, shared_gate: bool = False):
        self.hidden_size, self.ff, self.n_experts, self.top = int(hidden_size), int(expert_size), int(n_experts), int(top)
        self.route_scale, self.n_groups, self.keep = float(route_scale), int(n_groups), int(keep_groups)
        if self.n_experts % self.n_groups or not 1 <= self.keep <= self.n_groups:
            raise ValueError(f"{self.n_experts} experts do not form {self.n_groups} equal groups of which {self.keep} are kept")
        if not 1 <= self.top <= self.keep * (self.n_experts // self.n_groups):
            raise ValueError(f"{self.top} experts cannot be chosen from {self.keep} groups of {self.n_experts // self.n_groups}")
        self.logit_weights, self.bias_name = bool(logit_weights), bias_name
        if scores not in ("sigmoid", "softmax") or group_rule not in ("two_best", "best"):
            raise ValueError("scores are 'sigmoid' or 'softmax', group_rule is 'two_best' or 'best'")
        if self.logit_weights and (scores != "sigmoid" or renormalise):
            raise ValueError("logit weights come with a rule of their own for scores and weights")
        self.scores, self.group_rule, self.renormalise = scores, group_rule, bool(renormalise)
        self.shared_ff = int(shared_size) if shared_size else 0
        self.shared_gate = bool(shared_gate) and self.shared_ff > 0
        self.shared_as_expert = self.shared_gate and self.shared_ff == self.ff
        self.w_shared_gate_up = self.w_shared_down = None
        self.w_gate_up = self.w_down = self.w_router = self.correction = None
        # from this many (token, expert) pairs on, a bfloat16 step sorts its pairs by expert and runs each expert's rows
        # through one tensor-core product; below, every pair streams its expert's weights by itself
        self.grouped_from_pairs = 256

    def tensor_specs(self):
        W, ff = self.hidden_size, self.ff
        specs = {}
        for e in range(self.n_experts):
            specs[f"e{e}.gate"] = TensorSpec((ff, W))
            specs[f"e{e}.up"] = TensorSpec((ff, W))
            specs[f"e{e}.down"] = TensorSpec((W, ff))
        specs["router"] = TensorSpec((self.n_experts, W), init=(0.0, 0.5))
        # softmax scores are small numbers: a correction of the usual size would decide the choice alone
        spread = 0.3 if self.scores == "sigmoid" else 0.3 / self.n_experts
        if self.bias_name is not None:
            specs[self.bias_name] = TensorSpec((self.n_experts,), "vector", init=(0.0, spread))
        if self.shared_ff:
            specs["shared.gate"] = TensorSpec((self.shared_ff, W))
            specs["shared.up"] = TensorSpec((self.shared_ff, W))
            specs["shared.down"] = TensorSpec((W, self.shared_ff))
            if self.shared_gate:
                specs["shared.sg"] = TensorSpec((1, W), init=(0.0, 0.1))
        return specs

    def load(self, tensors):
        E = self.n_experts
        names = [f"e{e}" for e in range(E)] + (["shared"] if self.shared_as_expert else [])
        mats = [tensors[f"{name}.{part}"] for name in names for part in ("gate", "up", "down")]
        kind = torch.float32 if any(m.dtype == torch.float32 for m in mats) else mats[0].dtype
        self.w_gate_up = torch.stack([torch.stack([tensors[name + ".gate"].to(kind), tensors[name + ".up"].to(kind)]) for name in names]).contiguous()
        self.w_down = torch.stack([tensors[name + ".down"].to(kind) for name in names]).contiguous()
        router = [tensors["router"].float()] + ([tensors["shared.sg"].float()] if self.shared_gate else [])
        self.w_router = torch.cat(router, dim=0).contiguous()
        if self.bias_name is None:
            self.correction = torch.zeros(E, dtype=torch.float32, device=self.w_router.device)
        else:
            self.correction = tensors[self.bias_name].float().contiguous()
        if self.shared_ff and not self.shared_as_expert:
            gate, up, down = (tensors["shared." + part] for part in ("gate", "up", "down"))
            if gate.dtype != up.dtype:
                gate, up = gate.float(), up.float()
            # gate and up rows alternate: the activation is the product's output stage
            self.w_shared_gate_up = torch.stack([gate, up], dim=1).reshape(2 * self.shared_ff, self.hidden_size).contiguous()
            self.w_shared_down = down.contiguous()

    def weight_bytes(self):
        """What a single token reads: its ``top`` experts, the shared one and the router."""
        per_expert = (self.w_gate_up[0].numel() + self.w_down[0].numel()) * self.w_down.element_size()
        shared = sum(t.numel() * t.element_size() for t in (self.w_shared_gate_up, self.w_shared_down) if t is not None)
        return (self.top + (1 if self.shared_as_expert else 0)) * per_expert + self.w_router.numel() * 4 + shared

    def route(self, x: torch.Tensor):
        return F.route_groups(x, self.w_router, self.correction, self.top, self.n_groups, self.keep, self.route_scale,
                              logits=self.logit_weights, softmax=self.scores == "softmax", best_of_group=self.group_rule == "best",
                              renormalise=self.renormalise,
                              shared=("pair" if self.shared_as_expert else "weight") if self.shared_gate else None)

    def forward_added(self, x: torch.Tensor, ctx: StepContext, add: torch.Tensor | None) -> torch.Tensor:
        """``add + experts(x)`` as one 32-bit sum (``add``: another branch's output for the same tokens, or None)."""
        add_weight = None
        if self.shared_gate and add is not None:  # the sums' own place for another branch is taken: it is added behind them
            return F.scaled_sum(self.forward_added(x, ctx, None), 1.0, add.float(), 1.0)
        if self.shared_ff and not self.shared_as_expert:
            shared = linear(linear(x, self.w_shared_gate_up, swiglu=True), self.w_shared_down)
            add = shared if add is None else F.scaled_sum(add, 1.0, shared, 1.0).to(x.dtype)
        if self.shared_gate and not self.shared_as_expert:
            ids, weights, add_weight = self.route(x)
        else:
            ids, weights = self.route(x)
        pairs = ids.shape[1]  # of a token
        if x.shape[0] * self.top >= self.grouped_from_pairs and self.ff % 8 == 0 and grouped_product_ok(x, self.w_down):
            # many tokens: the pairs in the order of their experts, each expert's rows through one product
            ends, place_of, pair_at = F.experts_sort(ids, self.w_down.shape[0])
            rows = F.gather_rows(x, pair_at, pairs)
            act = F.swiglu(linear_grouped(rows, self.w_gate_up.view(-1, 2 * self.ff, self.hidden_size), ends))
            return F.experts_combine(linear_grouped(act, self.w_down, ends), place_of, weights, add, add_weight)
        return F.experts_pairwise(x, self.w_gate_up, self.w_down, ids, weights, add, add_weight)

    def forward(self, x, ctx: StepContext) -> torch.Tensor:
        return self.forward_added(x, ctx, None)


register_part("feed_forward", "routed_experts", RoutedExperts)
