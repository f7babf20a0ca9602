"""A recurrent mixer: a matrix memory per head with an exponential input gate and a forget gate (the mLSTM of xLSTM).

Per head, with ``q = W_q x * d^(-1/2)``, ``k = W_k x`` (heads of ``key_dim``) and ``v = W_v x`` (heads of ``value_dim``), the
logarithms of the two gates

    i = cap tanh((W_i x + b_i) / cap) ;     f = logsigmoid(cap tanh((W_f x + b_f) / cap))

and a state ``C [d, dv]``, ``n [d]`` and a running maximum ``m``, all zero at the start of a sequence:

    m' = max(f + m, i) ;  C <- e^(f + m - m') C + e^(i - m') k v^T ;  n <- e^(f + m - m') n + e^(i - m') k
    o = C^T q / (max(|n . q|, e^(-m')) + 1e-6)

Every head's ``o`` is divided by its root mean square, the concatenated heads are multiplied by a weight of all heads' size
(tensor ``norm``) and by the sigmoid of ``W_g x``, and go through ``W_o``.

The factor ``d^(-1/2)`` stands on k in the kernels: q and k only ever meet in products, so the numbers are the same.

What a sequence keeps between steps, all 32-bit: ``C`` with one more row, ``[heads, d + 1, dv]``, and ``n`` with one more
entry, ``[heads, d + 1]``.  The last row and entry hold ``m``: a copy for every column of the state and for ``n``, so that
blocks that own different columns of one head read and write nothing of one another's.

A step's kernels: the packed projection q | k | v | g | i | f; the recurrence, which reads it as it is; norm and gate; the
output projection.  In bfloat16 steps of one token a sequence the recurrence, norm and gate are one kernel, and in bfloat16
steps of many tokens the recurrence runs in chunks of 64 tokens whose inner work is matrix products, with norm and gate in
its last kernel; short portions and 32-bit runs go token by token (in a 32-bit run a token's sums have the same order
however a prompt is cut).
"""

from __future__ import annotations

import torch

from ..ops import functional as F
from ..ops.linear import linear
from .base import Mixer, StateRequest, StepContext, TensorSpec, register_part
from .delta_rule import _pad_rows

_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "i": "i", "i_bias": "i.b", "f": "f", "f_bias": "f.b", "norm": "norm", "o": "o"}


class MatrixMemory(Mixer):
    graph_safe = True  # kernels only; starts, slots and lengths are read from device memory
    chunked_from = 48  # steps whose longest sequence brings this many tokens take the chunked kernels (bfloat16 runs)

    def __init__(self, hidden_size: int, n_heads: int, key_dim: int, value_dim: int, gate_cap: float, norm_eps: float,
                 names: dict[str, str] | None = None):
        self.hidden_size, self.n_heads, self.d, self.dv = int(hidden_size), int(n_heads), int(key_dim), int(value_dim)
        self.gate_cap, self.norm_eps = float(gate_cap), float(norm_eps)
        if min(self.hidden_size, self.n_heads, self.d, self.dv) <= 0 or not self.gate_cap > 0:
            raise ValueError("matrix memory sizes and the gates' cap must be positive")
        self.names = {**_NAMES, **(names or {})}
        self.w_in = self.w_gates = self.gate_bias = self.norm_w = self.w_o = None

    def tensor_specs(self):
        n, W, H, d, dv = self.names, self.hidden_size, self.n_heads, self.d, self.dv
        return {
            n["q"]: TensorSpec((H * d, W)), n["k"]: TensorSpec((H * d, W)), n["v"]: TensorSpec((H * dv, W)),
            n["g"]: TensorSpec((H * dv, W)),
            n["i"]: TensorSpec((H, W)), n["i_bias"]: TensorSpec((H,), "vector", init=(-1.0, 1.0)),
            n["f"]: TensorSpec((H, W)), n["f_bias"]: TensorSpec((H,), "vector", init=(3.0, 1.5)),
            n["norm"]: TensorSpec((H * dv,), "vector"),
            n["o"]: TensorSpec((W, H * dv)),
        }

    def load(self, tensors):
        n = self.names
        mats = [tensors[n[key]] for key in ("q", "k", "v", "g", "i", "f")]
        if len({m.dtype for m in mats}) != 1:
            mats = [m.float() for m in mats]
        self.w_in = _pad_rows(torch.cat(mats, dim=0)).contiguous()
        self.w_o = tensors[n["o"]].contiguous()
        self.gate_bias = torch.cat([tensors[n["i_bias"]].float(), tensors[n["f_bias"]].float()]).contiguous()
        self.norm_w = tensors[n["norm"]].float().contiguous()

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o))

    def cache_request(self):
        return [StateRequest((self.n_heads, self.d + 1, self.dv), torch.float32), StateRequest((self.n_heads, self.d + 1), torch.float32)]

    def forward(self, x, ctx: StepContext, cache) -> torch.Tensor:
        if ctx.extras.get("cache_read_only", False):
            raise ValueError("a recurrent mixer advances its state at every step: it cannot run on another entry's storage")
        state, n_state = cache
        H, d, dv = self.n_heads, self.d, self.dv
        proj = linear(x, self.w_in)
        at = F.MemoryColumns(q=0, k=H * d, v=2 * H * d, g=2 * H * d + H * dv, i=2 * H * d + 2 * H * dv, f=2 * H * d + 2 * H * dv + H)
        core = (proj, at, self.gate_bias, self.gate_cap, state, n_state)
        steps = (ctx.cu_q, ctx.slots, ctx.n_seqs)
        half = ctx.dtype == torch.bfloat16 and proj.dtype == torch.bfloat16
        if half and ctx.all_single and F.memory_single_fits(d, dv):
            y = F.memory_single(*core, self.norm_w, self.norm_eps, *steps)
        elif half and ctx.max_q_len >= self.chunked_from and F.memory_chunked_fits(d, dv, at, proj.shape[1]):
            y = F.memory_chunked(*core, self.norm_w, self.norm_eps, *steps, ctx.max_q_len)
        else:  # few tokens a sequence, other sizes, and 32-bit runs (whose numbers do not depend on how a prompt is cut)
            o, den = F.memory_scan(*core, *steps)
            y = F.group_norm_gate(o.view(ctx.n_tokens, H * dv), dv, self.norm_w, proj, at.g, self.norm_eps, ctx.dtype, divisor=den)
        return linear(y, self.w_o)


register_part("mixer", "mlstm", MatrixMemory)
