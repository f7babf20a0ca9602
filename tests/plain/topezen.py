"""A plain, slow implementation of the Topezen decoder, written from the design's equations.

Whole sequences, no cache, one function per mechanism, PyTorch in one working precision
(float64 for the oracle).  It shares no code with the library under test: it reads a dict of
tensors keyed by the model file's names and the config as a plain dict.

Notation: T tokens, W the model width, H heads of ``d`` key and ``dv`` value entries.
"""

from __future__ import annotations

import math

import torch

# When set to torch.bfloat16 every matrix product rounds its operands and its result to that type and what a layer
# stores between its products is kept in it, while norms, angles, scores, softmax, routers, the recurrence and the
# residual sums stay in the working precision: the "standard low-precision implementation" that the bfloat16 tests
# measure the library against.
LOWP: torch.dtype | None = None


def kept(x: torch.Tensor) -> torch.Tensor:
    return x if LOWP is None else x.to(LOWP).to(x.dtype)


def mm(a: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    return a @ b if LOWP is None else kept(kept(a) @ kept(b))


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps): eps inside the root."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def soft_limit(z: torch.Tensor, cap: float | None) -> torch.Tensor:
    return z if cap is None else cap * torch.tanh(z / cap)


def turn_pairs(x: torch.Tensor, base: float) -> torch.Tensor:
    """x [T, heads, n]: entries 2i and 2i+1 turn together by position * base^(-2i/n)."""
    T, _, n = x.shape
    f = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=x.dtype)
    a = torch.arange(T, dtype=x.dtype)[:, None] * f[None, :]
    cos, sin = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * cos - v * sin
    out[..., 1::2] = v * cos + u * sin
    return out


def latent_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """Keys and values from one latent per position, queries through a latent of their own, one turned key part for all
    heads, a gate on every entry of the read-outs."""
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = mm(rms(mm(h, w[p + "dq"].T), eps) * w[p + "dq.norm"], w[p + "uq"].T).view(T, H, d + r)
    both = mm(h, w[p + "dkv"].T)
    c = rms(both[:, :rank], eps) * w[p + "dkv.norm"]
    k_turned = kept(turn_pairs(both[:, None, rank:], m["rot"]["base"])[:, 0])
    q_turned = kept(turn_pairs(q[..., d:], m["rot"]["base"]))
    k = mm(c, w[p + "uk"].T).view(T, H, d)
    v = mm(c, w[p + "uv"].T).view(T, H, dv)
    i = torch.arange(T)
    hidden = i[:, None] < i[None, :]
    outs = []
    for head in range(H):
        s = (q[:, head, :d] @ k[:, head].T + q_turned[:, head] @ k_turned.T) * m["scale"]
        outs.append(torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, head])
    o = torch.stack(outs, 1).reshape(T, H * dv)
    return mm(kept(o) * torch.sigmoid(mm(h, w[p + "g"].T)), w[p + "o"].T)


def matrix_memory(q, k, v, i, f):
    """One head.  q, k [T, d]; v [T, dv]; i, f [T] (logarithms of the input and the forget gate).  C [d, dv], n [d] and
    the running maximum m start at zero; per token m' = max(f + m, i), C = e^(f + m - m') C + e^(i - m') k v^T (n with k
    alone), o = C^T q / (max(|n . q|, e^(-m')) + 1e-6)."""
    T, d = q.shape
    C = torch.zeros(d, v.shape[1], dtype=q.dtype)
    n = torch.zeros(d, dtype=q.dtype)
    top = torch.zeros((), dtype=q.dtype)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        old_share, new_share = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        C = old_share * C + new_share * torch.outer(k[t], v[t])
        n = old_share * n + new_share * k[t]
        top = new
        out.append((C.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-top)) + 1e-6))
    return torch.stack(out)


def mlstm(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    T = h.shape[0]
    q = mm(h, w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = mm(h, w[p + "k"].T).view(T, H, d)
    v = mm(h, w[p + "v"].T).view(T, H, dv)
    i = soft_limit(mm(h, w[p + "i"].T) + w[p + "i.b"], cap)
    f = torch.nn.functional.logsigmoid(soft_limit(mm(h, w[p + "f"].T) + w[p + "f.b"], cap))
    outs = [rms(matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]), eps) for a in range(H)]
    o = torch.stack(outs, 1).reshape(T, H * dv) * w[p + "norm"]
    return mm(o * torch.sigmoid(mm(h, w[p + "g"].T)), w[p + "o"].T)


def visible(T: int, mask: dict | None) -> torch.Tensor:
    """[T, T]: whether position i (row) sees position j (column)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if mask:
        seen &= (i - j < mask["size"]) | (j < (mask.get("keep_first") or 0))
    return seen


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """Grouped heads; an RMS norm per query and key head; capped scores; a window beside which the first tokens stay
    visible; exp(sink) in the denominator."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = kept(rms(mm(h, w[p + "q"].T).view(T, H, d), eps) * w[p + "q.norm"])
    k = kept(rms(mm(h, w[p + "k"].T).view(T, G, d), eps) * w[p + "k.norm"])
    v = mm(h, w[p + "v"].T).view(T, G, dv)
    seen = visible(T, m.get("mask"))
    outs = []
    for head in range(H):
        kh = head // (H // G)
        s = soft_limit((q[:, head] @ k[:, kh].T) * m["scale"], m.get("softcap")).masked_fill(~seen, -math.inf)
        sink = w[p + "sink"][head]
        top = torch.maximum(s.amax(-1, keepdim=True), sink)
        e = torch.exp(s - top)
        outs.append((e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))) @ v[:, kh])
    return mm(torch.stack(outs, 1).reshape(T, H * dv), w[p + "o"].T)


def poly_norm(z: torch.Tensor, numbers: torch.Tensor, eps: float) -> torch.Tensor:
    a, b, c, e = numbers
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def dense_ff(h: torch.Tensor, w: dict, p: str, eps: float) -> torch.Tensor:
    return mm(poly_norm(mm(h, w[p + "up"].T), w[p + "act"], eps), w[p + "down"].T)


def gated_ff(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return mm(silu(mm(h, w[p + "gate"].T)) * mm(h, w[p + "up"].T), w[p + "down"].T)


def route(h: torch.Tensor, w: dict, p: str, r: dict, calls: list | None = None):
    """Chosen experts [T, top] and their weights.  Scores: the softmax over all experts.  Choice by score plus correction
    among the experts of the best groups (a group's score: its largest choice score); weights: the chosen experts'
    scores without the correction over their sum.  ``calls`` receives, per token, how far the closest of the two choices
    (groups, experts) is from going the other way, in units of the scores' deviation over the experts (infinite where everything is chosen)."""
    E, top = r["experts"], r["top"]
    seen = kept(h)  # the router may read the rounding that the experts read
    s = torch.softmax(seen @ w[p + "router"].T, -1)
    choice = s + w[p + "correction"]
    spread = choice.std(-1, correction=0)
    margin = torch.full_like(spread, math.inf)
    groups = r.get("groups")
    if groups and groups["keep"] < groups["count"]:
        n, keep = groups["count"], groups["keep"]
        per = choice.view(-1, n, E // n)
        best = per.amax(-1)
        ranked = best.sort(-1, descending=True)
        margin = torch.minimum(margin, (ranked.values[:, keep - 1] - ranked.values[:, keep]) / spread)
        allowed = torch.zeros_like(best, dtype=torch.bool).scatter_(1, ranked.indices[:, :keep], True)
        choice = choice.masked_fill(~allowed[:, :, None].expand_as(per).reshape(-1, E), -math.inf)
    ranked = choice.sort(-1, descending=True)
    if top < E:
        margin = torch.minimum(margin, (ranked.values[:, top - 1] - ranked.values[:, top]) / spread)
    if calls is not None:
        calls.append(margin)
    ids = ranked.indices[:, :top]
    share = s.gather(1, ids)
    return ids, share / (share.sum(-1, keepdim=True) + 1e-20)


def routed_ff(h: torch.Tensor, w: dict, p: str, mlp: dict, calls: list | None = None) -> torch.Tensor:
    ids, share = route(h, w, p, mlp["router"], calls)
    out = gated_ff(h, w, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += share[rows, place][:, None] * gated_ff(h[rows], w, f"{p}e{e}.")
    return out


MIXERS = {"mlstm": mlstm, "attention": attention, "latent_attention": latent_attention}


def forward(tokens: torch.Tensor, weights: dict, config: dict, dtype=torch.float64, keep_layers: list | None = None,
            calls: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``keep_layers``: a list that receives the stream after every layer; ``calls``:
    a list that receives every routed layer's margins (see ``route``)."""
    w = {name: (t.to(dtype) if t.is_floating_point() else t) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][tokens] * (config.get("embedding") or {"scale": 1.0})["scale"]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        normed = rms(x, eps)
        h = normed * w[p + "norm1"]
        total = x + torch.sigmoid(mm(h, w[p + "rg1"].T) + w[p + "rg1.b"]) * MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = normed * w[p + "norm2"]
            y = dense_ff(h, w, p + "mlp.", eps) if mlp["kind"] == "dense" else routed_ff(h, w, p + "mlp.", mlp, calls)
            total = total + torch.sigmoid(mm(h, w[p + "rg2"].T) + w[p + "rg2.b"]) * y
        x = total
        if keep_layers is not None:
            keep_layers.append(x)
    return mm(rms(x, eps) * w["final.norm"], w["head"].T)
