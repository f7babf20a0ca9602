"""A plain, slow implementation of the Katopel decoder, written from the design's equations.

Whole sequences, no cache, one function per mechanism, PyTorch in one working precision
(float64 for the oracle).  It shares no code with the library under test: it reads a dict of
tensors keyed by the model file's names and the config as a plain dict.

Notation: T tokens, W the model width, H heads and G key/value heads of ``d`` key and ``dv`` value entries.
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


def mm(a: torch.Tensor, b: torch.Tensor, bias: torch.Tensor | None = None) -> torch.Tensor:
    y = kept(a) @ kept(b)
    return kept(y if bias is None else y + bias)


def layer_norm(x: torch.Tensor, w: dict, name: str, eps: float) -> torch.Tensor:
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt(centred.pow(2).mean(-1, keepdim=True) + eps) * w[name] + w[name + ".b"]


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def turn_pairs(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, d]: of the first ``dims`` entries, 2i and 2i+1 turn together by position * base^(-2i/dims)."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype)
    a = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * f[None, :]
    cos, sin = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def same_chunk(T: int, size: int | None) -> torch.Tensor:
    """[T, T]: whether position i (row) sees position j (column)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i // size == j // size)


def chunked_attention(h: torch.Tensor, w: dict, p: str, m: dict) -> torch.Tensor:
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = mm(h, w[p + "q"].T, w[p + "q.b"]).view(T, H, d)
    k = mm(h, w[p + "k"].T, w[p + "k.b"]).view(T, G, d)
    v = mm(h, w[p + "v"].T, w[p + "v.b"]).view(T, G, dv)
    if m.get("rot"):
        q, k = (kept(turn_pairs(x, m["rot"]["base"], m["rot"]["dims"])) for x in (q, k))
    seen = same_chunk(T, (m.get("mask") or {}).get("size"))
    outs = []
    for head in range(H):
        g = head // (H // G)
        s = ((q[:, head] @ k[:, g].T) * m["scale"]).masked_fill(~seen, -math.inf)
        outs.append(torch.softmax(s, -1) @ v[:, g])
    return mm(torch.stack(outs, 1).reshape(T, H * dv), w[p + "o"].T)


def over_time(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """Per channel, x [T, C], taps [C, n]: y_t = sum_j taps[:, n-1-j] x_(t-j), zeros before the start."""
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(min(n, x.shape[0])):
        y[j:] += taps[:, n - 1 - j] * x[:x.shape[0] - j]
    return y


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, g, beta):
    """One head.  q, k [T, d]; v [T, dv]; g, beta [T].  S [d, dv] starts at zero; per token the state shrinks by g, the
    write moves what it holds under k towards v by beta, and the read sees that write."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out.append(S.T @ q[t])
    return torch.stack(out)


def delta_rule(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    part = {n: silu(over_time(mm(h, w[p + n].T), w[p + n + ".conv"])) for n in ("q", "k", "v")}
    q = unit(part["q"].view(T, G, d)) * d ** -0.5
    k = unit(part["k"].view(T, G, d))
    v = part["v"].view(T, H, dv)
    beta = torch.sigmoid(mm(h, w[p + "b"].T))
    g = torch.exp(-torch.exp(w[p + "A_log"]) * torch.nn.functional.softplus(mm(h, w[p + "a"].T) + w[p + "dt_bias"]))
    outs = []
    for head in range(H):
        a = head // (H // G)
        outs.append(rms(delta_scan(q[:, a], k[:, a], v[:, head], g[:, head], beta[:, head]), eps) * w[p + "norm"])
    y = torch.stack(outs, 1).reshape(T, H * dv) * silu(mm(h, w[p + "g"].T))
    return mm(y, w[p + "o"].T)


def two_mixers(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    left = chunked_attention(h, w, p + "left.", m["left"])
    right = delta_rule(h, w, p + "right.", m["right"], eps)
    return m.get("left_scale", 1.0) * left + m.get("right_scale", 1.0) * right


def gated_ff(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return mm(silu(mm(h, w[p + "gate"].T)) * mm(h, w[p + "up"].T), w[p + "down"].T)


def route(h: torch.Tensor, w: dict, p: str, r: dict, calls: list | None = None):
    """Chosen experts [T, top] and their weights: the largest logits, the softmax over those alone.  ``calls`` receives,
    per token, how far the choice is from going the other way, in units of the logits' deviation over the experts
    (infinite where everything is chosen)."""
    E, top = r["experts"], r["top"]
    z = kept(h) @ w[p + "router"].T  # the router may read the rounding that the experts read
    ranked = z.sort(-1, descending=True)
    if calls is not None:
        margin = torch.full_like(z[:, 0], math.inf)
        calls.append(margin if top == E else (ranked.values[:, top - 1] - ranked.values[:, top]) / z.std(-1, correction=0))
    return ranked.indices[:, :top], torch.softmax(ranked.values[:, :top], -1)


def routed_ff(h: torch.Tensor, w: dict, p: str, mlp: dict, calls: list | None = None) -> torch.Tensor:
    ids, share = route(h, w, p, mlp["router"], calls)
    out = torch.zeros_like(h)
    if mlp.get("shared"):
        out = out + torch.sigmoid(mm(h, w[p + "shared.sg"].T)) * gated_ff(h, w, p + "shared.")
    for e in range(mlp["router"]["experts"]):
        rows, place = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += share[rows, place][:, None] * gated_ff(h[rows], w, f"{p}e{e}.")
    return out


def run_order(config: dict) -> list[tuple[int, int | None]]:
    """(layer, pass that begins in front of it or None) in the order of execution."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(tokens: torch.Tensor, weights: dict, config: dict, dtype=torch.float64, keep_layers: list | None = None,
            calls: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``keep_layers``: a list that receives the stream after every layer run;
    ``calls``: a list that receives every routed layer's margins (see ``route``)."""
    w = {name: (t.to(dtype) if t.is_floating_point() else t) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    x = first = w["embed"][tokens] * (config.get("embedding") or {"scale": 1.0})["scale"]
    for i, begins in run_order(config):
        if begins is not None:
            if begins > 0:
                x = x + first
            x = x + w["loop.step"][begins]
        layer, p = config["layers"][i], f"l{i}."
        h = layer_norm(x, w, p + "norm1", eps)
        y = (delta_rule if layer["type"] == "delta" else two_mixers)(h, w, p + "mix.", layer["mixer"], eps)
        x = x + layer_norm(y, w, p + "norm1b", eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = layer_norm(x, w, p + "norm2", eps)
            y = gated_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(h, w, p + "mlp.", mlp, calls)
            x = x + layer_norm(y, w, p + "norm2b", eps)
        if keep_layers is not None:
            keep_layers.append(x)
    return mm(layer_norm(x, w, "final.norm", eps), w["embed"].T)
