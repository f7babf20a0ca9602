"""Katopel's mechanisms one at a time on the GPU, each against the plain implementation's function for it: the two layer norms
around a branch with every sum that may stand between them, biases and neighbouring entries turned together, the delta rule with
one decay per head in its three ways (token by token, in chunks, single tokens) from the packed projection to the gated
read-outs, attention within chunks with keys and values of different sizes and single keys that stand out far away, at page
borders and on both sides of every chunk's edge, the router with the shared expert's weight alone and inside the routed
feed-forward, two mixers in one pair of products, and layers that run several times with adds in front of a pass."""

import math

import pytest
import torch

from tests.plain import katopel as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64


def F():
    from gtar_kimik3_public_b200.ops import functional

    return functional


def _i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def _wide(t):
    return t.detach().double().cpu()


def _layout(lengths, starts=None):
    """tok_pos, tok_seq, cu_q for sequences that bring ``lengths`` tokens from positions ``starts`` on."""
    starts = starts or [0] * len(lengths)
    pos, seq, cu = [], [], [0]
    for s, (n, at) in enumerate(zip(lengths, starts)):
        pos += list(range(at, at + n))
        seq += [s] * n
        cu.append(cu[-1] + n)
    return _i32(pos), _i32(seq), _i32(cu)


def _paged(ks, vs, dtype, seed=0):
    """Pages that hold the sequences' keys ``ks[s] [L, G, d]`` and values ``vs[s] [L, G, dv]`` in a scrambled order, the
    rest NaN; slot of sequence ``s`` is ``n - 1 - s``."""
    n = len(ks)
    G, d, dv = ks[0].shape[1], ks[0].shape[2], vs[0].shape[2]
    per_seq = max(-(-k.shape[0] // PAGE) for k in ks)
    n_pages = n * per_seq + 3
    order = torch.randperm(n_pages, generator=torch.Generator().manual_seed(seed)).tolist()
    k_pages = torch.full((n_pages, G, PAGE, d), float("nan"), dtype=dtype, device=DEV)
    v_pages = torch.full((n_pages, G, PAGE, dv), float("nan"), dtype=dtype, device=DEV)
    table = torch.zeros(n, per_seq, dtype=torch.int32)
    slots = [n - 1 - s for s in range(n)]
    for s, (k, v) in enumerate(zip(ks, vs)):
        for i in range(-(-k.shape[0] // PAGE)):
            page = order.pop()
            table[slots[s], i] = page
            rows = slice(i * PAGE, min((i + 1) * PAGE, k.shape[0]))
            count = rows.stop - rows.start
            k_pages[page, :, :count] = k[rows].transpose(0, 1).to(dtype)
            v_pages[page, :, :count] = v[rows].transpose(0, 1).to(dtype)
    return F().PagedKV(k_pages, v_pages, table.to(DEV)), _i32(slots)


# ------------------------------------------------------------------ layer norms around a branch
def _norm(width, gen, eps):
    return (torch.randn(width, generator=gen, device=DEV), torch.randn(width, generator=gen, device=DEV), eps)


def _plain_norm(x, norm):
    return plain.layer_norm(x, {"n": _wide(norm[0]), "n.b": _wide(norm[1])}, "n", norm[2])


@pytest.mark.parametrize("width,y_dtype,z_dtype,norm_y,first,step,in_place", [
    (88, torch.float32, torch.float32, True, False, False, True), (42, torch.bfloat16, torch.bfloat16, True, True, True, False),
    (1027, torch.bfloat16, torch.float32, True, False, True, True), (2048, torch.bfloat16, torch.bfloat16, True, True, True, True),
    (1024, torch.float32, torch.bfloat16, False, True, False, False), (4100, torch.bfloat16, torch.bfloat16, True, False, False, True),
    (2500, torch.float32, torch.bfloat16, True, True, True, True), (3, torch.float32, torch.float32, True, True, True, True),
    (12288, torch.bfloat16, torch.float32, True, False, True, False), (5001, torch.float32, torch.float32, True, True, False, True),
    (96, None, torch.float32, False, True, True, False), (56, None, torch.bfloat16, False, False, True, True),
    (72, torch.bfloat16, None, True, False, False, True)])
def test_norms_around_a_branch_and_the_adds_between(width, y_dtype, z_dtype, norm_y, first, step, in_place):
    """Rows of very different sizes with a mean far from zero: a variance formed from the mean of squares would be off."""
    gen = torch.Generator(device=DEV).manual_seed(width)
    rand = lambda *shape: torch.randn(*shape, generator=gen, device=DEV)
    T = 13
    x = rand(T, width) * 3.0 + 20.0
    y = None if y_dtype is None else ((rand(T, width) + 5.0) * torch.logspace(-3, 2, T, device=DEV)[:, None]).to(y_dtype)
    ny = _norm(width, gen, 1e-3) if norm_y else None
    nz = None if z_dtype is None else _norm(width, gen, 1e-5)
    f, s = (rand(T, width) * 2.0 if first else None), (rand(width) if step else None)
    want = _wide(x)
    if y is not None:
        want = want + (_plain_norm(_wide(y), ny) if norm_y else _wide(y))
    want = want + (_wide(f) if first else 0.0) + (_wide(s) if step else 0.0)
    before = x.clone()
    out, z = F().layernorm_merge(x, y, ny, first=f, step=s, norm_z=nz, z_dtype=z_dtype or torch.float32, x_out=x if in_place else None)
    assert (out is x) == in_place and (in_place or torch.equal(x, before))
    size = 1.0 + want.abs().amax(-1)
    assert ((_wide(out) - want).abs().amax(-1) / size).max().item() < 2e-6
    if nz is None:
        assert z is None
        return
    assert z.dtype == z_dtype
    err = (_wide(z) - _plain_norm(want, nz)).abs().max().item()
    assert err < (1e-4 if z_dtype == torch.float32 else 4e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_norm_with_a_bias_over_chosen_rows(dtype):
    gen = torch.Generator(device=DEV).manual_seed(9)
    h, norm = torch.randn(20, 77, generator=gen, device=DEV) + 3.0, _norm(77, gen, 1e-2)
    rows = _i32([19, 0, 7])
    got = F().add_layernorm(h, None, norm[0], norm[2], dtype, rows, bias=norm[1])
    want = _plain_norm(_wide(h)[[19, 0, 7]], norm)
    assert (_wide(got) - want).abs().max().item() < (1e-5 if dtype == torch.float32 else 3e-2)
    plain_row = F().add_layernorm(h, None, norm[0], norm[2], torch.float32, rows)
    assert (_wide(plain_row) + _wide(norm[1]) - want).abs().max().item() < 1e-5


# ------------------------------------------------------------------ biases, neighbours turned together
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,rot,at", [(6, 2, 16, 24, 6, 0), (2, 1, 10, 14, 10, 8), (4, 4, 64, 64, 32, 0), (3, 1, 128, 40, 2, 24),
                                             (2, 2, 40, 8, 0, 16)])
def test_biases_and_neighbours_turned_together(dtype, H, G, d, dv, rot, at):
    gen = torch.Generator(device=DEV).manual_seed(H * d + rot)
    lengths, starts, base = [3, 40, 1], [0, 60, 255], 50.0
    pos, seq, _ = _layout(lengths, starts)
    T, nq, nk = sum(lengths), H * d, G * d
    proj = torch.randn(T, at + nq + nk + G * dv + 5, generator=gen, device=DEV).to(dtype)
    bias = torch.randn(nq + nk + G * dv, generator=gen, device=DEV) * 2.0
    angle = torch.arange(300, dtype=torch.float64)[:, None] * torch.tensor([base ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)])[None, :]
    cos, sin = (angle.cos().float().to(DEV), angle.sin().float().to(DEV)) if rot else (None, None)
    blank = [torch.zeros(n + a, G, d) for n, a in zip(lengths, starts)], [torch.zeros(n + a, G, dv) for n, a in zip(lengths, starts)]
    kv, slots = _paged(*blank, dtype)
    q = F().heads_prepare(proj, at, at + nq, at + nq + nk, H, G, d, dv, pos, seq, slots, rot=rot, cos=cos, sin=sin, kv=kv, max_position=299,
                          bias=bias, bias_at=at, neighbours=True)
    p = _wide(proj)[:, at:at + nq + nk + G * dv] + _wide(bias)
    tol = 4e-5 if dtype == torch.float32 else 4e-2
    table = kv.block_table.cpu()
    for s, (n, a) in enumerate(zip(lengths, starts)):
        rows = slice(sum(lengths[:s]), sum(lengths[:s]) + n)
        at_place = lambda t, heads, size: torch.cat([torch.zeros(a, heads, size, dtype=torch.float64), t.reshape(n, heads, size)])
        turned = lambda t, heads: plain.turn_pairs(at_place(t, heads, d), base, rot)[a:] if rot else t.reshape(n, heads, d)
        want_q, want_k, want_v = turned(p[rows, :nq], H), turned(p[rows, nq:nq + nk], G), p[rows, nq + nk:].reshape(n, G, dv)
        assert (_wide(q[rows]) - want_q).abs().max().item() < tol
        for t in range(n):
            page = int(table[int(slots[s]), (a + t) // PAGE])
            assert (_wide(kv.k[page, :, (a + t) % PAGE]) - want_k[t]).abs().max().item() < tol
            assert (_wide(kv.v[page, :, (a + t) % PAGE]) - want_v[t]).abs().max().item() < tol


# ------------------------------------------------------------------ the delta rule with one decay per head
class DeltaCase:
    """Sequences whose packed projections are given; the plain read-outs (norm and gate behind them) and last states."""

    def __init__(self, H, G, d, dv, taps, lengths, dtype, seed=0):
        self.hd = F().DeltaHeads(H, G, d, dv, taps)
        gen = torch.Generator().manual_seed(seed + H * d + dv)
        rand = lambda *shape: torch.randn(*shape, generator=gen)
        hd, self.eps, self.lengths, self.dtype = self.hd, 1e-4, lengths, dtype
        self.at = 16  # the mixer's columns stand inside wider rows
        self.rows = [rand(n, self.at + hd.columns + (-hd.columns) % 8).to(dtype) for n in lengths]
        self.conv, self.a_log, self.dt = rand(hd.channels, taps) * 0.5, rand(H) * 0.7 - 1.5, rand(H) - 1.0
        self.norm = 1.0 + 0.3 * rand(dv)
        self.want, self.states = [], []
        for rows in self.rows:
            x = rows.double()[:, self.at:self.at + hd.columns]
            n = x.shape[0]
            act = plain.silu(plain.over_time(x[:, :hd.channels], self.conv.double()))
            q = plain.unit(act[:, :G * d].view(n, G, d)) * d ** -0.5
            k = plain.unit(act[:, G * d:2 * G * d].view(n, G, d))
            v = act[:, 2 * G * d:].view(n, H, dv)
            beta = torch.sigmoid(x[:, hd.channels:hd.channels + H])
            g = torch.exp(-torch.exp(self.a_log.double()) * torch.nn.functional.softplus(x[:, hd.channels + H:hd.gate_at] + self.dt.double()))
            outs, states = [], []
            for h in range(H):
                a = h // (H // G)
                outs.append(plain.rms(plain.delta_scan(q[:, a], k[:, a], v[:, h], g[:, h], beta[:, h]), self.eps) * self.norm.double())
                # the state behind the last token, read with the unit vectors of every key entry
                last = torch.eye(d, dtype=torch.float64)
                probe = [plain.delta_scan(torch.cat([q[:-1, a], last[i:i + 1]]), k[:, a], v[:, h], g[:, h], beta[:, h])[-1] for i in range(min(d, 3))]
                states.append(torch.stack(probe))
            self.want.append(torch.stack(outs, 1).reshape(n, H * dv) * plain.silu(x[:, hd.gate_at:]))
            self.states.append(torch.stack(states))

    def run(self, cuts, way, slots=(5, 0, 3), out_scale=1.0):
        """``cuts``: per step, how many tokens each sequence brings (0: not in the step).  Returns the read-outs and the state."""
        hd, n_seqs = self.hd, len(self.lengths)
        state = torch.full((7, *hd.state_shape()), float("nan"), device=DEV)
        ring = torch.full((7, *hd.ring_shape()), float("nan"), device=DEV)
        state[list(slots[:n_seqs])] = 0.0
        ring[list(slots[:n_seqs])] = 0.0
        conv, a_log, dt, norm = self.conv.t().contiguous().to(DEV), self.a_log.to(DEV), self.dt.to(DEV), self.norm.to(DEV)
        done, outs = [0] * n_seqs, [[] for _ in range(n_seqs)]
        width = hd.n_heads * hd.dv
        for cut in cuts:
            live = [i for i in range(n_seqs) if cut[i]]
            proj = torch.cat([self.rows[i][done[i]:done[i] + cut[i]] for i in live]).contiguous().to(DEV)
            pos, seq, cu = _layout([cut[i] for i in live], [done[i] for i in live])
            places, lens = _i32([slots[i] for i in live]), _i32([done[i] + cut[i] for i in live])
            out = torch.full((proj.shape[0], width + 12), 7.0, dtype=self.dtype, device=DEV)
            single = max(cut) == 1 and way in ("single", "mixed")
            if single:
                F().delta_head_single(proj, self.at, hd, conv, ring, a_log, dt, norm, state, pos, seq, places, self.eps, out, 8, out_scale)
            else:
                chunks = way in ("chunks", "mixed")
                x = F().delta_head_prepare(proj, self.at, hd, conv, ring, a_log, dt, pos, seq, cu, places, rounded=chunks)
                if hd.taps > 1:
                    F().conv_ring(proj, self.at, hd, ring, cu, lens, places)
                if chunks:
                    o = F().delta_chunked(x, state, cu, places, len(live), max(cut))
                else:
                    o = F().delta_scan(x.q, x.k, x.v, x.g, x.beta, state, cu, places, len(live))
                F().group_norm_gate(o.view(proj.shape[0], -1), hd.dv, norm, proj, self.at + hd.gate_at, self.eps, self.dtype, "silu", out=out,
                                    out_at=8, out_scale=out_scale)
            assert (out[:, :8] == 7.0).all() and (out[:, 8 + width:] == 7.0).all()
            for n, i in enumerate(live):
                outs[i].append(out[int(cu[n]):int(cu[n + 1]), 8:8 + width])
                done[i] += cut[i]
        assert done == list(self.lengths)
        untouched = [s for s in range(7) if s not in slots[:n_seqs]]
        assert torch.isnan(state[untouched]).all() and torch.isnan(ring[untouched]).all()
        return [torch.cat(o) for o in outs], state[list(slots[:n_seqs])]

    def check(self, outs, state, what, out_scale=1.0):
        exact = self.dtype == torch.float32
        for i, want in enumerate(self.want):
            err = (_wide(outs[i]) / out_scale - want).abs()
            size = 1.0 + want.abs().max().item()
            assert torch.isfinite(outs[i].float()).all(), what
            # a read-out that its norm brings up from nearly nothing carries the rounding of the activations up with it
            assert err.max().item() < (5e-4 if exact else 0.6) * size, f"{what}, sequence {i}: {err.max().item():.3e}"
            assert err.mean().item() < (5e-6 if exact else 8e-3) * size, f"{what}, sequence {i}, mean: {err.mean().item():.3e}"
            s = self.states[i]
            off = (_wide(state[i])[:, :s.shape[1]] - s).abs().max().item()
            assert off < (2e-5 if exact else 2e-2) * (1.0 + s.abs().max().item()), f"{what}, state {i}: {off:.3e}"


HEADS = [
    # H, G, d, dv, taps
    (4, 2, 24, 40, 3), (2, 2, 64, 16, 1), (6, 2, 16, 24, 6), (5, 5, 8, 8, 2), (2, 1, 128, 128, 4), (3, 1, 32, 64, 4), (1, 1, 72, 144, 4),
    (2, 1, 48, 256, 4), (2, 2, 96, 32, 5),
]
ODD_HEADS = [(3, 1, 10, 7, 4), (2, 2, 30, 22, 3), (2, 1, 130, 36, 4), (1, 1, 300, 20, 2), (5, 1, 6, 9, 6), (1, 1, 256, 64, 4)]
LENS = [150, 1, 70]
CUTS = {
    "whole": [LENS],
    "portions": [[64, 1, 2], [2, 0, 3], [3, 0, 64], [67, 0, 1], [14, 0, 0]],
    "tokens": [[100, 1, 65]] + [[1, 0, 1]] * 5 + [[1, 0, 0]] * 45,
}


@pytest.mark.parametrize("H,G,d,dv,taps", HEADS + ODD_HEADS)
def test_delta_rule_in_32_bit_under_every_cut(H, G, d, dv, taps):
    """Token by token, and single tokens where a block holds the head; the token-by-token kernel's numbers do not depend on
    the cut at all."""
    case = DeltaCase(H, G, d, dv, taps, LENS, torch.float32)
    fits = F().delta_head_single_fits(d, dv)
    results = {}
    for name, cuts in CUTS.items():
        results[name] = case.run(cuts, "scan")
        case.check(*results[name], f"scan, {name}")
        if name == "tokens" and fits:
            case.check(*case.run(cuts, "single"), f"single, {name}")
    for name in ("portions", "tokens"):
        assert all(torch.equal(a, b) for a, b in zip(results[name][0], results["whole"][0]))
        assert torch.equal(results[name][1], results["whole"][1])
    if fits:  # from the very first token on
        case.check(*case.run([[1, 1, 1]] + [[1, 0, 1]] * 69 + [[1, 0, 0]] * 80, "single", out_scale=0.5), "single from the start", 0.5)


@pytest.mark.parametrize("H,G,d,dv,taps", HEADS)
def test_delta_rule_in_chunks_under_every_cut(H, G, d, dv, taps):
    case = DeltaCase(H, G, d, dv, taps, LENS, torch.bfloat16)
    for name, cuts in CUTS.items():
        case.check(*case.run(cuts, "chunks", out_scale=2.0), f"chunks, {name}", 2.0)
        case.check(*case.run(cuts, "mixed"), f"chunks and single tokens, {name}")
        case.check(*case.run(cuts, "scan"), f"scan, {name}")


@pytest.mark.parametrize("H,G,d,dv,lengths,decay,wave", [(2, 1, 64, 64, [300, 64, 1, 65], 0.02, None), (4, 4, 128, 48, [257, 130], 2.0, None),
                                                         (3, 3, 40, 24, [200], 0.0, 2), (2, 1, 16, 144, [129, 128, 127], 0.3, 1),
                                                         (20, 20, 128, 128, [90, 70], 0.1, None), (1, 1, 8, 8, [64], 40.0, None)])
def test_chunks_against_the_recurrence_on_the_same_numbers(monkeypatch, H, G, d, dv, lengths, decay, wave):
    """The chunked form alone on given rounded vectors: what it leaves out of its split operands is far below bfloat16.  Decays
    from none to so strong that nothing survives a token, and waves of one and two chunks."""
    gen = torch.Generator().manual_seed(d + dv)
    T = sum(lengths)
    q, k, v = (torch.randn(T, n, size, generator=gen).bfloat16() for n, size in ((G, d), (G, d), (H, dv)))
    rq, rk = (1.0 / torch.sqrt(x.double().pow(2).sum(-1) + 1e-6) for x in (q, k))
    k[3:9] = k[3]  # the same key many times: the triangular system is far from the identity
    rk[3:9] = rk[3]
    log_g, beta = -torch.rand(T, H, generator=gen) * decay, torch.sigmoid(torch.randn(T, H, generator=gen) * 2.0)
    start = torch.randn(len(lengths), H, d, dv, generator=gen)
    x = F().DeltaInputs(q.to(DEV), k.to(DEV), v.to(DEV), log_g.to(DEV), beta.to(DEV), (rq * d ** -0.5).float().to(DEV), rk.float().to(DEV))
    cu = _i32([0] + [sum(lengths[:i + 1]) for i in range(len(lengths))])
    if wave:
        monkeypatch.setattr(F(), "DELTA_WORKSPACE_BYTES", wave * 2 * 4 * 64 * 64 * len(lengths) * H)
    state = start.clone().to(DEV)
    got = F().delta_chunked(x, state, cu, _i32(range(len(lengths))), len(lengths), max(lengths))
    at = 0
    for i, n in enumerate(lengths):
        for h in range(H):
            a = h // (H // G)
            S = start[i, h].double()
            kk, qq = k[at:at + n, a].double() * rk[at:at + n, a, None], q[at:at + n, a].double() * rq[at:at + n, a, None] * d ** -0.5
            worst = 0.0
            for t in range(n):
                S = S * math.exp(log_g[at + t, h].item())
                S = S + torch.outer(kk[t], beta[at + t, h].double() * (v[at + t, h].double() - S.T @ kk[t]))
                worst = max(worst, (_wide(got[at + t, h]) - S.T @ qq[t]).abs().max().item())
            assert worst < 1e-4, f"sequence {i} head {h}: {worst:.3e}"
            assert (_wide(state[i, h]) - S).abs().max().item() < 2e-4
        at += n


@pytest.mark.parametrize("way", ["scan", "chunks", "single"])
def test_delta_rule_remembers_a_far_token(way):
    """A value written at the first token, with no decay and later keys orthogonal to the first, is read back 300 tokens later;
    with a decay it is gone by its power."""
    d, dv, n = 16, 8, 301
    for rate in (0.0, 0.01):
        q, k = torch.zeros(n, 1, d), torch.zeros(n, 1, d)
        k[0, 0, 3] = 1.0
        for t in range(1, n):
            k[t, 0, 4 + t % 12] = 1.0
        q[-1, 0, 3] = 1.0
        v = torch.randn(n, 1, dv, generator=torch.Generator().manual_seed(3)).bfloat16()
        ones, log_g = torch.ones(n, 1, device=DEV), torch.full((n, 1), -rate, device=DEV)
        state = torch.zeros(1, 1, d, dv, device=DEV)
        cu, slot = _i32([0, n]), _i32([0])
        if way == "chunks":
            x = F().DeltaInputs(q.bfloat16().to(DEV), k.bfloat16().to(DEV), v.to(DEV), log_g, ones, ones, ones)
            o = F().delta_chunked(x, state, cu, slot, 1, n)
        elif way == "scan":
            o = F().delta_scan(q.to(DEV), k.to(DEV), v.float().to(DEV), log_g.exp(), ones, state, cu, slot, 1)
        else:
            parts = [F().delta_scan(q[t:t + 1].to(DEV), k[t:t + 1].to(DEV), v[t:t + 1].float().to(DEV), log_g[t:t + 1].exp(), ones[t:t + 1], state,
                                    _i32([0, 1]), slot, 1) for t in range(n)]
            o = torch.cat(parts)
        want = v[0, 0].double() * math.exp(-rate * (n - 1))
        assert (_wide(o[-1, 0]) - want).abs().max().item() < 2e-5
        assert o[:-1].abs().max().item() < 1e-5


# ------------------------------------------------------------------ attention within chunks
def _plain_chunked(q, k, v, scale, chunk):
    q, k, v = _wide(q), _wide(k), _wide(v)
    L, H, _ = q.shape
    seen = plain.same_chunk(L, chunk or None)
    outs = []
    for h in range(H):
        g = h // (H // k.shape[1])
        outs.append(torch.softmax(((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf), -1) @ v[:, g])
    return torch.stack(outs, 1)


SIZES = [
    # H, G, d, dv, chunk
    (6, 2, 16, 24, 17), (4, 1, 64, 128, 64), (2, 2, 40, 8, 65), (3, 1, 128, 256, 100), (3, 1, 96, 200, 50), (5, 1, 8, 64, 1),
    (4, 2, 128, 64, 0), (2, 1, 72, 136, 200), (4, 4, 64, 64, 130), (2, 1, 128, 128, 33), (3, 1, 10, 14, 20), (8, 1, 64, 104, 128),
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,chunk", SIZES)
def test_chunked_attention_prompts_portions_and_single_tokens(dtype, H, G, d, dv, chunk):
    """Sequences of unequal length in one launch: all their tokens, the last portion of each, their last tokens alone, on the
    exact kernel (bit-equal however cut) and, where it takes the sizes, on the tensor cores with the walk over the keys cut
    into parts; read-outs into columns of wider rows, times a constant."""
    gen = torch.Generator(device=DEV).manual_seed(H * d + chunk)
    lengths = [333, 77, 1]
    qs, ks, vs = ([torch.randn(L, n, size, generator=gen, device=DEV).to(dtype) for L in lengths] for n, size in ((H, d), (G, d), (G, dv)))
    scale = 1.7 * d ** -0.5
    kv, slots = _paged(ks, vs, dtype)
    want = [_plain_chunked(q, k, v, scale, chunk) for q, k, v in zip(qs, ks, vs)]
    exact = []
    for starts in ([0, 0, 0], [139, 70, 0], [332, 76, 0]):
        pos, seq, cu = _layout([L - a for L, a in zip(lengths, starts)], starts)
        q = torch.cat([q[a:] for q, a in zip(qs, starts)]).contiguous()
        ref = torch.cat([w[a:] for w, a in zip(want, starts)])
        got = F().attention_scored_exact(q, kv, pos, seq, slots, scale, chunk=chunk)
        exact.append(got)
        assert (_wide(got) - ref).abs().max().item() < (3e-5 if dtype == torch.float32 else 3e-2), f"queries from {starts}"
        rows = torch.full((q.shape[0], H * dv + 24), 9.0, dtype=dtype, device=DEV)
        calls = [lambda: F().attention_scored_exact(q, kv, pos, seq, slots, scale, chunk=chunk, out=rows, out_at=16, out_scale=-0.5)]
        if dtype == torch.bfloat16 and F().attention_scored_fits(d, dv):
            longest = max(L - a for L, a in zip(lengths, starts))
            for parts in (1, 2, 3, 9):
                calls.append(lambda parts=parts: F().attention_scored(q, kv, cu, _i32(lengths), slots, longest, scale, n_parts=parts, chunk=chunk,
                                                                      out=rows, out_at=16, out_scale=-0.5))
        for call in calls:
            rows.fill_(9.0)
            call()
            assert (rows[:, :16] == 9.0).all() and (rows[:, 16 + H * dv:] == 9.0).all()
            wide = _wide(rows[:, 16:16 + H * dv]).view(-1, H, dv) / -0.5
            assert torch.isfinite(wide).all() and (wide - ref).abs().max().item() < (3e-5 if dtype == torch.float32 else 4e-2)
    assert F().attention_scored_fits(d, dv) == (d % 8 == 0 and dv % 8 == 0)
    whole = exact[0]
    assert torch.equal(exact[1], torch.cat([whole[139:333], whole[333 + 70:410], whole[410:]]))
    assert torch.equal(exact[2], torch.stack([whole[332], whole[333 + 76], whole[410]]))


EDGES = [
    # chunk, reader i, key j, seen
    (0, 700, 3, True),       # far back, no chunks
    (0, 700, 63, True),      # the last place of the first page
    (0, 700, 64, True),      # the first place of the second
    (0, 700, 700, True),     # the token itself
    (80, 639, 560, True),    # the last place of a chunk reads the first
    (80, 639, 559, False),   # and not the one before it
    (80, 640, 639, False),   # the first place of a chunk does not read its neighbour
    (80, 640, 640, True),
    (64, 127, 64, True),     # chunks that are pages
    (64, 128, 127, False),
    (200, 399, 200, True),   # an edge in the middle of a page
    (200, 399, 199, False),
    (33, 65, 33, True),
    (33, 66, 65, False),
    (1, 300, 300, True),     # a chunk of the token itself
    (1, 300, 299, False),
    (5, 4, 0, True),         # the first tokens of a sequence
    (5, 5, 4, False),
    (500, 40, 0, True),      # a chunk longer than the sequence
    (512, 700, 512, True),   # far back inside a long chunk, on a page's border
    (512, 700, 511, False),
    (640, 639, 0, True),
]


@pytest.mark.parametrize("dtype,d,dv,parts", [(torch.float32, 16, 20, 0), (torch.bfloat16, 10, 14, 0), (torch.bfloat16, 64, 64, 4),
                                              (torch.bfloat16, 88, 176, 1), (torch.bfloat16, 64, 128, 4), (torch.bfloat16, 128, 256, 4)])
@pytest.mark.parametrize("chunk,i,j,seen", EDGES)
def test_chunked_attention_sees_one_key_or_not(dtype, d, dv, parts, chunk, i, j, seen):
    """Among hundreds of small keys one is made to stand out for the query at ``i`` (its score is large, its value is 100 in one
    entry).  If ``j`` is visible from ``i`` that entry of the output is near 100, else near 0: in a whole prompt, in a portion
    that starts in the middle of a tile of rows, and for the token at ``i`` alone over the cache."""
    H, G = 4, 2
    L = i + 5
    gen = torch.Generator(device=DEV).manual_seed(i + j)
    q, k, v = ((torch.randn(L, n, size, generator=gen, device=DEV) * 0.05).to(dtype) for n, size in ((H, d), (G, d), (G, dv)))
    head, kv_head = 3, 1
    q[i, head] = 0.0
    q[i, head, d - 3] = 8.0
    k[j, kv_head, d - 3] = 8.0
    v[j, kv_head] = 0.0
    v[j, kv_head, dv - 2] = 100.0
    kv, slots = _paged([k], [v], dtype, seed=j)
    want = _plain_chunked(q, k, v, 0.5, chunk)
    for first in sorted({0, max(0, i - 37), i}):
        rows = q[first:].contiguous() if first < i else q[i:i + 1].contiguous()
        length = L if first < i else i + 1
        pos, seq, cu = _layout([length - first], [first])
        if parts:
            got = F().attention_scored(rows, kv, cu, _i32([length]), slots, length - first, 0.5, n_parts=parts, chunk=chunk)
        else:
            got = F().attention_scored_exact(rows, kv, pos, seq, slots, 0.5, chunk=chunk)
        value = got[i - first, head, dv - 2].item()
        assert (value > 90.0) == seen and (abs(value) < 2.0) != seen, f"key {j} from {i} (rows from {first}): {value}"
        ref = want[first:] if first < i else want[i:i + 1]
        assert (_wide(got) - ref).abs().max().item() < (2e-4 if dtype == torch.float32 else 0.4)


# ------------------------------------------------------------------ the router and the routed feed-forward
@pytest.mark.parametrize("E,top,T,W", [(6, 2, 50, 88), (9, 3, 7, 40), (4, 4, 33, 64), (40, 5, 130, 96), (1, 1, 20, 24), (63, 6, 700, 72)])
def test_router_with_the_shared_experts_weight(E, top, T, W):
    gen = torch.Generator().manual_seed(E * T)
    h, w_r, w_s = torch.randn(T, W, generator=gen), torch.randn(E, W, generator=gen), torch.randn(1, W, generator=gen) * 0.2
    calls: list = []
    want_ids, want_w = plain.route(h.double(), {"r.router": w_r.double()}, "r.", {"experts": E, "top": top}, calls)
    want_s = torch.sigmoid(h.double() @ w_s.double().T)[:, 0]
    clear = calls[0] > 1e-4
    rows, zeros = torch.cat([w_r, w_s]).to(DEV), torch.zeros(E, device=DEV)
    ids, weights = F().route_groups(h.to(DEV), rows, zeros, top, 1, 1, 1.0, logits=True, shared="pair")
    assert ids.shape == (T, top + 1) and (ids[:, top] == E).all()
    assert (_wide(weights[:, top]) - want_s).abs().max().item() < 1e-5
    ids2, weights2, share = F().route_groups(h.to(DEV), rows, zeros, top, 1, 1, 1.0, logits=True, shared="weight")
    assert torch.equal(ids2, ids[:, :top]) and torch.equal(weights2, weights[:, :top]) and torch.equal(share, weights[:, top])
    assert torch.equal(ids2.cpu().long()[clear], want_ids[clear])
    assert (_wide(weights2)[clear] - want_w[clear]).abs().max().item() < 1e-5
    bare, bare_w = F().route_groups(h.to(DEV), rows[:E].contiguous(), zeros, top, 1, 1, 1.0, logits=True)
    assert torch.equal(bare, ids2) and torch.equal(bare_w, weights2)


@pytest.mark.parametrize("dtype,T", [(torch.float32, 9), (torch.bfloat16, 5), (torch.bfloat16, 300)])
@pytest.mark.parametrize("shared", [None, 24, 40])
def test_routed_feed_forward_with_a_gated_shared_expert(dtype, T, shared):
    """Every token takes all experts (no choice can go the other way): few tokens pair by pair, many through grouped products;
    the shared expert as one more expert (of the experts' size), by itself (another size) and absent; and another branch's output
    folded into the sum."""
    from gtar_kimik3_public_b200.parts.base import StepContext, build_part

    W, ff, E = 88, 24, 3
    part = build_part("feed_forward", "routed_experts", hidden_size=W, expert_size=ff, n_experts=E, top=E, logit_weights=True, bias_name=None,
                      shared_size=shared, shared_gate=True)
    assert part.shared_as_expert == (shared == ff)
    gen = torch.Generator().manual_seed(T + (shared or 0))
    tensors = {n: (torch.randn(s.shape, generator=gen) * (1.0 if n in ("router", "shared.sg") else 0.2)).to(dtype) for n, s in part.tensor_specs().items()}
    assert ("shared.sg" in tensors) == (shared is not None)
    part.load({n: t.to(DEV) for n, t in tensors.items()})
    x = torch.randn(T, W, generator=gen).to(dtype)
    mlp = {"router": {"experts": E, "top": E}, **({"shared": {"ff": shared}} if shared else {})}
    want = plain.routed_ff(x.double(), {"m." + n: t.double() for n, t in tensors.items()}, "m.", mlp)
    got = part.forward(x.to(DEV), None)
    assert got.dtype == torch.float32
    tol = 2e-5 if dtype == torch.float32 else 3e-2 * (1.0 + want.abs().max().item())
    assert (_wide(got) - want).abs().max().item() < tol
    other = torch.randn(T, W, generator=gen).to(dtype)
    assert (_wide(part.forward_added(x.to(DEV), None, other.to(DEV))) - want - other.double()).abs().max().item() < tol
    if shared:
        without = plain.routed_ff(x.double(), {"m." + n: t.double() for n, t in tensors.items()}, "m.", {"router": mlp["router"]})
        assert (want - without).abs().max().item() > 10 * tol, "the shared expert changes nothing: the test would not see it dropped"


# ------------------------------------------------------------------ layers that run several times
def test_a_loop_around_blocks_that_leave_the_adds_to_the_model():
    """The run list's adds with blocks of another kind (pre-norm, which hand their last branch on unadded): the model's step
    equals the same blocks called by hand with the sums formed outside."""
    from gtar_kimik3_public_b200.engine.step import SequenceStep, plan_step
    from gtar_kimik3_public_b200.models.model import Model, StepTable, looped_run_list
    from gtar_kimik3_public_b200.registry import architecture, config_from_dict
    from gtar_kimik3_public_b200.weights.random_init import load_random_weights
    from tests.tiny_configs import TINY_A

    config = config_from_dict(TINY_A)
    n = len(architecture("transformer").build_plan(config).layers)
    for start, stop, times, steps in ((0, n, 2, True), (n - 1, n, 3, False), (1, n, 1, True)):
        plan = architecture("transformer").build_plan(config)
        width = plan.embedding.hidden_size
        plan.run_list = looped_run_list(n, start, stop, times, steps=steps)
        plan.steps = StepTable(times, width) if steps else None
        model = Model(plan, config, torch.float32, torch.device(DEV))
        load_random_weights(model, seed=3)
        tokens = list(range(5, 25))
        got, want = [], None
        for by_hand in (False, True):
            cache = model.make_cache(128, 1)
            slot = cache.open()
            past = cache.grow(slot, len(tokens))
            cache.sync()
            ctx = plan_step([SequenceStep(slot, past, tokens, list(range(len(tokens))))], torch.float32, model.device, model.vocab_size)
            with torch.no_grad():
                if not by_hand:
                    got = model.step(ctx, cache)
                    continue
                model.prepare(ctx.max_position)
                first = plan.embedding.forward(ctx.tokens)
                h = first.clone()
                ctx.extras["cache_read_only"] = False
                done = {}
                for index, entry in enumerate(plan.run_list):
                    if entry.layer == start:
                        t = done.get(start, 0)
                        h = h + (first if t else 0.0) + (plan.steps.table[t] if steps else 0.0)
                    done[entry.layer] = done.get(entry.layer, 0) + 1
                    h, pending = plan.layers[entry.layer].forward(h.contiguous(), None, ctx, cache.view(index))
                    h = h if pending is None else h + pending
                want = plan.head.forward(plan.final_norm.forward(h, None, torch.float32, rows=ctx.want_rows))
        assert done[start] == times and len(plan.run_list) == n + (times - 1) * (stop - start)
        assert (_wide(got) - _wide(want)).abs().max().item() < 2e-5 * (1.0 + want.abs().max().item())
