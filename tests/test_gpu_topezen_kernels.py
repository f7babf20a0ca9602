"""Topezen's mechanisms one at a time on the GPU, each against the plain implementation's function for it: the two gates with
both adds and the next norms, the activation over three powers of a row, the router (softmax scores, best of a group,
renormalised weights) alone and inside the routed feed-forward with its shared expert, the norms per query and key head,
the matrix memory's three ways (token by token, in chunks, single tokens), and scored attention with capped scores, a window
that keeps the first tokens and a sink, with keys that stand out far away, at page borders and on both sides of every
window's edge, on the exact kernel and on the tensor cores."""

import math

import pytest
import torch

from tests.plain import topezen as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64


def F():
    from gtar_kimik3_public_b200.ops import functional

    return functional


def _i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


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


# ------------------------------------------------------------------ gates, adds, next norms
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,second,norms", [(88, "same", 2), (42, "wide", 2), (1027, "same", 1), (2048, "wide", 2), (40, None, 2),
                                                (96, None, 0), (64, "wide", 0)])
def test_gated_branches_and_next_norms(dtype, width, second, norms):
    gen = torch.Generator(device=DEV).manual_seed(width)
    rand = lambda *shape: torch.randn(*shape, generator=gen, device=DEV)
    T, eps = 21, 1e-5
    x, y1 = rand(T, width) * 2.0, rand(T, width).to(dtype)
    y2 = None if second is None else rand(T, width).to(dtype if second == "same" else torch.float32) * 3.0
    z = rand(T, width * (1 if second is None else 2)).to(dtype)
    b1, b2, g1, g2 = rand(width), rand(width), -1.3, 0.6
    wide = lambda t: t.double().cpu()
    want = wide(x) + torch.sigmoid(g1 * wide(z[:, :width]) + wide(b1)) * wide(y1)
    if y2 is not None:
        want = want + torch.sigmoid(g2 * wide(z[:, width:]) + wide(b2)) * wide(y2)
    stream = x.clone()
    u, n1, n2 = F().gated_merge(stream, dtype, z=z, branch_1=y1, gate_gain_1=g1, bias_1=b1, branch_2=y2, gate_gain_2=g2, bias_2=b2,
                                gain_1=0.7 if norms else None, gain_2=-2.0 if norms == 2 else None, next_eps=eps)
    assert (wide(stream) - want).abs().max().item() < 5e-6
    normed = plain.rms(want, eps)
    tol = 5e-6 if dtype == torch.float32 else 2e-2
    for got, gain in ((u, 1.0), (n1, 0.7), (n2, -2.0)):
        if got is None:
            assert norms == 0 or (gain == -2.0 and norms == 1)
            continue
        assert got.dtype == dtype and (wide(got) - gain * normed).abs().max().item() < tol * max(1.0, abs(gain))
    # the norms alone, without a branch: the stream is left as it is
    before = stream.clone()
    v, m1, _ = F().gated_merge(stream, dtype, gain_1=0.7, next_eps=eps)
    assert torch.equal(stream, before)
    if norms:
        assert torch.equal(v, u) and torch.equal(m1, n1)


# ------------------------------------------------------------------ the dense feed-forward's activation
@pytest.mark.parametrize("dtype_in,dtype_out,width", [(torch.float32, torch.float32, 50), (torch.bfloat16, torch.bfloat16, 4608),
                                                      (torch.float32, torch.bfloat16, 1001), (torch.bfloat16, torch.bfloat16, 72)])
def test_activation_norms_three_powers(dtype_in, dtype_out, width):
    gen = torch.Generator(device=DEV).manual_seed(width)
    z = (torch.randn(13, width, generator=gen, device=DEV) * torch.logspace(-3, 1, 13, device=DEV)[:, None]).to(dtype_in)
    numbers = (0.7, -0.4, 1.3, 0.25)
    got = F().poly_norm(z, numbers, 1e-6, dtype_out).double().cpu()
    want = plain.poly_norm(z.double().cpu(), torch.tensor(numbers, dtype=torch.float64), 1e-6)
    err = ((got - want).abs() / (1.0 + want.abs())).max().item()
    assert err < (3e-6 if dtype_out == torch.float32 else 5e-3)
    # the small rows are where eps shows: without it the cube's norm would be of order one
    assert want[0].abs().max().item() < 4.0 and plain.rms(z.double().cpu() ** 3, 1e-6)[0].abs().max().item() < 1e-3


# ------------------------------------------------------------------ the router
@pytest.mark.parametrize("n_experts,top,groups,T,W", [(6, 2, (3, 2), 50, 88), (9, 3, (3, 1), 7, 40), (4, 4, (1, 1), 33, 64),
                                                      (40, 5, (8, 3), 130, 96), (64, 6, (8, 4), 200, 72), (5, 1, (5, 2), 20, 24)])
def test_router_softmax_scores_best_of_group_renormalised(n_experts, top, groups, T, W):
    gen = torch.Generator().manual_seed(n_experts * T)
    h = torch.randn(T, W, generator=gen)
    w_r = torch.randn(n_experts, W, generator=gen) * 0.2
    # corrections far below zero: every choice score is negative, and a group that is out must not come back as zero
    correction = torch.randn(n_experts, generator=gen) * 0.2 - 2.0
    ids, weights = F().route_groups(h.to(DEV), w_r.to(DEV), correction.to(DEV), top, *groups, 1.0, softmax=True, best_of_group=True,
                                    renormalise=True)
    calls: list = []
    rule = {"experts": n_experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}}
    want_ids, want = plain.route(h.double(), {"r.router": w_r.double(), "r.correction": correction.double()}, "r.", rule, calls)
    clear = calls[0] > 1e-4
    assert clear.sum() > 0.9 * T
    assert torch.equal(ids.cpu().long()[clear], want_ids[clear])
    assert (weights.double().cpu() - want)[clear].abs().max().item() < 1e-5
    assert (weights.sum(-1) - 1.0).abs().max().item() < 1e-5
    # what another rule would have chosen is not the same: two best of a group added, scores without the correction
    for other in (dict(best_of_group=False), dict(softmax=False)):
        if groups[0] > 1 and n_experts > groups[0]:
            their, _ = F().route_groups(h.to(DEV), w_r.to(DEV), correction.to(DEV), top, *groups, 1.0,
                                        **{**dict(softmax=True, best_of_group=True, renormalise=True), **other})
            assert groups[1] == groups[0] or not torch.equal(their.sort(-1).values, ids.sort(-1).values), f"{other} changes no choice"


@pytest.mark.parametrize("dtype,T", [(torch.float32, 9), (torch.bfloat16, 5), (torch.bfloat16, 300)])
def test_routed_feed_forward_with_a_shared_expert(dtype, T):
    """Few tokens (every pair by itself) and many (pairs sorted by expert through grouped products)."""
    from gtar_kimik3_public_b200.parts.base import build_part

    W, ff, n, top, shared = 64, 24, 6, 2, 40
    gen = torch.Generator().manual_seed(T)
    sizes = [(f"e{e}.", ff) for e in range(n)] + [("shared.", shared)]
    w = {name + k: (torch.randn(*shape, generator=gen) * 0.1).to(torch.bfloat16).float()
         for name, f in sizes for k, shape in (("gate", (f, W)), ("up", (f, W)), ("down", (W, f)))}
    w["router"] = torch.randn(n, W, generator=gen) * 0.3
    w["correction"] = torch.randn(n, generator=gen) * 0.05
    part = build_part("feed_forward", "routed_experts", hidden_size=W, expert_size=ff, n_experts=n, top=top, n_groups=3, keep_groups=2,
                      scores="softmax", group_rule="best", renormalise=True, shared_size=shared)
    assert set(part.tensor_specs()) == set(w)
    part.load({name: t.to(DEV).to(torch.float32 if name in ("router", "correction") else dtype) for name, t in w.items()})
    h = (torch.randn(T, W, generator=gen) * 1.5).to(dtype)
    got = part.forward(h.to(DEV), None)
    mlp = {"router": {"experts": n, "top": top, "groups": {"count": 3, "keep": 2}}, "shared": {"ff": shared}}
    calls: list = []
    plain.LOWP = None if dtype == torch.float32 else torch.bfloat16
    try:
        want = plain.routed_ff(h.double(), {"m." + k: t.double() for k, t in w.items()}, "m.", mlp, calls)
    finally:
        plain.LOWP = None
    clear = calls[0] > 1e-4
    assert got.dtype == torch.float32 and clear.sum() > 0.9 * T
    assert (got.double().cpu() - want)[clear].abs().max().item() < (2e-5 if dtype == torch.float32 else 3e-2)
    assert part.weight_bytes() == ((top * ff + shared) * 3 * W) * (4 if dtype == torch.float32 else 2) + n * W * 4


# ------------------------------------------------------------------ norms per query and key head, into the pages
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv", [(6, 2, 16, 24), (5, 1, 10, 14), (2, 2, 64, 64), (3, 1, 128, 40)])
def test_norms_per_head_write_the_pages(dtype, H, G, d, dv):
    gen = torch.Generator(device=DEV).manual_seed(H * d)
    T, start = 75, 50  # over a page border
    width = (H + G) * d + G * dv
    proj = torch.randn(T, width + 3, generator=gen, device=DEV).to(dtype)
    wq, wk = 1.0 + 0.3 * torch.randn(d, generator=gen, device=DEV), 1.0 + 0.3 * torch.randn(d, generator=gen, device=DEV)
    total = start + T
    kv, slots = _paged([torch.zeros(total, G, d, device=DEV)], [torch.zeros(total, G, dv, device=DEV)], dtype)
    pos, seq, _ = _layout([T], [start])
    q = F().heads_prepare(proj, 0, H * d, (H + G) * d, H, G, d, dv, pos, seq, slots, unit_eps=1e-5, w_q=wq, w_k=wk, kv=kv)
    wide = proj.double().cpu()
    want_q = plain.rms(wide[:, :H * d].view(T, H, d), 1e-5) * wq.double().cpu()
    want_k = plain.rms(wide[:, H * d:(H + G) * d].view(T, G, d), 1e-5) * wk.double().cpu()
    want_v = wide[:, (H + G) * d:width].view(T, G, dv)
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    assert (q.double().cpu() - want_q).abs().max().item() < tol
    table = kv.block_table[slots[0]].tolist()
    for t in range(T):
        page, at = table[(start + t) // PAGE], (start + t) % PAGE
        assert (kv.k[page, :, at].double().cpu() - want_k[t]).abs().max().item() < tol
        assert torch.equal(kv.v[page, :, at].double().cpu(), want_v[t])


# ------------------------------------------------------------------ the matrix memory
class Memory:
    """A packed projection of random numbers with its gates' biases, and the plain read-outs after norm, weight and gate."""

    def __init__(self, H, d, dv, lengths, cap, dtype, seed=0, gate_size=1.0, edit=None):
        gen = torch.Generator().manual_seed(seed + 7 * d + dv)
        self.H, self.d, self.dv, self.cap, self.lengths, self.eps = H, d, dv, cap, lengths, 1e-6
        a = [0, H * d, 2 * H * d, 2 * H * d + H * dv, 2 * H * d + 2 * H * dv, 2 * H * d + 2 * H * dv + H]
        self.at = F().MemoryColumns(q=a[0], k=a[1], v=a[2], g=a[3], i=a[4], f=a[5])
        width = a[5] + H
        self.ends = [sum(lengths[:s + 1]) for s in range(len(lengths))]
        proj = torch.randn(self.ends[-1], width + (-width) % 8, generator=gen)
        proj[:, a[4]:width] *= gate_size
        if edit is not None:
            edit(proj, self.at)
        self.bias = torch.cat([torch.randn(H, generator=gen) - 0.5, 2.0 * torch.randn(H, generator=gen) + 2.0])
        self.norm_w = 1.0 + 0.2 * torch.randn(H * dv, generator=gen)
        self.proj = proj.to(dtype).to(DEV)
        self.gate_bias, self.weight = self.bias.to(DEV), self.norm_w.to(DEV)
        self.want = torch.cat([self._plain(self.rows(s).double().cpu()) for s in range(len(lengths))])

    def rows(self, s, start=0, stop=None):
        begin = self.ends[s] - self.lengths[s]
        return self.proj[begin + start:self.ends[s] if stop is None else begin + stop]

    def _plain(self, x):
        H, d, dv, at = self.H, self.d, self.dv, self.at
        i = plain.soft_limit(x[:, at.i:at.i + H] + self.bias[:H].double(), self.cap)
        f = torch.nn.functional.logsigmoid(plain.soft_limit(x[:, at.f:at.f + H] + self.bias[H:].double(), self.cap))
        outs = []
        for h in range(H):
            q, k = x[:, at.q + h * d:at.q + (h + 1) * d] * d ** -0.5, x[:, at.k + h * d:at.k + (h + 1) * d]
            outs.append(plain.rms(plain.matrix_memory(q, k, x[:, at.v + h * dv:at.v + (h + 1) * dv], i[:, h], f[:, h]), self.eps))
        return torch.stack(outs, 1).reshape(-1, H * dv) * self.norm_w.double() * torch.sigmoid(x[:, at.g:at.g + H * dv])

    def states(self, n=None):
        n = n or len(self.lengths)
        return torch.zeros(n, self.H, self.d + 1, self.dv, device=DEV), torch.zeros(n, self.H, self.d + 1, device=DEV)

    def run(self, way, proj, counts, states, slots):
        cu = _i32([sum(counts[:s]) for s in range(len(counts) + 1)])
        core = (proj.contiguous(), self.at, self.gate_bias, self.cap, *states)
        steps = (cu, _i32(slots), len(counts))
        if way == "single":
            return F().memory_single(*core, self.weight, self.eps, *steps)
        if way == "chunks":
            return F().memory_chunked(*core, self.weight, self.eps, *steps, max(counts))
        o, den = F().memory_scan(*core, *steps)
        return F().group_norm_gate(o.view(proj.shape[0], self.H * self.dv), self.dv, self.weight, proj.contiguous(), self.at.g, self.eps,
                                   proj.dtype, divisor=den)


MEMORIES = [
    # H, d, dv, lengths, cap, size of the gates' numbers
    (2, 16, 16, [5, 1, 33], 5.0, 1.0),
    (3, 48, 80, [70, 17], 11.0, 4.0),
    (1, 128, 144, [130], 15.0, 2.0),
    (3, 10, 7, [40, 2], 3.0, 2.0),       # no multiple of 4
    (2, 20, 12, [65], 8.0, 8.0),         # gates that open and shut from token to token
    (1, 132, 20, [40], 6.0, 1.0),
    (1, 264, 16, [20, 3], 6.0, 1.0),
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,dv,lengths,cap,gate_size", MEMORIES)
def test_memory_token_by_token_whole_and_in_portions(dtype, H, d, dv, lengths, cap, gate_size):
    m = Memory(H, d, dv, lengths, cap, dtype, gate_size=gate_size)
    tol = 2e-4 if dtype == torch.float32 else 2e-2
    slots = list(range(len(lengths)))[::-1]
    states = m.states()
    whole = m.run("scan", m.proj, lengths, states, slots)
    assert (whole.double().cpu() - m.want).abs().max().item() < tol
    # the running maximum stands behind the state, one copy a column and one behind n
    C, n = states
    assert torch.equal(C[:, :, d], n[:, :, d, None].expand(-1, -1, dv))
    pieces = [[] for _ in lengths]
    states2 = m.states()
    for step in (2, 1, 3, 16, 200):
        done = [sum(p.shape[0] for p in pieces[s]) for s in range(len(lengths))]
        live = [s for s in range(len(lengths)) if done[s] < lengths[s]]
        if not live:
            break
        counts = [min(step, lengths[s] - done[s]) for s in live]
        out = m.run("scan", torch.cat([m.rows(s, done[s], done[s] + c) for s, c in zip(live, counts)]), counts, states2, [slots[s] for s in live])
        for s, rows in zip(live, out.split(counts)):
            pieces[s].append(rows)
    assert torch.equal(torch.cat([torch.cat(p) for p in pieces]), whole), "portions are not bit-equal to the whole"
    assert all(torch.equal(a, b) for a, b in zip(states, states2))


@pytest.mark.parametrize("H,d,dv,lengths,cap,gate_size", [
    (2, 16, 16, [64], 5.0, 1.0), (3, 48, 96, [300, 64, 1, 65], 11.0, 4.0), (2, 128, 128, [200, 129], 15.0, 1.0), (1, 64, 256, [128, 63], 15.0, 8.0),
    (1, 256, 512, [190], 15.0, 2.0), (2, 32, 80, [191, 2], 3.0, 2.0), (1, 16, 272, [100], 1.0, 3.0), (4, 80, 48, [65, 127, 128], 20.0, 12.0)])
def test_memory_in_chunks(H, d, dv, lengths, cap, gate_size):
    """Chunks of 64 tokens against the plain read-outs and, closer than bfloat16 can show, against the states that the
    token-by-token kernel leaves; then the second half of every sequence from the states after the first."""
    m = Memory(H, d, dv, lengths, cap, torch.bfloat16, gate_size=gate_size)
    slots = [2 * s + 1 for s in range(len(lengths))][::-1]
    one, two, three = (m.states(2 * len(lengths) + 1) for _ in range(3))
    got = m.run("chunks", m.proj, lengths, one, slots)
    assert (got.double().cpu() - m.want).abs().max().item() < 1e-2 * m.want.abs().max().item()
    m.run("scan", m.proj, lengths, two, slots)
    for a, b in zip(one, two):
        assert (a - b).abs().max().item() < 5e-5 * max(1.0, b.abs().max().item())
        assert torch.equal(a[0], torch.zeros_like(a[0])), "a slot that is not in the step was written"
    halves = [n // 2 for n in lengths]
    live = [s for s in range(len(lengths)) if halves[s] > 0]
    first = m.run("chunks", torch.cat([m.rows(s, 0, halves[s]) for s in live]), [halves[s] for s in live], three, [slots[s] for s in live])
    rest = m.run("chunks", torch.cat([m.rows(s, halves[s]) for s in range(len(lengths))]), [n - h for n, h in zip(lengths, halves)], three, slots)
    first = dict(zip(live, first.split([halves[s] for s in live])))
    joined = torch.cat([torch.cat([first[s], r]) if s in first else r for s, r in enumerate(rest.split([n - h for n, h in zip(lengths, halves)]))])
    assert (joined.double().cpu() - m.want).abs().max().item() < 1e-2 * m.want.abs().max().item()
    assert (three[0] - two[0]).abs().max().item() < 5e-5 * max(1.0, two[0].abs().max().item())


def test_memory_in_waves_of_chunks(monkeypatch):
    """With room for a few chunk states only, the chunks of a long prompt go through it in waves."""
    m = Memory(2, 32, 48, [450, 70, 130], 9.0, torch.bfloat16, gate_size=3.0)
    one, two = m.states(), m.states()
    whole = m.run("chunks", m.proj, m.lengths, one, [0, 1, 2])
    monkeypatch.setattr(F(), "DECAY_WORKSPACE_FLOATS", 2 * 3 * 2 * (32 * 48 + 32))
    waves = m.run("chunks", m.proj, m.lengths, two, [0, 1, 2])
    assert torch.equal(whole, waves) and torch.equal(one[0], two[0]) and torch.equal(one[1], two[1])


@pytest.mark.parametrize("H,d,dv,lengths,cap,gate_size", [(2, 16, 16, [9, 4, 1], 5.0, 1.0), (3, 48, 96, [40, 17], 11.0, 4.0), (2, 128, 144, [20, 30], 15.0, 2.0),
                                                          (1, 256, 512, [6], 15.0, 2.0), (2, 20, 12, [40], 3.0, 8.0), (1, 300, 320, [5, 2], 4.0, 1.0)])
def test_memory_single_tokens(H, d, dv, lengths, cap, gate_size):
    """One token of every sequence a step, the shorter ones leaving: read-outs and states as token by token."""
    m = Memory(H, d, dv, lengths, cap, torch.bfloat16, gate_size=gate_size)
    slots = [s + 1 for s in range(len(lengths))]
    one, two = m.states(len(lengths) + 1), m.states(len(lengths) + 1)
    m.run("scan", m.proj, lengths, two, slots)
    out = [[] for _ in lengths]
    for t in range(max(lengths)):
        live = [s for s in range(len(lengths)) if lengths[s] > t]
        rows = m.run("single", torch.cat([m.rows(s, t, t + 1) for s in live]), [1] * len(live), one, [slots[s] for s in live])
        for s, row in zip(live, rows):
            out[s].append(row)
    got = torch.cat([torch.stack(rows) for rows in out])
    assert (got.double().cpu() - m.want).abs().max().item() < 1e-2 * m.want.abs().max().item()
    for a, b in zip(one, two):
        assert (a - b).abs().max().item() < 1e-5 * max(1.0, b.abs().max().item())
    assert torch.equal(one[0][:, :, d], one[1][:, :, d, None].expand(-1, -1, dv))


@pytest.mark.parametrize("way,dtype", [("scan", torch.float32), ("scan", torch.bfloat16), ("chunks", torch.bfloat16), ("mixed", torch.bfloat16)])
def test_memory_remembers_a_far_token(way, dtype):
    """One token's input gate is wide open, a later one's a little, all others' are shut and nothing is forgotten: the first one's
    value is what a far token with the same query reads; with one forget gate shut in between it is the later one's."""
    H, d, dv, T, far = 1, 32, 48, 300, 5
    for forgotten in (False, True):
        def edit(proj, at):
            proj[:, at.q:at.v + dv] *= 0.1
            proj[:, at.i] = -40.0
            proj[far, at.i] = 10.0
            proj[210, at.i] = -5.0
            proj[:, at.f] = 60.0
            if forgotten:
                proj[200, at.f] = -80.0
            proj[far, at.k:at.k + d] = torch.arange(d) / 8.0
            proj[299, at.q:at.q + d] = torch.arange(d) / 8.0
            proj[far, at.v:at.v + dv] = torch.arange(dv) - 20.0
            proj[210, at.k:at.k + d] = torch.arange(d) / 8.0
            proj[210, at.v:at.v + dv] = torch.arange(dv).flip(0) - 20.0

        m = Memory(H, d, dv, [T], 30.0, dtype, edit=edit)
        states = m.states()
        if way == "mixed":  # a prompt in chunks, short portions, single tokens
            parts = [m.run("chunks", m.rows(0, 0, 150), [150], states, [0]), m.run("scan", m.rows(0, 150, 170), [20], states, [0])]
            parts += [m.run("single", m.rows(0, t, t + 1), [1], states, [0]) for t in range(170, 230)]
            parts.append(m.run("chunks", m.rows(0, 230), [70], states, [0]))
            got = torch.cat(parts)
        else:
            got = m.run(way, m.proj, [T], states, [0])
        assert (got.double().cpu() - m.want).abs().max().item() < (1e-3 if dtype == torch.float32 else 3e-2)
        shape = (got[299].double().cpu() / (m.norm_w.double() * torch.sigmoid(m.proj[299, m.at.g:m.at.g + dv].double().cpu()))).view(-1)
        value = torch.arange(dv, dtype=torch.float64) - 20.0
        alike = torch.dot(shape, value) / (shape.norm() * value.norm())
        assert (alike > 0.99) == (not forgotten) and (alike < 0.5) == forgotten


def test_memory_running_maximum_starts_at_zero():
    """A first token whose gates are both far below zero: its denominator is e^(-m) with m = f, not with m = i."""
    def edit(proj, at):
        proj[0, at.i], proj[0, at.f] = -9.0, -3.0

    m = Memory(1, 16, 16, [1], 20.0, torch.float32, edit=edit)
    m.bias.zero_()
    m.gate_bias.zero_()
    C, n = m.states()
    o, den = F().memory_scan(m.proj, m.at, m.gate_bias, m.cap, C, n, _i32([0, 1]), _i32([0]), 1)
    f = -math.log1p(math.exp(20.0 * math.tanh(3.0 / 20.0)))
    assert abs(n[0, 0, 16].item() - f) < 1e-5
    assert abs(den[0, 0].item() - max(math.exp(-f), 0.0) - 1e-6) < 1e-3, "e^(-m) is what divides: the sum of the keys is tiny"


def test_norm_with_a_weight_of_the_whole_row_and_divisors():
    gen = torch.Generator(device=DEV).manual_seed(3)
    T, H, dv = 7, 3, 20
    x, gate = torch.randn(T, H * dv, generator=gen, device=DEV), torch.randn(T, H * dv + 5, generator=gen, device=DEV)
    weight, den = torch.randn(H * dv, generator=gen, device=DEV), torch.rand(T, H, generator=gen, device=DEV) * 1e-2 + 1e-4
    got = F().group_norm_gate(x, dv, weight, gate, 5, 1e-1, torch.float32, divisor=den)
    o = plain.rms(x.double().cpu().view(T, H, dv) / den.double().cpu()[..., None], 1e-1).reshape(T, H * dv)
    want = o * weight.double().cpu() * torch.sigmoid(gate[:, 5:].double().cpu())
    assert (got.double().cpu() - want).abs().max().item() < 1e-5
    plain_row = F().group_norm_gate(x, dv, weight[:dv].contiguous(), gate, 5, 1e-1, torch.float32)
    o = plain.rms(x.double().cpu().view(T, H, dv), 1e-1) * weight[:dv].double().cpu()
    assert (plain_row.double().cpu() - o.reshape(T, H * dv) * torch.sigmoid(gate[:, 5:].double().cpu())).abs().max().item() < 1e-5


# ------------------------------------------------------------------ scored attention: cap, window with kept first tokens, sink
def _plain_scored(q, k, v, scale, window, keep, softcap, sink):
    q, k, v = q.double().cpu(), k.double().cpu(), v.double().cpu()
    L, H, _ = q.shape
    G = k.shape[1]
    seen = plain.visible(L, {"size": window, "keep_first": keep} if window else None)
    outs = []
    for h in range(H):
        s = plain.soft_limit((q[:, h] @ k[:, h // (H // G)].T) * scale, softcap or None).masked_fill(~seen, -math.inf)
        top = torch.maximum(s.amax(-1, keepdim=True), sink[h].double().cpu())
        e = torch.exp(s - top)
        outs.append((e / (e.sum(-1, keepdim=True) + torch.exp(sink[h].double().cpu() - top))) @ v[:, h // (H // G)])
    return torch.stack(outs, 1)


RULES = [
    # H, G, d, dv, window, keep_first, cap
    (6, 2, 16, 24, 17, 3, 4.0),
    (4, 1, 32, 32, 64, 70, 1.5),
    (2, 2, 40, 8, 70, 0, 30.0),
    (3, 1, 24, 40, 0, 0, 2.0),
    (5, 1, 10, 14, 1, 1, 2.0),
    (4, 2, 64, 64, 65, 66, 3.0),
    (6, 2, 64, 64, 17, 3, 2.0),
    (4, 1, 128, 128, 130, 5, 5.0),
    (2, 2, 128, 128, 0, 0, 1.0),
    (2, 1, 64, 64, 1, 1, 8.0),
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,window,keep,cap", RULES)
def test_capped_scores_prompts_portions_and_single_tokens(dtype, H, G, d, dv, window, keep, cap):
    """Sequences of unequal length in one launch: all their tokens, the last portion of each, their last tokens alone, on the
    exact kernel (bit-equal however cut) and, where it takes the sizes, on the tensor cores with the walk over the keys cut
    into parts.  The products are several times the cap."""
    gen = torch.Generator(device=DEV).manual_seed(H * d + window)
    lengths = [333, 77, 1]
    qs, ks, vs = ([torch.randn(L, n, size, generator=gen, device=DEV).to(dtype) for L in lengths] for n, size in ((H, d), (G, d), (G, dv)))
    sink = torch.randn(H, generator=gen, device=DEV) + 1.0
    scale = 4.0 * d ** -0.5
    kv, slots = _paged(ks, vs, dtype)
    want = [_plain_scored(q, k, v, scale, window, keep, cap, sink) for q, k, v in zip(qs, ks, vs)]
    uncapped = _plain_scored(qs[0], ks[0], vs[0], scale, window, keep, 0, sink)
    assert window == 1 or (uncapped - want[0]).abs().max().item() > 0.2 or cap > 8.0, "the cap changes nothing: a test would not see it dropped"
    exact = []
    for starts in ([0, 0, 0], [139, 70, 0], [332, 76, 0]):
        pos, seq, cu = _layout([L - a for L, a in zip(lengths, starts)], starts)
        q = torch.cat([q[a:] for q, a in zip(qs, starts)]).contiguous()
        ref = torch.cat([w[a:] for w, a in zip(want, starts)])
        got = F().attention_scored_exact(q, kv, pos, seq, slots, scale, window, keep, sink=sink, softcap=cap)
        exact.append(got)
        assert (got.double().cpu() - ref).abs().max().item() < (3e-5 if dtype == torch.float32 else 3e-2), f"queries from {starts}"
        if dtype == torch.bfloat16 and d == dv and d in (64, 128):
            longest = max(L - a for L, a in zip(lengths, starts))
            for parts in (1, 2, 3, 9):
                fast = F().attention_scored(q, kv, cu, _i32(lengths), slots, longest, scale, window, keep, n_parts=parts, sink=sink, softcap=cap)
                assert torch.isfinite(fast).all()
                assert (fast.double().cpu() - ref).abs().max().item() < 4e-2, f"queries from {starts}, {parts} parts"
    whole = exact[0]
    assert torch.equal(exact[1], torch.cat([whole[139:333], whole[333 + 70:410], whole[410:]]))
    assert torch.equal(exact[2], torch.stack([whole[332], whole[333 + 76], whole[410]]))


EDGES = [
    # window, keep_first, reader i, key j, seen
    (0, 0, 700, 3, True),        # far back, no window
    (0, 0, 700, 63, True),       # the last place of the first page
    (0, 0, 700, 64, True),       # the first place of the second
    (0, 0, 700, 700, True),      # the token itself
    (96, 20, 700, 605, True),    # just inside the window
    (96, 20, 700, 604, False),   # just outside
    (96, 20, 700, 19, True),     # the last kept first token
    (96, 20, 700, 20, False),    # the first that is not kept
    (96, 20, 700, 0, True),
    (64, 65, 200, 64, True),     # more kept tokens than a page: the second page's first place
    (64, 65, 200, 65, False),
    (64, 65, 200, 136, False),
    (33, 1, 127, 95, True),      # an edge in the middle of a block of 32 keys
    (33, 1, 127, 94, False),
    (32, 0, 128, 97, True),      # an edge on a block's border
    (32, 0, 128, 96, False),
    (1, 0, 300, 300, True),      # a window of the token itself
    (1, 0, 300, 299, False),
    (5, 2, 3, 0, True),          # the first tokens of a sequence: the window has not left anything yet
    (500, 0, 40, 1, True),       # a window longer than the sequence
    (128, 64, 640, 513, True),   # edges on page borders
    (128, 64, 640, 512, False),
    (128, 64, 640, 63, True),
    (128, 64, 640, 64, False),
]


@pytest.mark.parametrize("dtype,d,parts", [(torch.float32, 16, 0), (torch.bfloat16, 24, 0), (torch.bfloat16, 64, 1), (torch.bfloat16, 64, 4),
                                           (torch.bfloat16, 128, 4)])
@pytest.mark.parametrize("window,keep,i,j,seen", EDGES)
def test_capped_scores_see_one_key_or_not(dtype, d, parts, window, keep, i, j, seen):
    """Among hundreds of small keys one is made to stand out for the query at ``i`` (its capped score is large, its value is
    100 in one entry).  If ``j`` is visible from ``i`` that entry of the output is near 100, else near 0: in a whole prompt, in
    a portion that starts in the middle of a tile of rows, and for the token at ``i`` alone over the cache."""
    H, G, dv = 4, 2, d if parts else 20
    L = i + 5
    gen = torch.Generator(device=DEV).manual_seed(i + j)
    q, k, v = ((torch.randn(L, n, size, generator=gen, device=DEV) * 0.05).to(dtype) for n, size in ((H, d), (G, d), (G, dv)))
    head, kv_head = 3, 1
    q[i, head] = 0.0
    q[i, head, 2] = 8.0
    k[j, kv_head, 2] = 8.0
    v[j, kv_head] = 0.0
    v[j, kv_head, 7] = 100.0
    sink = torch.full((H,), 2.0, device=DEV)
    cap = 25.0  # the score that stands out: 25 tanh(32 / 25) = 21
    kv, slots = _paged([k], [v], dtype, seed=j)
    want = _plain_scored(q, k, v, 0.5, window, keep, cap, sink)
    for first in sorted({0, max(0, i - 37), i}):
        rows = q[first:].contiguous() if first < i else q[i:i + 1].contiguous()
        length = L if first < i else i + 1
        pos, seq, cu = _layout([length - first], [first])
        if parts:
            got = F().attention_scored(rows, kv, cu, _i32([length]), slots, length - first, 0.5, window, keep, n_parts=parts, sink=sink, softcap=cap)
        else:
            got = F().attention_scored_exact(rows, kv, pos, seq, slots, 0.5, window, keep, sink=sink, softcap=cap)
        value = got[i - first, head, 7].item()
        assert (value > 90.0) == seen and (abs(value) < 2.0) != seen, f"key {j} from {i} (rows from {first}): {value}"
        ref = want[first:] if first < i else want[i:i + 1]
        assert (got.double().cpu() - ref).abs().max().item() < (2e-4 if dtype == torch.float32 else 0.4)


def test_a_sink_is_neither_scaled_nor_capped():
    """A token that sees itself alone: its share is e^s / (e^s + e^sink) with the capped score s and the sink as it is stored."""
    H, d, cap = 2, 64, 3.0
    q, k, v = torch.zeros(2, H, d, device=DEV), torch.zeros(2, 1, d, device=DEV), torch.full((2, 1, d), 4.0, device=DEV)
    q[:, :, 0], k[:, :, 0] = 4.0, 2.0  # every product 8, times 0.5
    sink = torch.tensor([5.0, 1.0], device=DEV)  # the first lies above the cap
    s = cap * math.tanh(4.0 / cap)
    for dtype in (torch.float32, torch.bfloat16):
        kv, slots = _paged([k.to(dtype)], [v.to(dtype)], dtype)
        pos, seq, cu = _layout([2])
        got = [F().attention_scored_exact(q.to(dtype), kv, pos, seq, slots, 0.5, 1, 0, sink=sink, softcap=cap)]
        if dtype == torch.bfloat16:
            got.append(F().attention_scored(q.to(dtype), kv, cu, _i32([2]), slots, 2, 0.5, 1, 0, sink=sink, softcap=cap))
        for out in got:
            for head in range(H):
                share = math.exp(s) / (math.exp(s) + math.exp(sink[head].item()))
                assert (out[:, head].double() - 4.0 * share).abs().max().item() < (1e-5 if dtype == torch.float32 else 2e-2)
