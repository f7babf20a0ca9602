"""The Katopel engine against the plain implementation on configurations and schedules drawn from a seed: two to four layers of
the two kinds in any order, loops over any run of them one to three times, head counts, key and value sizes (64, 128 and 256 among
the attention's, sizes that the kernels pad and sizes that they do not take), chunks from 1 position to several pages and
none, rotations of none, part and all of a head with several bases, convolutions of 1 to 6 taps, dense, routed (with a shared
expert of the experts' size, of another and without) and no feed-forwards, widths that are no power of two; batches of one to
six requests whose prompts end on, before and after the edges of a cache page and of the recurrence's chunks, decoded one token
a step for 0 to 70 steps (a request that is through leaves its batch), and a second batch that takes the first one's slots.
Every page starts as NaN, and so does the state of every slot that is not in use.

float32 runs are compared everywhere, within 2e-4 of the float64 oracle.  bfloat16 runs draw routers that choose every
expert (one token sent to another expert changes later logits by order one, see the helpers of the fixed
configurations) and norms with an eps that a nearly zero branch feels, and may err three times as much as the plain
implementation with bfloat16 products and storage."""

import random
import tempfile

import pytest
import torch

from tests.katopel_configs import attention, delta, dense, layer, model, moe, pair
from tests.plain import katopel as plain
from tests.plain.weights import read_safetensors

pytestmark = pytest.mark.gpu

LENGTHS = [1, 2, 3, 15, 17, 31, 33, 47, 48, 63, 64, 65, 100, 127, 128, 129, 191, 200, 257, 300]


def drawn_delta(rng: random.Random) -> dict:
    G = rng.choice([1, 2, 3])
    return delta(G * rng.choice([1, 2, 5]), G, rng.choice([6, 8, 10, 16, 24, 32, 48, 64, 72, 128]), rng.choice([5, 8, 12, 16, 24, 40, 64, 96, 128]),
                 rng.choice([1, 2, 3, 4, 4, 6]))


def drawn_config(rng: random.Random, all_chosen: bool) -> dict:
    width = rng.choice([40, 72, 90, 96, 136, 264])
    layers = []
    for _ in range(rng.choice([2, 3, 4])):
        if rng.random() < 0.4:
            mixer = drawn_delta(rng)
        else:
            G = rng.choice([1, 2, 3])
            dim = rng.choice([8, 10, 16, 24, 40, 64, 64, 96, 128])
            vdim = dim if rng.random() < 0.4 else rng.choice([6, 10, 16, 48, 64, 80, 128, 256])
            left = attention(G * rng.choice([1, 2, 4, 5]), G, dim, vdim, rng.choice([1.0, 2.0, 0.5]) * dim ** -0.5,
                             chunk=rng.choice([None, 1, 2, 31, 64, 65, 100, 200]), rot=rng.choice([None, 2, 4, dim // 4 * 2, dim]),
                             base=rng.choice([37.0, 1e4, 3e5]))
            mixer = pair(left, drawn_delta(rng), rng.choice([None, 0.65, -1.2]), rng.choice([None, 1.2, 0.4]))
        ff = rng.choice(["dense", "moe", "moe", None])
        if ff == "dense":
            mlp = dense(rng.choice([24, 50, 200]))
        elif ff == "moe":
            experts, inner = rng.choice([1, 2, 4, 6, 9]), rng.choice([8, 20, 40])
            mlp = moe(inner, experts, experts if all_chosen else rng.randrange(1, experts + 1), shared=rng.choice([None, inner, inner, 30]))
        else:
            mlp = None
        layers.append(layer(mixer, mlp))
    loop = None
    if rng.random() < 0.8:
        start = rng.randrange(len(layers))
        loop = (start, rng.randrange(start + 1, len(layers) + 1), rng.choice([1, 2, 3]))
    eps = rng.choice([3e-3, 2e-2]) if all_chosen else rng.choice([1e-6, 1e-5, 3e-4])
    return model(rng.choice([100, 257, 1000]), width, eps, rng.choice([None, 0.5, 3.0, width ** 0.5]), layers, loop=loop)


def oracle_and_yardstick(tokens, weights, cfg, with_yardstick):
    ids = torch.tensor(tokens)
    oracle = plain.forward(ids, weights, cfg, torch.float64)
    if not with_yardstick:
        return oracle, 0.0
    plain.LOWP = torch.bfloat16
    try:
        low = plain.forward(ids, weights, cfg, torch.float32).double()
    finally:
        plain.LOWP = None
    return oracle, (low - oracle).abs().max().item()


@pytest.mark.parametrize("seed,dtype", [(s, "float32") for s in range(1, 13)] + [(s, "bfloat16") for s in range(101, 113)])
def test_drawn_configuration_and_schedule(seed, dtype):
    from gtar_kimik3_public_b200.engine import Engine, StepEntry
    from gtar_kimik3_public_b200.generate import load
    from gtar_kimik3_public_b200.registry import config_from_dict
    from gtar_kimik3_public_b200.weights import write_random_model

    rng = random.Random(seed)
    cfg = drawn_config(rng, all_chosen=dtype == "bfloat16")
    n_req = rng.choice([1, 2, 3, 6])
    batches = [([rng.choice(LENGTHS) for _ in range(n_req)], [rng.choice([0, 1, 2, 5, 33, 70]) for _ in range(n_req)])
               for _ in range(2)]
    room = max(sum(-(-(n + d) // 64) * 64 for n, d in zip(*batch)) for batch in batches)  # one batch at a time
    what = f"seed {seed}: {cfg}, prompts and decoded tokens {batches}"
    with tempfile.TemporaryDirectory(prefix="gtar_test_drawn_") as folder:
        write_random_model(folder, config_from_dict(cfg), seed=seed, std=0.08)
        weights = read_safetensors(folder + "/model.safetensors")
        engine = Engine(load(folder, dtype, "cuda:0"), room, max_seqs=n_req)
        for group in engine.cache.kv_groups:
            for pages in (group.k, group.v):
                if pages is not None:
                    pages.fill_(float("nan"))
        for group in engine.cache.state_groups:
            group.state.fill_(float("nan"))
        for number, (prompts, decoded) in enumerate(batches):
            gen = torch.Generator().manual_seed(seed * 10 + number)
            requests = [torch.randint(0, cfg["vocab"], (n + d,), generator=gen).tolist() for n, d in zip(prompts, decoded)]
            checked = [oracle_and_yardstick(tokens, weights, cfg, dtype == "bfloat16") for tokens in requests]
            scale = max(o.abs().max().item() for o, _ in checked)
            limit = 2e-4 * max(1.0, scale) if dtype == "float32" else 3 * max(y for _, y in checked) + 2e-3 + scale / 256
            wants = [sorted({n - 1, rng.randrange(n), rng.randrange(n)}) for n in prompts]
            got = engine.step([StepEntry(i, requests[i][:prompts[i]], wants[i]) for i in range(n_req)]).double().cpu()
            assert torch.isfinite(got).all(), what
            row = 0
            for i in range(n_req):
                for place in wants[i]:
                    err = (got[row] - checked[i][0][place]).abs().max().item()
                    assert err < limit, f"{what}\n{dtype} batch {number} request {i} place {place} of its prompt: {err:.3e} (limit {limit:.3e})"
                    row += 1
            engine.end([i for i in range(n_req) if decoded[i] == 0])
            live = [i for i in range(n_req) if decoded[i] > 0]
            step = 0
            while live:
                got = engine.step([StepEntry(i, [requests[i][prompts[i] + step]], [0]) for i in live]).double().cpu()
                for row, i in enumerate(live):
                    err = (got[row] - checked[i][0][prompts[i] + step]).abs().max().item()
                    assert err < limit, f"{what}\n{dtype} batch {number} request {i} decoded token {step}: {err:.3e} (limit {limit:.3e})"
                step += 1
                engine.end([i for i in live if decoded[i] == step])
                live = [i for i in live if decoded[i] > step]
            engine.cache.check_invariants()
        engine.check()
        assert engine.cache.slots.n_used == 0
