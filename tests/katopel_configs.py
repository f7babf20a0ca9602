"""Small Katopel configurations for the tests.  They differ from one another in every size and option: the order of the two
kinds of layer, loops over the first layers, the middle, the last, one layer alone, all of them, once, twice and three times, and no
loop; head counts (one, several, value heads and query heads that share key heads two, three and five to one), key and value
sizes that are equal and that differ either way, sizes that the tensor-core kernels take as they are (64, 128), that they pad
(multiples of 8) and that they do not take (odd multiples), chunks of 1, shorter than a page, a page exactly, longer, and none,
rotations of all of a head, of part and of none with several bases, convolutions of 1 to 6 taps, dense, routed and no
feed-forward, routers that choose one expert, some and all, shared experts of the experts' size, of another and none, an
embedding constant that is 1 and that is not, widths that are no power of two.  The configurations named in ``ALL_CHOSEN`` route
every token to all of their experts: no rounding can change a choice there, so their bfloat16 logits are checked at every
position (see the helpers' rule for the others).

The norms behind a branch bring whatever the branch gives to size one: with random weights and a tiny eps, a token whose
branch happens to be nearly zero has its rounding brought to size one as well, and its bfloat16 error says nothing.  So the
deep configurations have an eps that such a token feels; the single-layer ones have a small eps."""


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attention(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None, base=10000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
    return m


def pair(left, right, left_scale=None, right_scale=None):
    m = {"left": left, "right": right}
    if left_scale is not None:
        m["left_scale"] = left_scale
    if right_scale is not None:
        m["right_scale"] = right_scale
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp):
    return {"type": "parallel" if "left" in mixer else "delta", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, scale, layers, loop=None):
    out = {"architecture": "Katopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        out["embedding"] = {"scale": scale}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


# the middle runs three times; heads that the tensor-core kernels pad; a shared expert of another size and one of the same
KAT_A = model(300, 88, 0.01, 3.0, [
    layer(delta(4, 2, 24, 40, 3), dense(120)),
    layer(pair(attention(6, 2, 16, 24, 0.3, chunk=17, rot=6, base=300.0), delta(3, 1, 16, 32, 4), 0.7, 1.3), moe(32, 6, 2, shared=40)),
    layer(delta(2, 2, 32, 16, 2), moe(24, 4, 1, shared=24)),
    layer(pair(attention(4, 4, 40, 8, 0.2, chunk=50, rot=40), delta(2, 1, 8, 24, 5), -0.5, 0.9), None),
], loop=(1, 3, 3))

# sizes of the tensor-core kernels without padding; the loop over everything; no chunks in one layer
KAT_B = model(257, 64, 0.004, None, [
    layer(pair(attention(4, 2, 64, 64, 0.125, chunk=64, rot=32), delta(2, 1, 64, 64, 4), 0.8, 0.4), moe(40, 4, 4, shared=40)),
    layer(delta(4, 4, 16, 16, 4), dense(96)),
    layer(pair(attention(2, 1, 128, 128, 0.07, rot=128, base=500.0), delta(2, 2, 128, 32, 4), 1.2, 0.55), moe(32, 3, 3, shared=16)),
], loop=(0, 3, 2))

# values wider than keys, 128 and 256 among them; the last layer alone runs twice; a pass that is the only one
KAT_C = model(190, 96, 0.01, 0.5, [
    layer(pair(attention(3, 1, 64, 128, 0.1, chunk=65, rot=2), delta(1, 1, 48, 144, 4), 1.0, 1.0), moe(48, 2, 2)),
    layer(pair(attention(2, 2, 128, 256, 0.09, chunk=100, rot=64, base=77.0), delta(4, 2, 128, 128, 4)), dense(80)),
    layer(delta(3, 3, 64, 96, 1), moe(16, 3, 3, shared=8)),
], loop=(2, 3, 2))

# sizes that are no multiple of 8 or 4, a chunk of one position, a single pass that still takes its vector
KAT_D = model(120, 42, 0.002, 6.3, [
    layer(delta(1, 1, 10, 7, 6), None),
    layer(pair(attention(5, 1, 10, 14, 0.4, chunk=1, rot=4, base=37.0), delta(5, 1, 6, 9, 3), 0.3, 2.0), dense(50)),
    layer(pair(attention(2, 2, 6, 11, 0.5, chunk=200), delta(2, 2, 7, 5, 2), 1.5, -0.7), moe(12, 5, 2, shared=12)),
    layer(delta(6, 2, 30, 22, 4), moe(9, 4, 3)),
], loop=(1, 3, 1))

# one mixer alone and nothing else, with the layer's norms
KAT_DELTA = model(97, 48, 1e-6, 2.0, [layer(delta(3, 1, 48, 32, 4), None)])
KAT_PAIR = model(101, 56, 1e-6, 1.0, [layer(pair(attention(4, 2, 64, 96, 0.15, chunk=33, rot=16), delta(2, 1, 32, 64, 4), 0.9, 0.8), None)])

KAT_CONFIGS = {"kat_a": KAT_A, "kat_b": KAT_B, "kat_c": KAT_C, "kat_d": KAT_D, "kat_delta": KAT_DELTA, "kat_pair": KAT_PAIR}
ALL_CHOSEN = ("kat_b", "kat_c", "kat_delta", "kat_pair")
