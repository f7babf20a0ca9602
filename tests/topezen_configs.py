"""Small Topezen configurations for the tests.  They differ from one another in every size and option: the order of the three
kinds of layer, head counts (one, several, query heads that share key heads two, three and five to one), key and value sizes
that are equal and that differ, sizes that the tensor-core kernels take (64, 128, latents of 64, memory heads of whole
sixteens) and sizes that they do not (odd multiples, no multiple of 4), windows of 1, shorter than a page, a page exactly and
longer, kept first tokens from none to more than the window and more than a page, scores with and without a cap or a
window, caps that bite, rotations over 2 to 32 entries with several bases, caps of the memory's gates that bite and that do
not, dense, routed and no feed-forward, routers with and without groups, with and without a shared expert, that choose one
expert, some and all, an embedding constant that is 1 and that is not, widths that are no power of two.  The configurations
named in ``ALL_CHOSEN`` route every token to all of their experts: no rounding can change a choice there, so their bfloat16
logits are checked at every position (see the helpers' rule for the others)."""


def memory(heads, dim, vdim, cap):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def scored(heads, kv_heads, dim, vdim, scale, softcap=None, window=None, keep=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if window is not None:
        m["mask"] = {"size": window} if keep is None else {"size": window, "keep_first": keep}
    return "attention", m


def latent(heads, dim, rot, vdim, q_rank, kv_rank, scale, base):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                                "rot": {"base": base, "dims": rot}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def model(vocab, width, eps, scale, layers):
    out = {"architecture": "Topezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        out["embedding"] = {"scale": scale}
    return out


TPZ_A = model(300, 88, 1e-5, 3.0, [
    layer(latent(3, 20, 12, 16, 40, 24, 0.2, 1000.0), moe(32, 6, 2, groups=(3, 2), shared=40)),
    layer(memory(3, 24, 40, 6.0), dense(120)),
    layer(scored(6, 2, 16, 24, 0.3, softcap=4.0, window=17, keep=3), None),
    layer(memory(2, 16, 16, 2.5), moe(24, 4, 1, groups=(4, 3), shared=16)),
    layer(scored(4, 4, 24, 24, 0.25, softcap=9.0), dense(72)),
])

# sizes of the tensor-core kernels: attention heads of 64, a latent of 64, memory heads of whole sixteens
TPZ_B = model(257, 64, 1e-6, None, [
    layer(memory(2, 32, 48, 10.0), moe(40, 4, 4, shared=24)),
    layer(scored(4, 2, 64, 64, 0.125, softcap=20.0, window=64, keep=2), dense(96)),
    layer(latent(4, 32, 16, 32, 48, 64, 0.15, 10000.0), moe(32, 6, 6, groups=(2, 2))),
    layer(scored(2, 1, 64, 64, 0.2, window=100, keep=70), None),
])

# heads of 128, memory heads wider than one tile of columns, a rotation over more entries than the unrotated part
TPZ_C = model(190, 96, 1e-5, 0.5, [
    layer(scored(3, 1, 128, 128, 0.07, softcap=3.0, window=65, keep=130), moe(48, 2, 2)),
    layer(memory(1, 64, 144, 15.0), dense(80)),
    layer(latent(2, 16, 32, 40, 24, 128, 0.12, 500.0), None),
    layer(memory(2, 16, 80, 1.0), moe(16, 3, 3, groups=(1, 1), shared=8)),
])

# a window of one position, sizes that are no multiple of 8 or 4, one head
TPZ_D = model(120, 42, 1e-4, 6.3, [
    layer(memory(1, 10, 7, 4.0), None),
    layer(scored(5, 1, 10, 14, 0.4, softcap=2.0, window=1, keep=1), dense(50)),
    layer(latent(5, 7, 2, 9, 11, 13, 0.3, 37.0), moe(8, 9, 3, groups=(3, 1), shared=10)),
    layer(scored(2, 2, 6, 6, 0.5, window=200, keep=0), moe(12, 5, 2)),
    layer(memory(3, 18, 22, 8.0), dense(24)),
])

# one mixer alone and nothing else, with the layer's gates and norms
TPZ_MEMORY = model(97, 48, 1e-6, 2.0, [layer(memory(2, 48, 32, 5.0), None)])
TPZ_LATENT = model(101, 56, 1e-6, 1.0, [layer(latent(3, 24, 16, 24, 32, 64, 0.3, 300.0), None)])
TPZ_SCORED = model(89, 40, 1e-6, 4.0, [layer(scored(4, 1, 64, 64, 0.3, softcap=6.0, window=33, keep=5), None)])

TPZ_CONFIGS = {"tpz_a": TPZ_A, "tpz_b": TPZ_B, "tpz_c": TPZ_C, "tpz_d": TPZ_D, "tpz_memory": TPZ_MEMORY, "tpz_latent": TPZ_LATENT,
               "tpz_scored": TPZ_SCORED}
ALL_CHOSEN = ("tpz_b", "tpz_c", "tpz_memory", "tpz_latent", "tpz_scored")
