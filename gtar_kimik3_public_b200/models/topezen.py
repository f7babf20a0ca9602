"""The Topezen decoder put together from parts.

Token embedding times a constant; per layer a ``GatedParallelBlock`` (two branches read the same stream, each through an RMS
norm with ONE number; every branch's result is multiplied entry by entry by the sigmoid of a projection of what the branch
reads, and both are added to the stream at once) around one of three mixers and a feed-forward (dense with the PolyNorm
activation, routed experts with a shared one, or none); the model's last norm (one number again); an output head of its own.
The mixers, by the layer's ``type``:

* ``latent_attention``: keys and values from one cached latent per position, queries through a latent of their own, the
  rotated parts paired entry with neighbour, a sigmoid gate per entry;
* ``mlstm``: a matrix memory with an exponential input gate and a forget gate per head;
* ``attention``: the scored attention of this library under another set of rules: an RMS norm with a weight per query and key
  head, no rotation, scores capped by a tanh, a window beside which the first tokens stay visible, a learned sink per head.

Each layer's sizes come from its own entry of the config, so layers may differ in everything and come in any order.
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.rg1``, ``l<i>.rg1.b``, ``l<i>.norm2``, ``l<i>.mlp.*``,
``l<i>.rg2``, ``l<i>.rg2.b``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.topezen import TopezenConfig
from ..parts.base import build_part
from ..parts.embedding import OutputHead, TokenEmbedding
from .model import ModelPlan, RunEntry


def build_topezen_plan(config: TopezenConfig) -> ModelPlan:
    width, eps = config.width, config.eps
    positions: dict = {}

    def rotation(rot: dict):
        """One table per distinct rotation (layers with the same constants read the same tables)."""
        key = (int(rot["dims"]), float(rot["base"]))
        if key not in positions:
            positions[key] = build_part("position", "rope", dim=key[0], base=key[1], precise=True)
        return positions[key]

    def norm(name: str):
        return build_part("norm", "rmsnorm_scalar", size=width, eps=eps, weight_name=name)

    layers = []
    for spec in config.layers:
        m = spec["mixer"]
        if spec["type"] == "latent_attention":
            mixer = build_part("mixer", "latent_attention", hidden_size=width, n_heads=m["heads"], head_dim=m["dim"],
                               rot_dim=m["rot_dim"], value_dim=m["vdim"], q_rank=m["q_rank"], kv_rank=m["kv_rank"], scale=m["scale"],
                               norm_eps=eps, position=rotation(m["rot"]), pairing="neighbours", gated=True)
        elif spec["type"] == "mlstm":
            mixer = build_part("mixer", "mlstm", hidden_size=width, n_heads=m["heads"], key_dim=m["dim"], value_dim=m["vdim"],
                               gate_cap=m["gate_cap"], norm_eps=eps)
        else:
            mask = m.get("mask") or {}
            mixer = build_part("mixer", "scored_attention", hidden_size=width, n_q_heads=m["heads"], n_kv_heads=m["kv_heads"],
                               key_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"], norm_eps=eps, head_norm=True,
                               softcap=m.get("softcap"), window=mask.get("size"), keep_first=mask.get("keep_first") or 0, sink="learned")
        mlp = spec.get("mlp")
        ffn = None
        if mlp is not None and mlp["kind"] == "dense":
            ffn = build_part("feed_forward", "poly_norm", hidden_size=width, intermediate_size=mlp["ff"], eps=eps)
        elif mlp is not None:
            r = mlp["router"]
            groups = r.get("groups") or {"count": 1, "keep": 1}
            ffn = build_part("feed_forward", "routed_experts", hidden_size=width, expert_size=mlp["expert"]["ff"], n_experts=r["experts"],
                             top=r["top"], n_groups=groups["count"], keep_groups=groups["keep"], scores="softmax", group_rule="best",
                             renormalise=True, shared_size=(mlp.get("shared") or {}).get("ff"))
        layers.append(build_part("block", "gated_parallel", width=width, norm_1=norm("norm1"), mixer=mixer,
                                 norm_2=norm("norm2") if ffn is not None else None, feed_forward=ffn))
    for block, follower in zip(layers, layers[1:]):
        block.next_block = follower
    return ModelPlan(
        embedding=TokenEmbedding(config.vocab, width, weight_name="embed", scale=config.embedding_scale),
        layers=layers,
        final_norm=norm("norm"),
        head=OutputHead(width, config.vocab, weight_name="head"),
        run_list=[RunEntry(i) for i in range(len(layers))],
        positions=list(positions.values()),
        embedding_prefix="",
        layer_prefix="l{}.",
        final_norm_prefix="final.",
        head_prefix="",
    )
