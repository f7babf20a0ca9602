"""The Katopel decoder put together from parts.

Token embedding times a constant; per layer a ``LayerNormBothSidesBlock`` (a layer norm with weight and bias before and after each
sublayer) around one of two mixers and a feed-forward (dense, routed experts with a gated shared one, or none); the model's last
layer norm; logits from the embedding table itself.  Some layers may run several times in a row: the run list names them once a
pass, each pass with storage of its own, and before a pass the embedding output and a vector of the pass are added to the
stream.  The mixers, by the layer's ``type``:

* ``delta``: the gated delta rule with one decay per head;
* ``parallel``: two mixers side by side on the same input, their results summed with two constants: attention within chunks of
  positions (left: biases on q, k and v, neighbouring entries rotated together on part of each head, keys and values of sizes
  of their own), and the gated delta rule (right).

Each layer's sizes come from its own entry of the config, so layers may differ in everything and come in any order.
Tensor names: ``embed``, ``loop.step``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.mlp.*``, ``l<i>.norm2b``,
``final.norm`` (every norm with its bias under ``.b``).
"""

from __future__ import annotations

from ..config.katopel import KatopelConfig
from ..parts.base import build_part
from ..parts.embedding import OutputHead, TokenEmbedding
from .model import ModelPlan, RunEntry, StepTable, looped_run_list


def build_katopel_plan(config: KatopelConfig) -> ModelPlan:
    width, eps = config.width, config.eps
    positions: dict = {}

    def rotation(rot: dict | None):
        """One table per distinct rotation (layers with the same constants read the same tables)."""
        if not rot or not rot["dims"]:
            return None
        key = (int(rot["dims"]), float(rot["base"]))
        if key not in positions:
            positions[key] = build_part("position", "rope", dim=key[0], base=key[1], precise=True)
        return positions[key]

    def norm(name: str):
        return build_part("norm", "layernorm", size=width, eps=eps, weight_name=name, bias_name=name + ".b")

    def delta_rule(m: dict):
        return build_part("mixer", "head_delta", hidden_size=width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"],
                          value_dim=m["vdim"], conv_taps=m["conv"], norm_eps=eps)

    def chunked_attention(m: dict):
        return build_part("mixer", "scored_attention", hidden_size=width, n_q_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"],
                          value_dim=m["vdim"], scale=m["scale"], norm_eps=eps, position=rotation(m.get("rot")), pairing="neighbours",
                          qkv_bias=True, chunk=(m.get("mask") or {}).get("size"))

    layers = []
    for spec in config.layers:
        m = spec["mixer"]
        if spec["type"] == "delta":
            mixer = delta_rule(m)
        else:
            left_scale, right_scale = (1.0 if m.get(key) is None else m[key] for key in ("left_scale", "right_scale"))
            mixer = build_part("mixer", "side_by_side", left=chunked_attention(m["left"]), right=delta_rule(m["right"]),
                               left_scale=left_scale, right_scale=right_scale)
        mlp = spec.get("mlp")
        ffn = None
        if mlp is not None and mlp["kind"] == "dense":
            ffn = build_part("feed_forward", "swiglu", hidden_size=width, intermediate_size=mlp["ff"], gate_name="gate", up_name="up",
                             down_name="down")
        elif mlp is not None:
            r = mlp["router"]
            ffn = build_part("feed_forward", "routed_experts", hidden_size=width, expert_size=mlp["expert"]["ff"], n_experts=r["experts"],
                             top=r["top"], logit_weights=True, bias_name=None, shared_size=(mlp.get("shared") or {}).get("ff"),
                             shared_gate=True)
        second = (norm("norm2"), norm("norm2b"))
        layers.append(build_part("block", "layernorm_both_sides", norm_1=norm("norm1"), mixer=mixer, norm_1b=norm("norm1b"),
                                 norm_2=second[0] if ffn is not None else None, feed_forward=ffn,
                                 norm_2b=second[1] if ffn is not None else None, unused=() if ffn is not None else second))
    embedding = TokenEmbedding(config.vocab, width, weight_name="embed", scale=config.embedding_scale)
    if config.loop is None:
        steps, run_list = None, [RunEntry(i) for i in range(len(layers))]
    else:
        start, stop, times = (int(config.loop[key]) for key in ("start", "stop", "times"))
        steps, run_list = StepTable(times, width), looped_run_list(len(layers), start, stop, times, steps=True)
    return ModelPlan(
        embedding=embedding,
        layers=layers,
        final_norm=norm("norm"),
        head=OutputHead(width, config.vocab, tied_to=embedding, weight_name="head"),
        run_list=run_list,
        positions=list(positions.values()),
        embedding_prefix="",
        layer_prefix="l{}.",
        final_norm_prefix="final.",
        head_prefix="",
        steps=steps,
    )
