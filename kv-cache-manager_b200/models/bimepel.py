"""Bimepel assembled from parts (registered as ``Bimepel``).

Every layer is a "parallel_norms" block, x += mixer(shift(norm1(x))) + ffn(norm2(x)), whose mixer reads each row mixed with
the row before it (token shift, per-request state in every layer).  The mixer is, by the layer's ``type``,

* "attention": grouped-query attention with weighted per-head norms of q and k ahead of the rotation, rotate-half rotary
  encoding (partial; YaRN-scaled), values divided by their root mean square, a chunked mask and an element-wise output
  gate (``attention_general``);
* "lightning": lightning attention, a linear recurrence with one constant decay per head (``lightning``);

the feed-forward is absent, dense (the clamped gated activation) or routed experts (sigmoid scores, the chosen scores
normalised to a sum of one before the scale).  A span of layers may run several times in a row with the same weights:
every pass is a run-order entry of its own (own pages, own state).  Final norm; the output head is the token table.

Checkpoint names: ``embed``, ``l<i>.norm1|norm2|shift``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``; linear weights
[out, in].  Fused at load: q|k|v|g of either mixer, gate|up of a dense feed-forward, the experts' matrices stacked.
"""
from __future__ import annotations

from ..config.model_config import BimepelConfig
from ..config.registry import register_architecture
from ..parts.base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, LayerCall
from ..parts.embedding import Embedding, LMHead
from .spec import ModelSpec, TensorBinding

GATE_ALPHA = 1.702            # the dense feed-forward's gate: g * sigmoid(GATE_ALPHA * g)


def build_bimepel(cfg: BimepelConfig, norm_init=("ones_jitter", 0.1)) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    embedding = Embedding(cfg.vocab, D)
    embed = TensorBinding(embedding, "weight", [("embed", (cfg.vocab, D))])
    bindings = [embed]
    blocks, ignorable = [], []

    def norm(name: str):
        part = NORMS.build("rmsnorm_f32", hidden=D, eps=eps, init=norm_init)
        bindings.append(TensorBinding(part, "weight", [(name, (D,))]))
        return part

    for i, layer in enumerate(cfg.layers):
        m, p = layer["mixer"], f"l{i}.mix."
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G, rot = m["kv_heads"], m.get("rot")
            position = (POSITION_ENCODINGS.build("rope", head_dim=dk, theta=rot["base"], rotary_dim=rot["dims"], pairing="half",
                                                 scaling=rot.get("scaling"))
                        if rot else POSITION_ENCODINGS.build("none"))
            mixer = MIXERS.build("attention_general", hidden=D, num_heads=H, num_kv_heads=G, dk=dk, dv=dv, position=position,
                                 scale=m["scale"], norm_eps=eps, qk_norm=True, value_norm=True, gate=True,
                                 chunk=(m.get("mask") or {}).get("size", 0))
            bindings += [TensorBinding(mixer.qkv, "weight", [(p + "q", (H * dk, D)), (p + "k", (G * dk, D)), (p + "v", (G * dv, D)),
                                                             (p + "g", (H * dv, D))]),
                         TensorBinding(mixer, "q_head_norm", [(p + "q.norm", (dk,))]),
                         TensorBinding(mixer, "k_head_norm", [(p + "k.norm", (dk,))])]
        else:                                             # "lightning" (the config has been validated)
            mixer = MIXERS.build("lightning", hidden=D, heads=H, dk=dk, dv=dv, decay=m["decay"], norm_eps=eps)
            bindings += [TensorBinding(mixer.qkvg, "weight", [(p + "q", (H * dk, D)), (p + "k", (H * dk, D)), (p + "v", (H * dv, D)),
                                                              (p + "g", (H * dv, D))]),
                         TensorBinding(mixer, "norm", [(p + "norm", (H * dv,))])]
        bindings.append(TensorBinding(mixer.o, "weight", [(p + "o", (D, H * dv))]))
        norm1 = norm(f"l{i}.norm1")
        norm2 = ffn = None
        mlp = layer.get("mlp")
        if mlp is None:                                   # a checkpoint may still carry the unused norm
            ignorable.append(f"l{i}.norm2")
        else:
            q = f"l{i}.mlp."
            if mlp["kind"] == "dense":
                F = mlp["ff"]
                ffn = FEED_FORWARDS.build("gated_mlp", hidden=D, intermediate=F, activation="clamped", limit=mlp["limit"], alpha=GATE_ALPHA)
                bindings += [TensorBinding(ffn.gate_up, "weight", [(q + "gate", (F, D)), (q + "up", (F, D))]),
                             TensorBinding(ffn.down, "weight", [(q + "down", (D, F))])]
            else:
                r, F = mlp["router"], mlp["expert"]["ff"]
                E = r["experts"]
                ffn = FEED_FORWARDS.build("routed_experts", hidden=D, experts=E, expert_ff=F, top=r["top"], scale=r.get("scale", 1.0),
                                          scores="sigmoid", renorm=True)
                bindings += [TensorBinding(ffn, "router", [(q + "router", (E, D))]),
                             TensorBinding(ffn, "gate_up", [(f"{q}e{e}.{n}", (F, D)) for e in range(E) for n in ("gate", "up")]),
                             TensorBinding(ffn, "down", [(f"{q}e{e}.down", (D, F)) for e in range(E)])]
            norm2 = norm(f"l{i}.norm2")
        block = BLOCKS.build("parallel_norms", norm1=norm1, mixer=mixer, norm2=norm2, ffn=ffn, token_shift=True)
        bindings.append(TensorBinding(block, "shift", [(f"l{i}.shift", (D,))]))
        blocks.append(block)
    n = len(cfg.layers)
    span = range(cfg.loop_start, cfg.loop_stop)
    order = [LayerCall(i) for i in (*range(cfg.loop_start), *(list(span) * cfg.loop_times), *range(cfg.loop_stop, n))]
    final_norm = norm("final.norm")
    head = LMHead(D, cfg.vocab)
    bindings.append(TensorBinding(head, "weight", [("head", (cfg.vocab, D))], tie_to=embed, tied=True))
    return ModelSpec(cfg, embedding, blocks, order, final_norm, head, bindings, ignorable=tuple(ignorable))


register_architecture("Bimepel", BimepelConfig, build_bimepel, replace=True)
