"""Pemorax assembled from parts (registered as ``Pemorax``).

Every layer is a "sandwich" block with plain RMS norms, x += norm_b(sublayer(norm(x))) for the mixer and, where the layer has
one, for the feed-forward.  The mixer ("parallel") is two mixers side by side that read the same rows, each result
divided by its root mean square and multiplied by a weight of its own, half of their sum being the mixer's result
(``side_by_side`` with ``out_norm``):

* left, grouped-query attention (``attention_general``): short convolutions of q, k and v over time, rotary encoding in
  interleaved pairs (partial; YaRN-scaled), capped scores, a sliding window that keeps a request's first tokens, one added
  to the softmax's denominator, an element-wise output gate;
* right, ``retention``: linear attention with a fixed decay per head, rotate-half rotary encoding, normalised heads and a
  SiLU gate;

the feed-forward is absent, dense with the tanh form of gelu, or routed experts (biased logits, the softmax over the
chosen ones as weights).  Final norm, output head.

Checkpoint names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.left.*``, ``l<i>.mix.right.*`` (``.out``: the weight
of a branch's norm), ``l<i>.mlp.*``, ``final.norm``, ``head``; linear weights [out, in].  Fused at load: q|k|v|g of either
mixer (and the two of a layer to one product), the three convolutions, the experts' matrices stacked.
"""
from __future__ import annotations

from ..config.model_config import PemoraxConfig
from ..config.registry import register_architecture
from ..parts.base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, LayerCall
from ..parts.embedding import Embedding, LMHead
from .spec import ModelSpec, TensorBinding


def _position(m: dict, pairing: str):
    rot = m.get("rot")
    if not rot:
        return POSITION_ENCODINGS.build("none")
    return POSITION_ENCODINGS.build("rope", head_dim=m["dim"], theta=rot["base"], rotary_dim=rot["dims"], pairing=pairing,
                                    scaling=rot.get("scaling"))


def build_pemorax(cfg: PemoraxConfig, norm_init=("ones_jitter", 0.1)) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    embedding = Embedding(cfg.vocab, D)
    bindings = [TensorBinding(embedding, "weight", [("embed", (cfg.vocab, D))])]
    blocks, ignorable = [], []

    def norm(name: str):
        part = NORMS.build("rmsnorm_f32", hidden=D, eps=eps, init=norm_init)
        bindings.append(TensorBinding(part, "weight", [(name, (D,))]))
        return part

    for i, layer in enumerate(cfg.layers):
        lm, rm, p = layer["mixer"]["left"], layer["mixer"]["right"], f"l{i}.mix."
        H, G, dk, dv, taps = lm["heads"], lm["kv_heads"], lm["dim"], lm["vdim"], lm.get("conv") or 0
        mask = lm.get("mask") or {}
        left = MIXERS.build("attention_general", hidden=D, num_heads=H, num_kv_heads=G, dk=dk, dv=dv, position=_position(lm, "interleaved"),
                            scale=lm["scale"], window=mask.get("size", 0), keep_first=mask.get("keep_first") or 0,
                            softcap=lm.get("softcap") or 0.0, sink_score=0.0, norm_eps=eps, gate=True, taps=taps)
        q = p + "left."
        bindings += [TensorBinding(left.qkv, "weight", [(q + "q", (H * dk, D)), (q + "k", (G * dk, D)), (q + "v", (G * dv, D)),
                                                        (q + "g", (H * dv, D))]),
                     TensorBinding(left.o, "weight", [(q + "o", (D, H * dv))])]
        if taps:
            bindings.append(TensorBinding(left, "conv", [(q + "q.conv", (H * dk, taps)), (q + "k.conv", (G * dk, taps)),
                                                         (q + "v.conv", (G * dv, taps))]))
        H, dk, dv = rm["heads"], rm["dim"], rm["vdim"]
        right = MIXERS.build("retention", hidden=D, heads=H, dk=dk, dv=dv, decay=rm["decay"], position=_position(rm, "half"), norm_eps=eps)
        q = p + "right."
        bindings += [TensorBinding(right.qkvg, "weight", [(q + "q", (H * dk, D)), (q + "k", (H * dk, D)), (q + "v", (H * dv, D)),
                                                          (q + "g", (H * dv, D))]),
                     TensorBinding(right.o, "weight", [(q + "o", (D, H * dv))])]
        mixer = MIXERS.build("side_by_side", left=left, right=right, left_scale=0.5, right_scale=0.5, out_norm=True, hidden=D,
                             norm_eps=eps, init=norm_init)
        bindings += [TensorBinding(mixer, "left_out", [(p + "left.out", (D,))]), TensorBinding(mixer, "right_out", [(p + "right.out", (D,))])]
        norm1, norm1b = norm(f"l{i}.norm1"), norm(f"l{i}.norm1b")
        norm2 = norm2b = ffn = None
        mlp = layer.get("mlp")
        if mlp is None:                                   # a checkpoint may still carry the unused norms
            ignorable.append(f"l{i}.norm2")
        else:
            q = f"l{i}.mlp."
            if mlp["kind"] == "dense":
                F = mlp["ff"]
                ffn = FEED_FORWARDS.build("dense_mlp", hidden=D, intermediate=F, activation="gelu_tanh")
                bindings += [TensorBinding(ffn.up, "weight", [(q + "up", (F, D))]), TensorBinding(ffn.down, "weight", [(q + "down", (D, F))])]
            else:
                E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
                ffn = FEED_FORWARDS.build("routed_experts", hidden=D, experts=E, expert_ff=F, top=mlp["router"]["top"],
                                          scores="softmax_chosen", router_bias=True)
                bindings += [TensorBinding(ffn, "router", [(q + "router", (E, D))]), TensorBinding(ffn, "router_bias", [(q + "router.b", (E,))]),
                             TensorBinding(ffn, "gate_up", [(f"{q}e{e}.{n}", (F, D)) for e in range(E) for n in ("gate", "up")]),
                             TensorBinding(ffn, "down", [(f"{q}e{e}.down", (D, F)) for e in range(E)])]
            norm2, norm2b = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b")
        blocks.append(BLOCKS.build("sandwich", norm1=norm1, mixer=mixer, norm1b=norm1b, norm2=norm2, ffn=ffn, norm2b=norm2b))
    final_norm = norm("final.norm")
    head = LMHead(D, cfg.vocab)
    bindings.append(TensorBinding(head, "weight", [("head", (cfg.vocab, D))]))
    return ModelSpec(cfg, embedding, blocks, [LayerCall(i) for i in range(len(blocks))], final_norm, head, bindings, ignorable=tuple(ignorable))


register_architecture("Pemorax", PemoraxConfig, build_pemorax, replace=True)
