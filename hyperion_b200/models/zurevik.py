"""Zurevik expressed as parts: a decoder whose two sublayers read the same stream through a norm each and are added to it together, whose
attention knows no positions but its windows, and whose feed-forwards are experts.

Every layer is the arrangement of side-by-side sublayers with norms of their own (h <- h + (mixer(norm1(h)) + ff(norm2(h)))).  Mixers:
differential attention inside a window beside which the first tokens stay visible (``differential_attention``), and windowed attention with
biases, a sink in the softmax and a gate per head (``sink_attention``), whose keys and values may be an earlier layer's: such a layer is a schedule
entry that reads the lender's cache, which keeps the widest window of those that read it.  Feed-forwards: squared-ReLU experts weighed by a
softmax over the chosen (``chosen_softmax_experts``), or none.  The embedding row is multiplied by ``embedding.scale``, the head has a matrix of its
own, and the logits pass a smooth cap.  Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
The design states no limit on positions; the engine's own limit of 2^30 stands in.
"""
from __future__ import annotations

from ..config.zurevik import ARCHITECTURE, ZurevikConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, Run
from .registry import Architecture, register_architecture

NO_POSITION_LIMIT = 1 << 30


def build_spec(config: ZurevikConfig) -> ModelSpec:
    width, eps = config.width, config.eps
    layers, schedule, tolerated = [], [], []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        m = layer.mixer
        sizes = {"hidden_size": width, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale, "window": m.window}
        lender = None
        if layer.type == "attention":
            mixer = PartSpec("differential_attention", prefix + "mix.", {**sizes, "diff": m.diff, "keep_first": m.keep_first, "eps": eps})
        else:
            lender = m.kv_from
            mixer = PartSpec("sink_attention", prefix + "mix.", {**sizes, "bias": True, "sink": True, "head_gate": True, "shares_kv": lender is not None,
                                                                "cache_window": config.cache_window(index if lender is None else lender)})
        norms = {"input": PartSpec("rmsnorm", prefix, {"hidden_size": width, "eps": eps, "weight_name": "norm1"})}
        feed_forward = None
        if layer.mlp is None:  # a checkpoint may carry the feed-forward's norm all the same; nothing reads it
            tolerated.append(prefix + "norm2")
        else:
            norms["feed_forward_in"] = PartSpec("rmsnorm", prefix, {"hidden_size": width, "eps": eps, "weight_name": "norm2"})
            feed_forward = PartSpec("chosen_softmax_experts", prefix + "mlp.", {"hidden_size": width, "experts": layer.mlp.experts, "top": layer.mlp.top,
                                                                                "expert_size": layer.mlp.ff, "activation": "relu_squared"})
        layers.append(LayerSpec(arrangement="side_by_side_two_norms", mixer=mixer, feed_forward=feed_forward, norms=norms))
        schedule.append(Run(index, reads_cache_of=lender))
    sizes = {"vocab_size": config.vocab, "hidden_size": width}
    return ModelSpec(
        architecture=ARCHITECTURE,
        hidden_size=width,
        vocab_size=config.vocab,
        max_positions=NO_POSITION_LIMIT,
        embedding=PartSpec("token_embedding", "", {**sizes, "weight_name": "embed", "scale": config.embedding_scale}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=PartSpec("rmsnorm", "final.", {"hidden_size": width, "eps": eps, "weight_name": "norm"}),
        head=PartSpec("linear_head", "", {**sizes, "weight_name": "head", "softcap": config.logit_softcap}),
        tolerated=tuple(tolerated),
    )


register_architecture(Architecture(ARCHITECTURE, ZurevikConfig.from_dict, build_spec, ZurevikConfig.to_dict))
