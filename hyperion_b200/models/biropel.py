"""Biropel expressed as parts: a decoder with several residual streams, whose mixers are attention alone or attention beside a recurrence.

Every layer is the arrangement of sublayers connected to the streams (``hyper_connected``: a sublayer reads one mixture of the streams through its norm and writes
to all of them; a connection per sublayer).  Mixers: windowed attention with biases, a rotation of part of every head and a gate per entry of its result
(``composed_attention``), over keys and values of its own or of an earlier layer (a schedule entry that reads the lender's cache, which keeps the widest window of those
that read it); and two mixers side by side whose results are normed before they are averaged (``parallel_normed_mixers``): windowed attention with a rotation
stretched to long texts and capped scores beside the state-space mixer of Mamba-2 (``mamba2``), or attention over every earlier key with unit-norm queries and
keys, a temperature by position and capped scores beside the matrix memory of xLSTM (``matrix_memory``).  Feed-forward: one without a gate, the square of relu, or
none.  The streams start as the normalised embedding row; the last norm reads their sum; the head has a matrix of its own.  Tensor names: ``embed``,
``embed.norm``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.*``, ``l<i>.hc2.*``, ``l<i>.mix.*`` (``l<i>.mix.left.*``, ``l<i>.mix.right.*``), ``l<i>.mlp.up``, ``l<i>.mlp.down``,
``final.norm``, ``head``.  The design states no limit on positions; the engine's own limit of 2^30 stands in.
"""
from __future__ import annotations

from ..config.biropel import ARCHITECTURE, AttentionSizes, BiropelConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, Run
from .registry import Architecture, register_architecture

NO_POSITION_LIMIT = 1 << 30


def _position(m: AttentionSizes) -> PartSpec | None:
    if m.rot is None or not m.rot.dims:
        return None
    if m.rot.scaling is None:
        return PartSpec("rope_half_partial", "", {"dims": m.rot.dims, "base": m.rot.base})
    s = m.rot.scaling
    return PartSpec("rope_half_slowed", "", {"dims": m.rot.dims, "base": m.rot.base, "factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow})


def build_spec(config: BiropelConfig) -> ModelSpec:
    width, eps = config.width, config.eps
    layers, schedule, tolerated = [], [], []

    def attention(prefix: str, m: AttentionSizes, **options) -> PartSpec:
        return PartSpec("composed_attention", prefix, {
            "hidden_size": width, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale, "softcap": m.softcap,
            "window": m.window, "position": _position(m), "temperature": (m.q_temp.coef, m.q_temp.every) if m.q_temp is not None else None, "eps": eps, **options})

    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        m = layer.mixer
        lender = None
        if layer.type == "attention":
            lender = m.kv_from
            mixer = attention(prefix + "mix.", m, bias=True, gate=True, shares_kv=lender is not None, cache_window=config.cache_window(index if lender is None else lender))
        else:
            r = m.right
            if layer.type == "parallel":
                right = PartSpec("mamba2", "right.", {"hidden_size": width, "heads": r.heads, "value_dim": r.vdim, "state": r.state, "groups": r.groups,
                                                      "norm_groups": r.norm_groups, "conv": r.conv, "eps": eps})
            else:
                right = PartSpec("matrix_memory", "right.", {"hidden_size": width, "heads": r.heads, "head_dim": r.dim, "value_dim": r.vdim, "gate_cap": r.gate_cap, "eps": eps})
            left = attention("left.", m.left, unit_norm=layer.type == "parallel_2")
            mixer = PartSpec("parallel_normed_mixers", prefix + "mix.", {"hidden_size": width, "branches": ((left, "left.out"), (right, "right.out")), "eps": eps, "scale": 0.5})

        def norm(name: str) -> PartSpec:
            return PartSpec("rmsnorm", prefix, {"hidden_size": width, "eps": eps, "weight_name": name})

        def connection(name: str) -> PartSpec:
            return PartSpec("hyper_connection", f"{prefix}{name}.", {"hidden_size": width, "streams": config.streams})

        norms, connections = {"input": norm("norm1")}, {"mixer": connection("hc1")}
        feed_forward = None
        if layer.ff is None:  # a checkpoint may carry the feed-forward's norm and connection all the same; nothing reads them
            tolerated += [prefix + name for name in ("norm2", "hc2.in", "hc2.out", "hc2.mix")]
        else:
            norms["post_mixer"], connections["feed_forward"] = norm("norm2"), connection("hc2")
            feed_forward = PartSpec("activated_mlp", prefix + "mlp.", {"hidden_size": width, "intermediate_size": layer.ff, "activation": "relu_squared",
                                                                       "names": {"up": "up", "down": "down"}})
        layers.append(LayerSpec(arrangement="hyper_connected", mixer=mixer, feed_forward=feed_forward, norms=norms, connections=connections))
        schedule.append(Run(index, reads_cache_of=lender))
    sizes = {"vocab_size": config.vocab, "hidden_size": width}
    return ModelSpec(
        architecture=ARCHITECTURE,
        hidden_size=width,
        vocab_size=config.vocab,
        max_positions=NO_POSITION_LIMIT,
        embedding=PartSpec("token_embedding", "", {**sizes, "weight_name": "embed", "norm_weight_name": "embed.norm", "eps": eps}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=PartSpec("rmsnorm", "final.", {"hidden_size": width, "eps": eps, "weight_name": "norm"}),
        head=PartSpec("linear_head", "", {**sizes, "weight_name": "head"}),
        tolerated=tuple(tolerated),
    )


register_architecture(Architecture(ARCHITECTURE, BiropelConfig.from_dict, build_spec, BiropelConfig.to_dict))
