"""Several residual streams, and how a sublayer reads from and writes to them (hyper-connections).

Instead of one row x per token a model may carry ``streams`` of them, x_0 .. x_(S-1), all equal to the embedding row at the start.  A sublayer's connection
holds three small tensors: ``in`` [S], ``out`` [S] and ``mix`` [S, S] (indexed from, to):
    u = sum_s in[s] x_s;   y = sublayer(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y   for all t at once, from the old streams
and the model's last norm reads the sum of the streams.  The streams are float, [tokens, S, hidden]; until the first write one row per
token stands for all of them.  Everything between a sublayer's last product and the next one's first is one launch (``ops.hyper_connect``).

``hyper_connection``: parameters ``hidden_size``, ``streams``.  Tensors: in, out, mix.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .. import ops
from ..ops.basic import LARGEST_STREAMS
from .base import BuildContext, Connection, WeightSpec, register_connection
from .norm import NormedSum, StreamDelta
from .spec import PartSpec


class HyperConnection(Connection):
    def __init__(self, spec: PartSpec, build: BuildContext):
        super().__init__(spec, build)
        self.hidden, self.streams = int(spec.params["hidden_size"]), int(spec.params["streams"])
        if not 1 <= self.streams <= LARGEST_STREAMS:
            raise ValueError(f"{self.streams} residual streams: 1 to {LARGEST_STREAMS} are supported")

    def weights(self) -> dict[str, WeightSpec]:
        # random weights: a sublayer reads and passes on the streams' mean, and its result joins all of them
        s = self.streams
        return {"in": WeightSpec((s,), mean=1.0 / s), "out": WeightSpec((s,), mean=1.0), "mix": WeightSpec((s, s), mean=1.0 / s)}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.w_read, self.share, self.mix = (tensors[name].to(torch.float32).contiguous() for name in ("in", "out", "mix"))

    def kernel_modules(self):
        return [ops.streams_module(self.streams)]

    @staticmethod
    def _pending(delta) -> dict:
        """What ``delta`` has to write, as arguments of ``ops.hyper_connect``."""
        if delta is None:
            return {}
        if not isinstance(delta, StreamDelta):
            raise ValueError("a layer with several residual streams stands behind one without")
        written, y = delta.connection, delta.y
        if isinstance(y, NormedSum):
            norms = tuple(y.weights) + (None,) * (2 - len(y.weights))
            return {"results": y.results, "norms": norms, "result_eps": y.eps, "result_scale": y.scale, "mix": written.mix, "share": written.share}
        if hasattr(y, "tensor") and not hasattr(y, "partials"):
            y = y.tensor()
        return {"results": (y,), "mix": written.mix, "share": written.share}

    def read(self, h, pending, norm):
        return ops.hyper_connect(h, self.streams, self.w_read, norm.weight, norm.eps, norm.dtype, **self._pending(pending))

    def read_sum(self, h, pending, norm, rows):
        """The norm behind the last layer: of the sum of the streams, of the listed rows only; the streams themselves are not written."""
        every = rows if rows is not None else torch.arange(h.shape[0], dtype=torch.int32, device=h.device)
        return ops.hyper_connect(h, self.streams, None, norm.weight, norm.eps, norm.dtype, rows=every, **self._pending(pending))[0]


register_connection("hyper_connection", HyperConnection)
