"""Windowed grouped-query attention with a sink in the softmax and a gate per head, over keys and values of its own or of another entry of
the schedule.

    q, k, v = W_q x + b_q, W_k x + b_k, W_v x + b_v;   weights over the seen keys: exp(s_j) / (sum_j exp(s_j) + exp(sink_h)), s = (q . k) * scale
    y = W_o [head h's result times sigmoid(W_g x)_h, heads side by side]

Position p sees the positions j with 0 <= p - j < ``window`` (0: every earlier one); nothing is rotated.  Query head h reads key/value head
h // (heads / kv_heads).  With ``shares_kv`` the part has no key and value projections and reads the cache of the schedule entry its own
entry names, with queries, window, sink and gate of its own.  The cache keeps ``cache_window`` positions (the widest window that reads
it; 0: all), which is the part's own window unless stated.

Per step: one product to [q | k | v | gate] (or [q | gate]) kept in float; one kernel that adds the biases and stores (``ops.heads_store``);
attention, which takes window, sink and gate as arguments; the output product.  In bfloat16, with keys and values of one size that is a multiple
of 16 up to 256, the tensor-core kernels of the package's other attentions run (tcgen05 tiles for prompt portions of heads of 64 and 128, split
keys for decoded tokens); everything else, and float32, runs in ``csrc/attention_generic.cu``.  Scores, sink, softmax and gate are float.

Parameters: ``hidden_size``, ``heads``, ``kv_heads``, ``head_dim``, ``value_dim`` (``head_dim`` unless stated), ``scale``, ``window``, ``cache_window``,
``bias`` (bool), ``sink`` (bool), ``head_gate`` (bool), ``shares_kv`` (bool).  Tensors: q, k, v (a bias is its matrix's name with ``.b`` added), sink, g, o.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .. import ops
from ..ops import attention as fast_attention
from .attention import GroupedQueryAttention
from .base import BuildContext, Mixer, PagedKV, PagedTokens, WeightSpec, register_mixer
from .spec import PartSpec

LARGEST_HEAD = 640  # csrc/attention_generic.cu


def _common_dtype(tensors) -> torch.dtype:
    return torch.float32 if any(t.dtype == torch.float32 for t in tensors) else tensors[0].dtype


class SinkAttention(GroupedQueryAttention):
    """Shares the planning and the launches of the tensor-core path with its base; everything else is its own."""

    def __init__(self, spec: PartSpec, build: BuildContext):
        Mixer.__init__(self, spec, build)
        p = spec.params
        self.hidden, self.heads, self.kv_heads = int(p["hidden_size"]), int(p["heads"]), int(p["kv_heads"])
        self.head_dim = int(p["head_dim"])
        self.value_dim = int(p.get("value_dim") or self.head_dim)
        self.scale = float(p.get("scale", self.head_dim ** -0.5))
        self.window, self.softcap = int(p.get("window") or 0), 0.0
        self.cache_window = int(p["cache_window"]) if p.get("cache_window") is not None else self.window
        self.bias, self.has_sink, self.has_gate = bool(p.get("bias", False)), bool(p.get("sink", False)), bool(p.get("head_gate", False))
        self.shares_kv = bool(p.get("shares_kv", False))
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.kv_heads} key/value heads do not divide {self.heads} heads")
        if max(self.head_dim, self.value_dim) > LARGEST_HEAD:
            raise ValueError(f"heads of {self.head_dim} / {self.value_dim} are above the kernel's limit of {LARGEST_HEAD}")
        if self.cache_window and (not self.window or self.window > self.cache_window):
            raise ValueError(f"a cache of {self.cache_window} positions is narrower than the window of {self.window or 'all'} that reads it")
        self.q_width, self.k_width = self.heads * self.head_dim, self.kv_heads * self.head_dim
        self.v_width, self.core_width = self.kv_heads * self.value_dim, self.heads * self.value_dim
        self.fast = self.dtype == torch.bfloat16 and self.value_dim == self.head_dim and fast_attention.supported(self.head_dim) and self.scale > 0

    @property
    def _projected(self) -> tuple[tuple[str, int], ...]:
        own = () if self.shares_kv else (("k", self.k_width), ("v", self.v_width))
        return (("q", self.q_width), *own)

    def weights(self) -> dict[str, WeightSpec]:
        wanted = {name: WeightSpec((width, self.hidden)) for name, width in self._projected}
        if self.bias:
            wanted.update({name + ".b": WeightSpec((width,)) for name, width in self._projected})
        if self.has_sink:
            wanted["sink"] = WeightSpec((self.heads,))
        if self.has_gate:
            wanted["g"] = WeightSpec((self.heads, self.hidden))
        wanted["o"] = WeightSpec((self.hidden, self.core_width))
        return wanted

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        mats = [tensors[name] for name, _ in self._projected]
        if self.has_gate:  # the gate's rows, padded so that the product's rows stay whole 16-byte pieces
            rows = -(-self.heads // 8) * 8
            gate = torch.zeros((rows, self.hidden), dtype=tensors["g"].dtype, device=tensors["g"].device)
            gate[: self.heads] = tensors["g"]
            mats.append(gate)
        dtype = _common_dtype(mats)
        self.w_in = torch.cat([m.to(dtype) for m in mats], dim=0).contiguous()
        self.b_in = torch.cat([tensors[name + ".b"].to(torch.float32) for name, _ in self._projected], dim=0).contiguous() if self.bias else None
        self.w_o = tensors["o"].contiguous()
        self.sink = tensors["sink"].to(torch.float32).contiguous() if self.has_sink else None

    def cache_request(self):
        if self.shares_kv:
            return None
        if self.value_dim == self.head_dim:
            return PagedKV(self.kv_heads, self.head_dim, self.cache_window)
        return PagedTokens((self.kv_heads,), (self.head_dim + self.value_dim,), self.cache_window)

    def kernel_modules(self):
        modules = [("heads_prepare", {}), ("sgemm_f32", {}) if self.dtype == torch.float32 else ("gemm_tcgen05", {})]
        if not self.fast:
            return modules + [("attention_generic", {})]
        if self.head_dim % 64 == 0:
            modules.append(("attention_tma", {"HB_HEAD_DIM": self.head_dim}))
        else:
            modules.append(("attention_bf16", {"HB_HEAD_DIM": self.head_dim}))
        if self.head_dim in (64, 128):
            modules.append(("attention_tcgen05", {"HB_HEAD_DIM": self.head_dim}))
        return modules

    def forward(self, x, step, cache, own_cache):
        if cache is None or own_cache == self.shares_kv:
            raise ValueError("this attention writes a cache of its own or reads the one its schedule entry names; the schedule gave it another")
        proj = ops.linear(x, self.w_in, None, torch.float32)
        k_off = self.q_width
        v_off = k_off + self.k_width
        q = torch.empty((x.shape[0], self.q_width), dtype=self.dtype, device=x.device)
        where = {} if self.shares_kv else {"cache": cache.kv, "block_table": cache.block_table, "token_row": step.token_row, "page_size": cache.page_size}
        ops.heads_store(proj, 0, k_off, v_off, self.heads, self.kv_heads, self.head_dim, self.value_dim, step.positions, q_out=q, bias=self.b_in, **where)
        gate = proj[:, sum(width for _, width in self._projected):][:, : self.heads] if self.has_gate else None
        if self.fast:
            attn = self._attend_fast(q, step, cache, sinks=self.sink, gate=gate)
        else:
            attn = ops.attention_general(q, self.heads, self.kv_heads, self.head_dim, self.value_dim, cache.kv, cache.block_table, step.token_row, step.positions,
                                         cache.page_size, self.scale, 0.0, self.window, sinks=self.sink, gate=gate, gate_per_head=True)
        return ops.linear(attn, self.w_o, None, self.dtype, may_leave_partials=True)  # the result is a residual delta


register_mixer("sink_attention", SinkAttention)
