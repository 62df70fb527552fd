"""Grouped-query attention put together from steps that are each an option: biases, a unit norm of queries and keys, a rotation, a temperature on the queries,
a cap on the scores, a sliding window, a gate per entry of the result, and keys and values of its own or of another entry of the schedule.

    q, k, v = W_q x (+ b_q), W_k x (+ b_k), W_v x (+ b_v)
    q, k <- q / sqrt(mean(q^2) + eps) per head (``unit_norm``), turned by their position (``position``)
    q    <- q * (1 + coef * ln(floor((p + 1) / every) + 1))                                     (``temperature``)
    s    =  (q . k) * scale, then cap * tanh(s / cap) (``softcap``), over the positions j with 0 <= p - j < window (0: every earlier one)
    y    =  W_o [softmax(s) v, heads side by side] * sigmoid(W_g x)                             (``gate``)

Query head h reads key/value head h // (heads / kv_heads).  The part is a branch (``parts/branch.py``): it also runs beside another mixer on the same input.
With ``shares_kv`` it has no key and value projections and reads the cache of the schedule entry its own entry names, with everything else of its own.  The cache
keeps ``cache_window`` positions (the widest window that reads it; 0: all), which is the part's own window unless stated.

Per step: one product to [q | k | v | gate] kept in float; one kernel that adds the biases, norms, turns and stores (``ops.heads_store``); attention;
the gate; the output product.  In bfloat16, with keys and values of one size that is a multiple of 16 up to 256, the tensor-core kernels of
the package's other attentions run (tcgen05 tiles for prompt portions of heads of 64 and 128, split keys for decoded tokens); everything else, and
float32, runs in ``csrc/attention_generic.cu``, which applies the gate itself.  Norms, angles, temperature, scores, cap, softmax and gate are float.

Parameters: ``hidden_size``, ``heads``, ``kv_heads``, ``head_dim``, ``value_dim`` (``head_dim`` unless stated), ``scale``, ``softcap`` (0 = none), ``window``,
``cache_window``, ``bias`` (bool: on q, k and v), ``unit_norm`` (bool), ``eps``, ``position`` (a PartSpec or None), ``temperature`` ((coef, every) or None), ``gate``
(bool), ``shares_kv`` (bool).  Tensors: q, k, v (a bias is its matrix's name with ``.b`` added), g, o.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .. import ops
from ..ops import attention as fast_attention
from .attention import GroupedQueryAttention
from .base import POSITIONS, BuildContext, PagedKV, PagedTokens, WeightSpec, make, register_mixer
from .branch import Branch
from .spec import PartSpec

LARGEST_HEAD = 640  # csrc/attention_generic.cu


class ComposedAttention(Branch):
    out_name = "o"

    def __init__(self, spec: PartSpec, build: BuildContext):
        super().__init__(spec, build)
        p = spec.params
        self.hidden, self.heads, self.kv_heads = int(p["hidden_size"]), int(p["heads"]), int(p["kv_heads"])
        self.head_dim = int(p["head_dim"])
        self.value_dim = int(p.get("value_dim") or self.head_dim)
        self.scale, self.softcap = float(p.get("scale", self.head_dim ** -0.5)), float(p.get("softcap") or 0.0)
        self.window = int(p.get("window") or 0)
        self.cache_window = int(p["cache_window"]) if p.get("cache_window") is not None else self.window
        self.bias, self.gated, self.shares_kv = bool(p.get("bias", False)), bool(p.get("gate", False)), bool(p.get("shares_kv", False))
        self.unit_norm, self.eps = bool(p.get("unit_norm", False)), float(p.get("eps", 0.0))
        self.temperature = (float(p["temperature"][0]), int(p["temperature"][1])) if p.get("temperature") is not None else None
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.kv_heads} key/value heads do not divide {self.heads} heads")
        if max(self.head_dim, self.value_dim) > LARGEST_HEAD:
            raise ValueError(f"heads of {self.head_dim} / {self.value_dim} are above the kernel's limit of {LARGEST_HEAD}")
        if self.cache_window and (not self.window or self.window > self.cache_window):
            raise ValueError(f"a cache of {self.cache_window} positions is narrower than the window of {self.window or 'all'} that reads it")
        if self.temperature is not None and self.temperature[1] < 1:
            raise ValueError(f"a temperature that grows every {self.temperature[1]} positions")
        self.position = make(POSITIONS, p["position"], build) if p.get("position") is not None else None
        if self.position is not None and not hasattr(self.position, "inv_freq"):
            raise ValueError("this attention's rotation takes frequencies: 'rope_half_partial', 'rope_half_slowed' or 'rope_interleaved'")
        if self.position is not None and self.position.dims > self.head_dim:
            raise ValueError(f"a rotation of {self.position.dims} entries in heads of {self.head_dim}")
        self.q_width, self.k_width = self.heads * self.head_dim, self.kv_heads * self.head_dim
        self.v_width, self.core_width = self.kv_heads * self.value_dim, self.heads * self.value_dim
        self.projected = (("q", self.q_width),) + (() if self.shares_kv else (("k", self.k_width), ("v", self.v_width)))
        self.in_names = tuple(name for name, _ in self.projected) + (("g",) if self.gated else ())
        self.gate_off = sum(width for _, width in self.projected)
        self.in_width = self.gate_off + (self.core_width if self.gated else 0)
        self.fast = self.dtype == torch.bfloat16 and self.value_dim == self.head_dim and fast_attention.supported(self.head_dim) and self.scale > 0

    def weights(self) -> dict[str, WeightSpec]:
        wanted = {name: WeightSpec((width, self.hidden)) for name, width in self.projected}
        if self.bias:
            wanted.update({name + ".b": WeightSpec((width,)) for name, width in self.projected})
        if self.gated:
            wanted["g"] = WeightSpec((self.core_width, self.hidden))
        wanted["o"] = WeightSpec((self.hidden, self.core_width))
        return wanted

    def load_core(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.b_in = torch.cat([tensors[name + ".b"].to(torch.float32) for name, _ in self.projected], dim=0).contiguous() if self.bias else None

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
        if self.gated:
            modules.append(("elementwise", {}))
        modules.append(("attention_tma" if self.head_dim % 64 == 0 else "attention_bf16", {"HB_HEAD_DIM": self.head_dim}))
        if self.head_dim in (64, 128):
            modules.append(("attention_tcgen05", {"HB_HEAD_DIM": self.head_dim}))
        return modules

    step_plans = GroupedQueryAttention.step_plans  # the rows of a step cut into tiles and single tokens, as for every attention of the package
    _attend_fast = GroupedQueryAttention._attend_fast
    _longest_short_row = staticmethod(GroupedQueryAttention._longest_short_row)

    def forward(self, x, step, cache, own_cache):
        if cache is None or own_cache == self.shares_kv:
            raise ValueError("this attention writes a cache of its own or reads the one its schedule entry names; the schedule gave it another")
        return super().forward(x, step, cache, True)

    def core(self, proj, col0, step, cache, out, scale):
        rows = proj[:, col0 : col0 + self.in_width]
        k_off, v_off = self.q_width, self.q_width + self.k_width
        q = torch.empty((proj.shape[0], self.q_width), dtype=self.dtype, device=proj.device)
        where = {} if self.shares_kv else {"cache": cache.kv, "block_table": cache.block_table, "token_row": step.token_row, "page_size": cache.page_size}
        if self.position is not None and self.position.dims:
            where.update(inv_freq=self.position.inv_freq, rot_dims=self.position.dims, rot_half=bool(getattr(self.position, "half", False)),
                         amplitude=float(getattr(self.position, "amplitude", 1.0)))
        ops.heads_store(rows, 0, k_off, v_off, self.heads, self.kv_heads, self.head_dim, self.value_dim, step.positions, q_out=q, bias=self.b_in, eps=self.eps,
                        unit_norm=self.unit_norm, temperature=self.temperature, **where)
        if self.fast:
            # the tensor-core kernels store rows in 16-byte pieces: columns of a wider buffer whose rows do not start on such a piece
            # are filled through a buffer of their own
            direct = out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0
            target = out if direct else torch.empty((proj.shape[0], self.core_width), dtype=self.dtype, device=proj.device)
            self._attend_fast(q, step, cache, out=target)
            if not direct:
                out.copy_(target)
            if self.gated:
                ops.sigmoid_gate_(out, rows, self.gate_off, scale)
            elif scale != 1.0:
                out.mul_(scale)
            return
        ops.attention_general(q, self.heads, self.kv_heads, self.head_dim, self.value_dim, cache.kv, cache.block_table, step.token_row, step.positions, cache.page_size,
                              self.scale, self.softcap, self.window, gate=rows if self.gated else None, gate_off=self.gate_off, out_scale=scale, out=out)
        if not self.gated and scale != 1.0:
            out.mul_(scale)


register_mixer("composed_attention", ComposedAttention)
