"""Differential attention: two softmax maps per head over the same values, the second taken off the first.

    q [heads, 2, d], k [kv_heads, 2, d], v [kv_heads, e] = W_q x, W_k x, W_v x;  every query and key of a map passes an RMS norm over d
    (one weight for all queries, one for all keys);  a_m = softmax over the seen keys of (q_m . k_m) * scale, applied to v
    w = exp(lq1 . lk1) - exp(lq2 . lk2) + diff          one number per layer
    o = a_1 - w a_2;   o <- o / sqrt(mean(o^2) + eps) * (1 - diff);   y = W_o [o heads side by side * sigmoid(W_g x)]

Position p sees the positions j <= p with p - j < ``window`` (0: every one of them) or j < ``keep_first``; nothing is rotated.  Query
head h reads key/value head h // (heads / kv_heads).  The pages of a window are given back while the request lives, those of the kept
first positions stay.

Per step: one product to [q | k | v | g] kept in float; one kernel that norms and stores (``ops.heads_store``); attention; the output product.
A head's two keys lie side by side in its pages, so that in bfloat16, when they are together as wide as a value (2 d = e, a multiple of 16), the
tensor-core kernels of the package's other attentions read them: prompt portions with e = 128 take the tcgen05 kernel, whose two halves
are then the two maps and which finishes the heads itself (difference, norm, gate); decoded tokens, and other sizes, run the kernels of
heads of 2 d with every map a virtual head whose query is zero in the other map's half, and ``csrc/attention_combine.cu`` merges and
finishes.  Everything else, and float32, runs in ``csrc/attention_generic.cu`` with a float result, finished by the same kernel.  Norms,
scores, softmax, w, the difference and what follows it are float; a value is rounded once where it is stored.

Parameters: ``hidden_size``, ``heads``, ``kv_heads``, ``head_dim`` (d), ``value_dim`` (e), ``scale``, ``diff``, ``window``, ``keep_first``, ``eps``.
Tensors: q, k, v, q.norm, k.norm, lq1, lk1, lq2, lk2, g, o.
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


class DifferentialAttention(Mixer):
    def __init__(self, spec: PartSpec, build: BuildContext):
        super().__init__(spec, build)
        p = spec.params
        self.hidden, self.heads, self.kv_heads = int(p["hidden_size"]), int(p["heads"]), int(p["kv_heads"])
        self.head_dim, self.value_dim = int(p["head_dim"]), int(p["value_dim"])
        self.scale, self.diff, self.eps = float(p["scale"]), float(p["diff"]), float(p["eps"])
        self.window = int(p.get("window") or 0)
        self.keep_first = int(p.get("keep_first") or 0) if self.window else 0
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.kv_heads} key/value heads do not divide {self.heads} heads")
        if max(self.head_dim, self.value_dim) > LARGEST_HEAD:
            raise ValueError(f"heads of {self.head_dim} / {self.value_dim} are above the kernels' limit of {LARGEST_HEAD}")
        self.q_width, self.k_width = 2 * self.heads * self.head_dim, 2 * self.kv_heads * self.head_dim
        self.v_width, self.core_width = self.kv_heads * self.value_dim, self.heads * self.value_dim
        self.fast = self.dtype == torch.bfloat16 and fast_attention.differential_supported(self.head_dim, self.value_dim) and self.scale > 0

    def weights(self) -> dict[str, WeightSpec]:
        h, d = self.hidden, self.head_dim
        wanted = {"q": WeightSpec((self.q_width, h)), "k": WeightSpec((self.k_width, h)), "v": WeightSpec((self.v_width, h)), "g": WeightSpec((self.core_width, h)),
                  "o": WeightSpec((h, self.core_width)), "q.norm": WeightSpec((d,), init="one_plus_normal"), "k.norm": WeightSpec((d,), init="one_plus_normal")}
        wanted.update({name: WeightSpec((d,)) for name in ("lq1", "lk1", "lq2", "lk2")})
        return wanted

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        mats = [tensors[name] for name in ("q", "k", "v", "g")]
        dtype = _common_dtype(mats)
        self.w_in = torch.cat([m.to(dtype) for m in mats], dim=0).contiguous()
        self.w_o = tensors["o"].contiguous()
        self.q_norm, self.k_norm = tensors["q.norm"].to(torch.float32).contiguous(), tensors["k.norm"].to(torch.float32).contiguous()
        first, second = ((tensors["lq" + i].to(torch.float64) * tensors["lk" + i].to(torch.float64)).sum().exp() for i in ("1", "2"))
        self.map_weight = float(first - second) + self.diff

    def cache_request(self):
        if 2 * self.head_dim == self.value_dim:
            return PagedKV(self.kv_heads, self.value_dim, self.window, self.keep_first)
        return PagedTokens((self.kv_heads,), (2 * self.head_dim + self.value_dim,), self.window, keep_first=self.keep_first)

    def kernel_modules(self):
        modules = [("heads_prepare", {}), ("attention_combine", {}), ("sgemm_f32", {}) if self.dtype == torch.float32 else ("gemm_tcgen05", {})]
        if not self.fast:
            return modules + [("attention_generic", {})]
        if self.value_dim % 64 == 0:
            modules.append(("attention_tma", {"HB_HEAD_DIM": self.value_dim}))
        else:
            modules.append(("attention_bf16", {"HB_HEAD_DIM": self.value_dim}))
        if self.value_dim == 128:
            modules.append(("attention_tcgen05", {"HB_HEAD_DIM": 128}))
        return modules

    def step_plans(self):
        """As for a grouped-query attention of 2 * heads heads of e entries."""
        if not self.fast:
            return {}
        return GroupedQueryAttention.plans_for(2 * self.heads, self.kv_heads, self.value_dim, self._tile_rows)

    def _tile_rows(self, page_size) -> int:
        return fast_attention.differential_tile_rows(self.value_dim, page_size)

    def _attend_fast(self, q, gate, step, cache, out):
        heads, kv_heads = 2 * self.heads, self.kv_heads
        size = self._tile_rows(step.host.get("page_size"))
        key = f"attn_tiles_{fast_attention.tile_tokens(heads, kv_heads, size)}"
        n_tiles, n_items = step.host.get(key, 0), step.host.get("attn_items", 0)
        after = (self.scale, self.window, self.keep_first, gate, self.map_weight, self.eps, 1.0 - self.diff, out)
        if n_tiles:
            fast_attention.differential_tiles(q, self.heads, cache.kv, cache.block_table, step.token_row, step.positions, step.extra[key], n_tiles, *after)
        if n_items:  # after the tiles: where those finish all tokens' rows through a buffer, the single tokens' rows are written again here
            longest = step.host.get("context_cap") or GroupedQueryAttention._longest_short_row(step.rows)
            if self.window:
                longest = min(longest, self.window + self.keep_first + 2 * fast_attention.KEY_TILE)
            splits = fast_attention.choose_splits(n_items, heads, kv_heads, longest)
            fast_attention.differential_tokens(q, self.heads, cache.kv, cache.block_table, step.token_row, step.positions, step.extra["attn_items"], n_items, splits, *after)

    def forward(self, x, step, cache, own_cache):
        if cache is None or not own_cache:
            raise ValueError("this attention writes a paged cache of its own; the schedule gave it none")
        proj = ops.linear(x, self.w_in, None, torch.float32)
        k_off = self.q_width
        v_off = k_off + self.k_width
        q = torch.empty((x.shape[0], self.q_width), dtype=self.dtype, device=x.device)
        ops.heads_store(proj, 0, k_off, v_off, self.heads, self.kv_heads, self.head_dim, self.value_dim, step.positions, q_out=q, maps=2, q_norm=self.q_norm,
                        k_norm=self.k_norm, eps=self.eps, cache=cache.kv, block_table=cache.block_table, token_row=step.token_row, page_size=cache.page_size)
        gate = proj[:, v_off + self.v_width:]
        out = torch.empty((x.shape[0], self.core_width), dtype=self.dtype, device=x.device)
        if self.fast:
            self._attend_fast(q, gate, step, cache, out)
        else:
            maps = ops.attention_general(q, self.heads, self.kv_heads, self.head_dim, self.value_dim, cache.kv, cache.block_table, step.token_row, step.positions,
                                         cache.page_size, self.scale, 0.0, self.window, keep_first=self.keep_first, maps=2, wide_out=True)
            fast_attention.differential_combine(maps, None, None, x.shape[0], self.heads, 1, self.value_dim, self.map_weight, self.eps, 1.0 - self.diff, gate, out)
        return ops.linear(out, self.w_o, None, self.dtype, may_leave_partials=True)  # the result is a residual delta


register_mixer("differential_attention", DifferentialAttention)
