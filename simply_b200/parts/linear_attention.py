"""Gated linear attention: a recurrent mixer whose state decays per key channel.

Per head a matrix S [head_dim, value_dim] (float32, zero at a request's start, one per request in
a state slot) that every token updates and then reads:

  q_t = W_q y_t * head_dim^(-1/2),  k_t = W_k y_t      [heads, head_dim]
  v_t = W_v y_t                                        [heads, value_dim]
  f_t = sigmoid(W_a2 (W_a1 y_t) + b)^(1 / tau)         [heads, head_dim], through a low rank
  S_t = diag(f_t) S_(t-1) + k_t v_t^T
  o_t = S_t^T q_t

Each head's o is divided by its root mean square over value_dim, scaled per channel (one scale for
all heads), multiplied by silu(W_g y), and the heads side by side go through W_o.  q, k, v, the gate
and the low rank's first half come out of one fused product; the low rank's second half and
everything between it and the output projection is float32.
"""

from __future__ import annotations

from typing import Any

import torch

from simply_b200.cache.needs import SlotStateNeed
from simply_b200.parts.base import Mixer
from simply_b200.parts.linear import Linear, fuse_rows
from simply_b200.registry import MIXERS
from simply_b200.weights.loader import TensorSpec

_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "decay_in": "a1", "decay_out": "a2", "decay_bias": "a2.b",
          "norm": "norm", "out": "o"}


@MIXERS.register("gated_linear_attention")
class GatedLinearAttention(Mixer):

  graph_safe = True  # reads the step's device tensors only; rows that repeat a slot do not write its state

  def __init__(self, prefix: str, width: int, num_heads: int, head_dim: int, value_dim: int, tau: float, eps: float,
               decay_rank: int = -1, names: dict[str, str] | None = None):
    if not tau > 0:
      raise ValueError(f"{prefix}: tau must be positive, got {tau}")
    self.prefix, self.width = prefix, width
    self.num_heads, self.head_dim, self.value_dim = num_heads, head_dim, value_dim
    self.tau, self.eps = float(tau), float(eps)
    n = self.names = {**_NAMES, **(names or {})}
    qk, vv = num_heads * head_dim, num_heads * value_dim
    self.projections = [Linear(f"{prefix}.{n[role]}", rows, width)
                        for role, rows in (("q", qk), ("k", qk), ("v", vv), ("gate", vv))]
    self.decay_in = Linear(f"{prefix}.{n['decay_in']}", decay_rank, width)  # -1: the tensors' shapes give it
    self.decay_out = Linear(f"{prefix}.{n['decay_out']}", qk, decay_rank)
    self.o_proj = Linear(f"{prefix}.{n['out']}", width, vv)

  def _name(self, role: str) -> str:
    return f"{self.prefix}.{self.names[role]}"

  def cache_need(self):
    return SlotStateNeed((self.num_heads, self.head_dim, self.value_dim), "float32")

  def tensor_specs(self) -> list[TensorSpec]:
    specs = [p.spec() for p in self.projections + [self.decay_in, self.decay_out, self.o_proj]]
    return specs + [TensorSpec(self._name("decay_bias"), (self.num_heads * self.head_dim,), "scale", precision="stored"),
                    TensorSpec(self._name("norm"), (self.value_dim,), "gain")]

  def bind(self, tensors, ops) -> None:
    t = tensors
    w = fuse_rows([t[p.name] for p in self.projections + [self.decay_in]])  # q | k | v | gate | low rank
    self.rank = t[self.decay_in.name].shape[0]
    if t[self.decay_out.name].shape[1] != self.rank:
      raise ValueError(f"{self.prefix}: the low-rank pair does not fit")
    extra = -w.shape[0] % 8
    self.in_weight = torch.cat([w, w.new_zeros(extra, w.shape[1])]).contiguous() if extra else w
    # [rank, heads * head_dim]: neighbouring channels read neighbouring numbers
    self.decay_out_t = t[self.decay_out.name].float().t().contiguous()
    self.o_proj.bind(t)
    self.decay_bias = t[self._name("decay_bias")].float().contiguous()
    self.norm_weight = t[self._name("norm")].float().contiguous()

  def forward(self, x: torch.Tensor, ctx: Any, cache: Any, writes_cache: bool = True) -> torch.Tensor:
    ops = ctx.ops
    qk, vv = self.num_heads * self.head_dim, self.num_heads * self.value_dim
    pre = ops.linear(x, self.in_weight)
    o = ops.gated_linear_scan(pre, 2 * qk + 2 * vv, self.decay_out_t, self.decay_bias, self.tau, cache.storage, ctx,
                              num_heads=self.num_heads, head_dim=self.head_dim, value_dim=self.value_dim)
    y = ops.gated_head_norm(o, pre, 2 * qk + vv, self.norm_weight, self.eps, self.num_heads, self.value_dim, gate="silu")
    return self.o_proj(y, ctx)
