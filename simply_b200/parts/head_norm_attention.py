"""Grouped-query attention whose heads are normed one by one, with tied values and an output gate.

Beside `paged_attention` and `qk_norm_attention` for designs whose attention differs from them in
any of these, each switched by a parameter:

* rotary positions on the first `rotary["dims"]` dims of every q and k head, pairing neighbours
  (2i, 2i + 1) (`layout` "neighbours") or halves (i, i + dims/2) (`layout` "halves"), angle
  p * base^(-2i/dims);
* `head_norm`: after the rotation every q and k head is divided by its own root mean square
  (over head_dim, eps inside the root, no scale); with `head_norm_scale` before the rotation instead,
  and then scaled per channel (tensors `q.norm`, `k.norm`, each of head_dim numbers for all heads);
* `conv_taps` n: before norm and rotation every channel of q, k and v passes a causal convolution over
  time without an activation, y_t = sum_j w[:, j] u_(t - n + 1 + j) with zeros before the sequence's
  start (tensors `<name>.conv`, [channels, n]); the last n - 1 rows as projected are part of a
  request's state.  Convolution, norm, rotation and the store are one kernel;
* `tie_values`: there is no value projection: a key head as projected (before rotation and
  norm) is also the value head;
* score = q.k * score_scale, then `score_softcap` * tanh(score / score_softcap) before the softmax;
* causal, optionally over a window of `window` keys, and with it `keep_first` tokens at the sequence's
  start that stay visible (at their true positions) when the window has left them;
* `output_gate`: the heads side by side are multiplied by sigmoid(W_g y) before the output
  projection; the gate reads the mixer's input, like q and k.  `gate_per_head`: W_g has one row
  per head, and a head's whole result is multiplied by its one number;
* `value_dim`: value heads of another size than key heads (not with tied values);
* `projection_bias`: q, k and v each have a bias (tensor `<name>.b`), added in float32 to the
  projection before the rotation;
* `distance_bias`: the score of query i and key j loses r1_h * log(1 + r2_h * (i - j)), with two
  learned numbers per query head (tensors `r1`, `r2`), in float32;
* `distance_slopes`: the score loses slope_h * (i - j) with the fixed slopes 2^(-8 (h + 1) / heads);
* `chunk` C (in place of a window): a query sees the keys of its own chunk only, from
  (i // C) * C on, with chunks counted from the sequence's start;
* `sink`: the softmax's denominator also holds exp(sink_h), a learned number per head without a key
  or a value (tensor `sink`); `unit_sink`: a one joins the denominator, without a tensor;
* `project_kv=False`: the layer has no k and v tensors and reads the cache another layer writes.
  `cache_chunks`: the chunk sizes of all layers that read this layer's cache (None among them: one
  sees every token), which the cache has to serve.

q, k, (v) and the gate come out of one fused product.
"""

from __future__ import annotations

from typing import Any

import torch

from simply_b200.cache.needs import ChunkedKVNeed, PagedKVNeed, SlotStateNeed
from simply_b200.parts.base import Mixer
from simply_b200.parts.linear import Linear, fuse_rows
from simply_b200.parts.normed_attention import rotation_frequencies
from simply_b200.registry import MIXERS
from simply_b200.weights.loader import TensorSpec

_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "r1": "r1", "r2": "r2", "bias": "b",
          "sink": "sink", "norm": "norm", "conv": "conv"}


@MIXERS.register("head_norm_attention")
class HeadNormAttention(Mixer):

  graph_safe = True

  def __init__(self, prefix: str, width: int, num_heads: int, num_kv_heads: int, head_dim: int,
               score_scale: float, eps: float, score_softcap: float = 0.0, window: int | None = None,
               rotary: dict | None = None, head_norm: bool = True, tie_values: bool = True,
               output_gate: bool = True, names: dict[str, str] | None = None, value_dim: int | None = None,
               gate_per_head: bool = False, projection_bias: bool = False, distance_bias: bool = False,
               distance_slopes: bool = False, chunk: int | None = None, sink: bool = False, project_kv: bool = True,
               cache_chunks: tuple = (), head_norm_scale: bool = False, conv_taps: int = 0, keep_first: int = 0,
               unit_sink: bool = False):
    if num_heads % num_kv_heads:
      raise ValueError(f"{prefix}: num_heads {num_heads} is no multiple of num_kv_heads {num_kv_heads}")
    self.prefix, self.width = prefix, width
    self.num_heads, self.num_kv_heads, self.head_dim = num_heads, num_kv_heads, head_dim
    self.score_scale, self.eps = float(score_scale), float(eps)
    self.score_softcap = float(score_softcap or 0.0)
    self.window = window
    self.rotary = dict(rotary) if rotary else None
    if self.rotary:
      if self.rotary["dims"] % 2 or self.rotary["dims"] > head_dim:
        raise ValueError(f"{prefix}: {self.rotary['dims']} rotated dims do not fit a head of {head_dim}")
      if self.rotary.get("layout", "neighbours") not in ("neighbours", "halves"):
        raise ValueError(f"{prefix}: rotary layout must be 'neighbours' or 'halves'")
    self.head_norm, self.tie_values, self.output_gate = bool(head_norm), bool(tie_values), bool(output_gate)
    self.value_dim = head_dim if value_dim is None else int(value_dim)
    if self.tie_values and self.value_dim != head_dim:
      raise ValueError(f"{prefix}: tied values have the keys' size")
    self.gate_per_head, self.projection_bias = bool(gate_per_head), bool(projection_bias)
    self.distance_bias, self.distance_slopes = bool(distance_bias), bool(distance_slopes)
    if self.distance_bias and self.distance_slopes:
      raise ValueError(f"{prefix}: a score loses one kind of distance term")
    if chunk is not None and (window is not None or chunk <= 0):
      raise ValueError(f"{prefix}: a chunk has a positive size and takes the place of a window")
    self.chunk, self.has_sink, self.project_kv = chunk, bool(sink), bool(project_kv)
    self.unit_sink = bool(unit_sink)
    if self.has_sink and self.unit_sink:
      raise ValueError(f"{prefix}: the denominator holds one kind of sink")
    self.keep_first = int(keep_first or 0) if window is not None else 0  # (without a window every token stays)
    if self.keep_first and chunk is not None:
      raise ValueError(f"{prefix}: kept first tokens go with a window")
    self.head_norm_scale, self.conv_taps = bool(head_norm_scale), int(conv_taps or 0)
    if self.head_norm_scale and not self.head_norm:
      raise ValueError(f"{prefix}: scales of the heads' norms need the norms")
    if self._prepared and (self.tie_values or self.projection_bias or not self.project_kv):
      raise ValueError(f"{prefix}: convolutions and scaled head norms go with projected keys and values without biases")
    if self.conv_taps and not self.head_norm_scale:
      raise ValueError(f"{prefix}: convolutions go with scaled head norms")
    self.cache_chunks = tuple(cache_chunks)
    if self.tie_values and not self.project_kv:
      raise ValueError(f"{prefix}: tied values need a key projection")
    n = self.names = {**_NAMES, **(names or {})}
    self.q_proj = Linear(f"{prefix}.{n['q']}", num_heads * head_dim, width)
    self.k_proj = Linear(f"{prefix}.{n['k']}", num_kv_heads * head_dim, width) if self.project_kv else None
    self.v_proj = None if self.tie_values or not self.project_kv else Linear(f"{prefix}.{n['v']}", num_kv_heads * self.value_dim, width)
    gate_rows = num_heads if self.gate_per_head else num_heads * self.value_dim
    self.g_proj = Linear(f"{prefix}.{n['g']}", gate_rows, width) if self.output_gate else None
    self.o_proj = Linear(f"{prefix}.{n['o']}", width, num_heads * self.value_dim)
    self.in_weight = self.rot_freq = self.in_bias = self.distance = self.sink = None
    self.q_norm = self.k_norm = self.conv_weight = None
    self.gate_offset = 0

  @property
  def _prepared(self) -> bool:
    """Whether q, k and v take the kernel with convolutions and scaled norms to the cache."""
    return self.conv_taps > 0 or self.head_norm_scale

  def _inputs(self) -> list[Linear]:
    return [p for p in (self.q_proj, self.k_proj, self.v_proj, self.g_proj) if p is not None]

  def cache_need(self):
    value_dim = None if self.value_dim == self.head_dim else self.value_dim
    chunks = set(self.cache_chunks) | {self.chunk}
    if self.conv_taps > 1:
      channels = sum(p.out_features for p in (self.q_proj, self.k_proj, self.v_proj))
      return {"kv": self._kv_need(chunks, value_dim), "conv": SlotStateNeed((self.conv_taps - 1, channels), "float32")}
    return self._kv_need(chunks, value_dim)

  def _kv_need(self, chunks: set, value_dim: int | None) -> PagedKVNeed:
    if None in chunks:
      return PagedKVNeed(self.num_kv_heads, self.head_dim, self.window, value_dim=value_dim, keep_first=self.keep_first)
    return ChunkedKVNeed(self.num_kv_heads, self.head_dim, value_dim=value_dim, chunks=tuple(sorted(chunks)))

  def graph_plans(self, ops, batch: int, bucket: int, max_burst: int, page_size: int) -> list:
    opts: dict[str, Any] = {}  # (only what differs from the plain case)
    if self.chunk is not None:
      opts["key_chunk"] = self.chunk
    if self.value_dim != self.head_dim:
      opts["value_dim"] = self.value_dim
    if self.keep_first:
      opts["keep_first"] = self.keep_first
    plan = ops.attention_graph_plan(
        window=self.window, num_heads=self.num_heads, num_kv_heads=self.num_kv_heads, head_dim=self.head_dim,
        batch=batch, bucket=bucket, max_burst=max_burst, page_size=page_size, **opts)
    return [plan] if plan is not None else []

  def tensor_specs(self) -> list[TensorSpec]:
    specs = [p.spec() for p in self._inputs()] + [self.o_proj.spec()]
    if self.projection_bias:
      specs += [TensorSpec(f"{p.name}.{self.names['bias']}", (p.out_features,), "scale", precision="stored")
                for p in self._biased()]
    if self.distance_bias:
      specs += [TensorSpec(f"{self.prefix}.{self.names[r]}", (self.num_heads,), "gain", precision="stored")
                for r in ("r1", "r2")]
    if self.head_norm_scale:
      specs += [TensorSpec(f"{p.name}.{self.names['norm']}", (self.head_dim,), "gain") for p in (self.q_proj, self.k_proj)]
    if self.conv_taps:
      specs += [TensorSpec(f"{p.name}.{self.names['conv']}", (p.out_features, self.conv_taps), "gain")
                for p in (self.q_proj, self.k_proj, self.v_proj)]
    if self.has_sink:
      specs.append(TensorSpec(f"{self.prefix}.{self.names['sink']}", (self.num_heads,), "scale", precision="stored"))
    return specs

  def _biased(self) -> list[Linear]:
    return [p for p in (self.q_proj, self.k_proj, self.v_proj) if p is not None]

  def bind(self, tensors, ops) -> None:
    if self.head_dim % 2 == 0 and self.value_dim == self.head_dim:  # (the general kernel takes the rest)
      ops.check_attention(self.head_dim, self.num_heads, self.num_kv_heads)
    elif self.value_dim != self.head_dim:
      ops.check_attention(self.head_dim, self.num_heads, self.num_kv_heads, self.value_dim)
    w = fuse_rows([tensors[p.name] for p in self._inputs()])
    extra = -w.shape[0] % 8  # whole 16-byte groups of output features for the products' stores
    self.in_weight = torch.cat([w, w.new_zeros(extra, w.shape[1])]).contiguous() if extra else w
    self.gate_offset = sum(p.out_features for p in self._inputs()[:-1]) if self.output_gate else 0
    self.o_proj.bind(tensors)
    if self.projection_bias:
      self.in_bias = torch.cat([tensors[f"{p.name}.{self.names['bias']}"].float() for p in self._biased()]).contiguous()
    if self.distance_bias:  # [2, heads]: r1, then r2
      self.distance = torch.stack([tensors[f"{self.prefix}.{self.names[r]}"].float() for r in ("r1", "r2")]).contiguous()
    device = self.in_weight.device
    if self.distance_slopes:  # [1, heads]
      h = torch.arange(1, self.num_heads + 1, dtype=torch.float64)
      self.distance = torch.exp2(-8.0 * h / self.num_heads).float()[None].to(device).contiguous()
    if self.has_sink:
      self.sink = tensors[f"{self.prefix}.{self.names['sink']}"].float().contiguous()
    if self.unit_sink:
      self.sink = torch.zeros(self.num_heads, dtype=torch.float32, device=device)  # exp(0) = 1
    if self.head_norm_scale:
      self.q_norm, self.k_norm = (tensors[f"{p.name}.{self.names['norm']}"].float().contiguous()
                                  for p in (self.q_proj, self.k_proj))
    if self.conv_taps:  # [taps, channels]: neighbouring channels read neighbouring numbers
      conv = [tensors[f"{p.name}.{self.names['conv']}"].float() for p in (self.q_proj, self.k_proj, self.v_proj)]
      self.conv_weight = torch.cat(conv, dim=0).t().contiguous()
    if self.rotary:
      freq = rotation_frequencies(self.rotary["dims"], self.rotary["base"])
      self.rot_freq = torch.from_numpy(freq).to(self.in_weight.device)

  def _store_options(self) -> dict:
    """(only what differs from the plain case is passed on, so that a kernel table that predates
    an option still serves the models that do not use it)"""
    opts: dict[str, Any] = {}
    if self.value_dim != self.head_dim:
      opts["value_dim"] = self.value_dim
    if self.in_bias is not None:
      opts["bias"] = self.in_bias
    return opts

  def _attention_options(self) -> dict:
    opts: dict[str, Any] = {}
    if self.value_dim != self.head_dim:
      opts["value_dim"] = self.value_dim
    if self.distance is not None:
      opts["distance_bias"] = self.distance
    if self.sink is not None:
      opts["sink"] = self.sink
    if self.chunk is not None:
      opts["key_chunk"] = self.chunk
    if self.keep_first:
      opts["keep_first"] = self.keep_first
    return opts

  def forward(self, x: torch.Tensor, ctx: Any, cache: Any, writes_cache: bool = True) -> torch.Tensor:
    ops = ctx.ops
    if writes_cache and not self.project_kv:
      raise ValueError(f"{self.prefix}: a mixer without k/v projections cannot write a cache")
    conv_state = None
    if self.conv_taps > 1:
      conv_state, cache = cache["conv"].storage, cache["kv"]
    block_table = ctx.block_tables[cache.group]
    proj = ops.linear(x, self.in_weight)  # q | k | (v) | (gate)
    interleaved = bool(self.rotary) and self.rotary.get("layout", "neighbours") == "neighbours"
    if self._prepared:
      q = ops.conv_headnorm_rotate_store(
          proj, self.conv_weight, conv_state, self.q_norm, self.k_norm, self.eps, self.score_scale, self.rot_freq,
          interleaved=interleaved, num_heads=self.num_heads, num_kv_heads=self.num_kv_heads, head_dim=self.head_dim,
          value_dim=self.value_dim, storage=cache.storage if writes_cache else None, block_table=block_table, ctx=ctx)
    else:
      q = self._rotate_store(proj, interleaved, cache, writes_cache, block_table, ctx)
    o = ops.paged_attention(
        q, cache.storage, block_table, ctx, num_heads=self.num_heads, num_kv_heads=self.num_kv_heads,
        head_dim=self.head_dim, logit_softcap=self.score_softcap, window=self.window, **self._attention_options())
    if self.output_gate:
      o = ops.sigmoid_gate(o, proj, self.gate_offset, self.value_dim if self.gate_per_head else 1)
    return self.o_proj(o, ctx)

  def _rotate_store(self, proj, interleaved, cache, writes_cache, block_table, ctx) -> torch.Tensor:
    return ctx.ops.rotate_headnorm_store(
        proj, self.eps, self.score_scale, self.rot_freq, interleaved=interleaved,
        head_norm=self.head_norm, tie_values=self.tie_values, num_heads=self.num_heads,
        num_kv_heads=self.num_kv_heads if self.project_kv else 0, head_dim=self.head_dim,
        storage=cache.storage if writes_cache else None, block_table=block_table, ctx=ctx,
        **self._store_options())
