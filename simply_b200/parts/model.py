"""The generic decoder: embedding, layers in run order, final norm, output layer.

Built from a `ModelSpec` alone.  simply/model_lib.py:2935-3189 is the
reference's forward pass (embed :3000, blocks :3153-3167, final norm and head
:3183-3188); there the layer pattern is fixed by `block_attn_pattern`, here the
run order is a list that may repeat a layer or share a cache between calls.
Logits are computed only at the rows that are asked for (the reference
computes them for every token, :3186).
"""

from __future__ import annotations

from typing import Any

import torch

from simply_b200.cache.needs import PagedKVNeed
from simply_b200.config.model_spec import ModelSpec
from simply_b200.parts.base import Block, build_part
from simply_b200.parts.block import ResidualStream
from simply_b200.registry import BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, STREAM_INPUTS
from simply_b200.weights.loader import TensorSpec

# Importing the part modules registers the built-in parts.
from simply_b200.parts import attention as _attention  # noqa: F401
from simply_b200.parts import delta_rule as _delta_rule  # noqa: F401
from simply_b200.parts import experts as _experts  # noqa: F401
from simply_b200.parts import linear_attention as _linear_attention  # noqa: F401
from simply_b200.parts import forget_gate as _forget_gate  # noqa: F401
from simply_b200.parts import head_norm_attention as _head_norm_attention  # noqa: F401
from simply_b200.parts import hyper_connection as _hyper_connection  # noqa: F401
from simply_b200.parts import general_delta as _general_delta  # noqa: F401
from simply_b200.parts import latent_attention as _latent_attention  # noqa: F401
from simply_b200.parts import state_space as _state_space  # noqa: F401
from simply_b200.parts import normed_attention as _normed_attention  # noqa: F401
from simply_b200.parts import embedding as _embedding  # noqa: F401
from simply_b200.parts import feedforward as _feedforward  # noqa: F401
from simply_b200.parts import norm as _norm  # noqa: F401
from simply_b200.parts import position as _position  # noqa: F401
from simply_b200.parts import stream_input as _stream_input  # noqa: F401


class DecoderModel:

  def __init__(self, spec: ModelSpec):
    spec.validate()
    self.spec = spec
    self.embedding = build_part(EMBEDDINGS, spec.embedding)
    self.blocks: dict[str, Block] = {}
    for layer in spec.layers:
      mixer = build_part(MIXERS, layer.mixer)
      feed_forward = build_part(FEED_FORWARDS, layer.feed_forward)
      self.blocks[layer.name] = build_part(BLOCKS, layer.block, mixer=mixer,
                                           feed_forward=feed_forward)
    self.stream_inputs = {name: build_part(STREAM_INPUTS, part) for name, part in spec.stream_inputs.items()}
    self.final_norm = build_part(NORMS, spec.final_norm)
    self.head = build_part(HEADS, spec.head, embedding=self.embedding)
    self.cache_names = spec.cache_names()

  # ---- weights --------------------------------------------------------------
  def tensor_specs(self) -> list[TensorSpec]:
    specs = self.embedding.tensor_specs()
    for block in self.blocks.values():
      specs += block.tensor_specs()
    for part in self.stream_inputs.values():
      specs += part.tensor_specs()
    specs += self.final_norm.tensor_specs() + self.head.tensor_specs()
    names = [s.name for s in specs]
    if len(set(names)) != len(names):
      dup = sorted({n for n in names if names.count(n) > 1})
      raise ValueError(f"two parts claim the same tensor name(s): {dup}")
    return specs

  def bind(self, tensors: dict[str, torch.Tensor], ops: Any) -> None:
    self.embedding.bind(tensors, ops)
    for block in self.blocks.values():
      block.bind(tensors, ops)
    for part in self.stream_inputs.values():
      part.bind(tensors, ops)
    self.final_norm.bind(tensors, ops)
    self.head.bind(tensors, ops)

  def graph_safe(self) -> bool:
    """True if every part allows a decode step to be captured in a CUDA graph."""
    return (self.embedding.graph_safe and self.head.graph_safe and self.final_norm.graph_safe
            and all(b.graph_safe for b in self.blocks.values())
            and all(p.graph_safe for p in self.stream_inputs.values()))

  # ---- caches ---------------------------------------------------------------
  def cache_needs(self) -> dict[str, Any]:
    """Cache name -> need, taken from the call that writes the cache."""
    needs: dict[str, Any] = {}
    for call, cache in zip(self.spec.run_order, self.cache_names):
      need = self.blocks[call.layer].cache_need()
      if call.mixer_cache is not None:
        self._check_reader(call.layer, call.mixer_cache, need["mixer"], needs[call.mixer_cache]["mixer"])
        need = {key: part for key, part in need.items() if key != "mixer"}
      if call.writes_cache:
        if cache in needs and needs[cache] != need:
          raise ValueError(f"cache {cache!r} is written by calls with different needs")
        needs[cache] = need
    for call, cache in zip(self.spec.run_order, self.cache_names):
      if not call.writes_cache:
        self._check_reader(call.layer, cache, self.blocks[call.layer].cache_need(), needs[cache])
    return needs

  @staticmethod
  def _check_reader(layer: str, cache: str, need: Any, have: Any) -> None:
    """Refuses a layer that reads a cache of other shapes, or one that gives back what it needs."""
    same = not isinstance(have, dict) and not isinstance(need, dict) and isinstance(have, PagedKVNeed) == isinstance(
        need, PagedKVNeed) and all(
            getattr(need, f) == getattr(have, f) for f in ("num_kv_heads", "head_dim", "value_dim") if hasattr(have, f))
    if not same:
      raise ValueError(f"layer {layer!r} cannot read cache {cache!r}: {need} vs {have}")
    if isinstance(have, PagedKVNeed) and not have.covers(need):
      kept = f"a window of {have.window}" if have.window is not None else f"what {have} sees"
      raise ValueError(f"layer {layer!r} wants to see {need.window or 'all'} keys of cache {cache!r}, which keeps only {kept}")

  # ---- forward --------------------------------------------------------------
  def forward(self, ctx: Any, caches: dict[str, Any]) -> torch.Tensor | None:
    """Runs the step's tokens; returns float32 logits [R, vocab] at ctx.logit_rows."""
    first = self.embedding.forward(ctx)
    again = None
    if any(call.add_embedding for call in self.spec.run_order):
      # The stream is updated in place: what is added again later is a copy, in the activation
      # dtype where that holds the embedding exactly (then it rides along with the pending branch).
      exact = self.embedding.rides_exactly(ctx.ops.dtype) if hasattr(self.embedding, "rides_exactly") else False
      again = ctx.ops.cast(first, ctx.ops.dtype) if exact else first
      if again is first:
        again = first.clone()
    if self.stream_inputs:
      first, kept = first.clone(), first  # the stream is updated in place: the steps read a copy
    stream = ResidualStream(first)
    layer_outputs = ctx.memo.get("layer_outputs")  # a list: the stream after every layer call (debugging, tests)
    for call, cache in zip(self.spec.run_order, self.cache_names):
      if call.add_embedding:
        stream.add_input(again, ctx)
      if call.stream_input is not None:
        name, index = call.stream_input
        self.stream_inputs[name].forward(stream, kept, index, ctx)
      handle = caches.get(cache)
      if call.mixer_cache is not None:
        handle = {**(handle or {}), "mixer": caches[call.mixer_cache]["mixer"]}
      self.blocks[call.layer].forward(stream, ctx, handle, call.writes_cache and call.mixer_cache is None)
      if layer_outputs is not None:
        layer_outputs.append(stream.total(ctx))
    if ctx.logit_rows.numel() == 0:
      return None
    x = stream.normed(self.final_norm, ctx, rows=ctx.logit_rows)
    return self.head.forward(x, ctx)


def tensor_specs(spec: ModelSpec) -> list[TensorSpec]:
  return DecoderModel(spec).tensor_specs()
