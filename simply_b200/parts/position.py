"""Position encodings.  A position encoding hands the mixer rotation tables.

`rotary` is simply/utils/position_encoding.py:53-110: the two halves of a head
rotate together, timescale_j = theta ** (2j / head_dim), angle = position /
timescale / scale_factor, all in float32.  `none` rotates nothing.

`scaled_frequencies` serves the mixers that turn a part of their heads themselves.
"""

from __future__ import annotations

from typing import Any

import math

import numpy as np
import torch

from simply_b200.parts.base import PositionEncoding
from simply_b200.registry import POSITION_ENCODINGS


def scaled_frequencies(dims: int, base: float, scaling: dict | None = None) -> tuple[np.ndarray, float]:
  """Angle per position of each pair of `dims` rotated dims (float32 [dims / 2]) and the factor on the
  cosines and sines.  Without `scaling`: base^(-2 i / dims) and 1.  With YaRN's (factor, original,
  fast, slow): pairs that turn more than `fast` times over `original` positions keep their
  frequency, pairs that turn less than `slow` times have it divided by `factor`, in between a linear
  ramp over the pair's number; cosines and sines grow by 0.1 ln(factor) + 1."""
  i = np.arange(dims // 2, dtype=np.float64)
  freq = np.power(float(base), -2.0 * i / max(dims, 1))
  if not scaling:
    return freq.astype(np.float32), 1.0
  factor = float(scaling["factor"])

  def pair_turning(times: float) -> float:
    return dims * math.log(float(scaling["original"]) / (2.0 * math.pi * times)) / (2.0 * math.log(float(base)))

  lo = max(math.floor(pair_turning(float(scaling["fast"]))), 0)
  hi = min(math.ceil(pair_turning(float(scaling["slow"]))), dims - 1)
  slowed = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
  freq = freq / factor * slowed + freq * (1.0 - slowed)
  return freq.astype(np.float32), 0.1 * math.log(factor) + 1.0


@POSITION_ENCODINGS.register("rotary")
class RotaryEncoding(PositionEncoding):

  graph_safe = True

  def __init__(self, prefix: str = "", theta: float = 10000.0, scale_factor: float = 1.0):
    self.theta = float(theta)
    self.scale_factor = float(scale_factor)
    self._timescales: dict[tuple[int, str], torch.Tensor] = {}

  def timescale(self, head_dim: int, device) -> torch.Tensor:
    key = (head_dim, str(device))
    t = self._timescales.get(key)
    if t is None:
      half = head_dim // 2
      fraction = (2 * np.arange(half) / head_dim).astype(np.float32)
      t = torch.from_numpy(np.power(np.float32(self.theta), fraction).astype(np.float32)).to(device)
      self._timescales[key] = t
    return t

  def rotation_tables(self, ctx: Any, head_dim: int):
    key = ("rotary", self.theta, self.scale_factor, head_dim)
    tables = ctx.memo.get(key)
    if tables is None:
      tables = ctx.ops.rotation_tables(
          ctx.positions, self.timescale(head_dim, ctx.positions.device), self.scale_factor)
      ctx.memo[key] = tables
    return tables


@POSITION_ENCODINGS.register("none")
class NoPositionEncoding(PositionEncoding):

  graph_safe = True

  def __init__(self, prefix: str = ""):
    pass

  def rotation_tables(self, ctx: Any, head_dim: int):
    return None
