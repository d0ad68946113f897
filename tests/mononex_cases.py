"""Small Mononex configurations with random (and crafted) weights for the tests.

Every comparison is between the engine (with a kernel table: the CUDA one on a GPU, the plain
PyTorch statements on the CPU) and the plain NumPy model of `tests/plain/mononex_plain.py`, which
sees whole sequences and has no cache.  The ways of running an engine (one request cut into
portions, several side by side) are those of `tests/generax_cases.py`.
"""

from __future__ import annotations

import copy

import numpy as np
import torch

from simply_b200.config import config_from_dict
from simply_b200.parts.model import DecoderModel
from simply_b200.weights import random_tensors
from tests.generax_cases import build_engine, cuts_of, run_cuts, run_mixed  # noqa: F401
from tests.plain import mononex_plain as plain
from tests.tolerances import assert_logits_close as check_close  # noqa: F401


def attention(heads=4, kv_heads=2, dim=16, vdim=8, chunk=12, scale=0.3, kv_from=None):
  m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
  if chunk is not None:
    m["mask"] = {"size": chunk}
  if kv_from is not None:
    m["kv_from"] = kv_from
  return {"type": "attention", "mixer": m}


def latent(heads=3, dim=12, rot_dim=8, vdim=10, q_rank=20, kv_rank=14, dims=None, base=300.0, scale=0.3, factor=4.0,
           original=24, fast=2.0, slow=0.25, scaling=True):
  rot = {"dims": rot_dim if dims is None else dims, "base": base}
  if scaling:
    rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
  return {"type": "latent_attention", "mixer": {
      "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
      "scale": scale, "rot": rot}}


def gla(heads=2, dim=12, vdim=20, tau=8.0):
  return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def config(layers, ffs, width=40, vocab=83, eps=1e-5, rank=5, max_context=512):
  """`ffs`: the feed-forward's hidden size per layer, or None for a layer without one."""
  out = []
  for layer, ff in zip(layers, ffs):
    layer = copy.deepcopy(layer)
    layer["mlp"] = None if ff is None else {"kind": "dense", "ff": ff}
    out.append(layer)
  return {"architecture": "Mononex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out,
          "max_context": max_context, "decay_rank": rank}


# Models that differ in every size and switch.  A: every mixer, a layer that reads another's keys
# through smaller chunks than its owner's.  B: value heads larger than key heads, two readers of one cache (one
# through larger chunks, one with more query heads' worth of chunks equal to a page), one kv head, a
# ramp that covers no pair, a layer without feed-forward, tau of 1.  C: sizes without whole 16-byte groups.  D:
# equal key and value sizes, attention last, a chunk of one token, no YaRN, a rotation of a part of the
# rotated dims.
CONFIG_A = config(
    [attention(), latent(), gla(), attention(chunk=7, kv_from=0), latent(heads=2, dim=16, rot_dim=4, vdim=16, q_rank=12, kv_rank=20, original=64),
     gla(heads=3, dim=8, vdim=8, tau=16.0)],
    [56, 64, 40, 64, 24, 48])
CONFIG_B = config(
    [gla(heads=1, dim=20, vdim=12, tau=1.0), attention(heads=6, kv_heads=1, dim=8, vdim=24, chunk=9),
     attention(heads=6, kv_heads=1, dim=8, vdim=24, chunk=20, kv_from=1),
     latent(heads=4, dim=8, rot_dim=12, vdim=4, base=50.0, factor=1.5, original=2000, fast=32.0, slow=1.0),
     attention(heads=6, kv_heads=1, dim=8, vdim=24, chunk=8, kv_from=1, scale=0.5)],
    [32, None, 72, 40, 16], width=48, vocab=131, eps=1e-6, rank=3)
CONFIG_C = config(
    [latent(heads=3, dim=5, rot_dim=6, vdim=7, q_rank=9, kv_rank=7), attention(heads=3, kv_heads=3, dim=7, vdim=5, chunk=10),
     gla(heads=3, dim=5, vdim=7, tau=3.5)],
    [18, 14, 22], width=36, vocab=50, rank=2)
CONFIG_D = config(
    [gla(heads=2, dim=16, vdim=16), latent(heads=2, dim=8, rot_dim=8, vdim=8, q_rank=8, kv_rank=24, dims=4, scaling=False),
     attention(heads=2, kv_heads=2, dim=16, vdim=16, chunk=1), attention(heads=4, kv_heads=4, dim=12, vdim=12, chunk=33)],
    [32, 32, 32, None], width=32, vocab=60, rank=8)


def as_numpy(t):
  return {k: v.float().numpy().astype(np.float64) for k, v in t.items()}


def weights(cfg_dict, seed=0, matrix_std=None, scale_std=0.2):
  """bfloat16-representable random weights by tensor name (CPU)."""
  cfg = config_from_dict(cfg_dict)
  specs = DecoderModel(cfg.model_spec()).tensor_specs()
  std = matrix_std if matrix_std is not None else 1.0 / cfg_dict["width"] ** 0.5
  t = random_tensors(specs, seed, matrix_std=std, scale_std=scale_std, dtype=torch.bfloat16)
  gen = torch.Generator().manual_seed(seed + 1)

  def draw(name, std, mean=0.0):
    t[name] = (torch.randn(t[name].shape, generator=gen) * std + mean).to(torch.bfloat16)

  for name in list(t):
    if name == "embed":
      draw(name, 1.0)
    elif name.endswith(".sink"):
      draw(name, 1.0)
    elif name.endswith(".a2.b"):
      draw(name, 1.0, 1.0)
    elif name.endswith(".a2"):
      draw(name, 0.5)
    elif name.endswith(".shift"):
      t[name] = torch.rand(t[name].shape, generator=gen).to(torch.bfloat16)
    elif name.endswith(".mlp.down"):
      draw(name, 0.5 / t[name].shape[1] ** 0.5)
  return cfg, t


def plant_needle(cfg_dict, t, layer, needle, asker, strength=7.0):
  """In a model whose layer `layer` is its first: makes the key of token `needle` and the query of
  token `asker` point the same way in the last (unrotated) dim of every head, so that the score stands
  out however many other keys there are, and gives the needle a value of its own.  The token shift of
  that layer is switched off, so that a token's place among others does not matter."""
  m = cfg_dict["layers"][layer]["mixer"]
  p, width, eps = f"l{layer}.mix", cfg_dict["width"], cfg_dict["norm"]["eps"]
  gen = torch.Generator().manual_seed(77 + layer)
  for tok, sign in ((needle, 1.0), (asker, -1.0)):
    row = torch.zeros(width)
    row[(7 * tok + 3) % width] = 4.0 * sign
    row[(5 * tok + 1) % width] = 4.0
    t["embed"][tok] = row.to(torch.bfloat16)
  t[f"l{layer}.shift"] = torch.zeros_like(t[f"l{layer}.shift"])
  w = as_numpy(t)
  h = {tok: plain.zero_centred_norm(w["embed"][tok][None], w[f"l{layer}.norm1"], eps)[0] for tok in (needle, asker)}

  def bend(name, row, by):
    v = t[name].float()
    v[row] += torch.from_numpy(by).float()
    t[name] = v.to(torch.bfloat16)

  d = m["dim"]
  if cfg_dict["layers"][layer]["type"] == "attention":
    for g in range(m["kv_heads"]):
      bend(f"{p}.k", g * d + d - 1, strength * h[needle] / (h[needle] @ h[needle]))
    for a in range(m["heads"]):
      bend(f"{p}.q", a * d + d - 1, strength * h[asker] / (h[asker] @ h[asker]))
    seen, values = h[needle], f"{p}.v"
  else:
    cq = plain.unit_rms(h[asker][None] @ w[f"{p}.dq"].T, eps)[0] * w[f"{p}.dq.norm"]
    seen = plain.unit_rms((h[needle][None] @ w[f"{p}.dkv"].T)[:, :m["kv_rank"]], eps)[0] * w[f"{p}.dkv.norm"]
    per = d + m["rot_dim"]
    for a in range(m["heads"]):
      bend(f"{p}.uk", a * d + d - 1, strength * seen / (seen @ seen))
      bend(f"{p}.uq", a * per + d - 1, strength * cq / (cq @ cq))
    values = f"{p}.uv"
  v = t[values].float()
  v += 2.0 * torch.randn(v.shape[0], generator=gen)[:, None] * torch.from_numpy(seen).float()[None, :] / float(seen @ seen)
  t[values] = v.to(torch.bfloat16)
  return t
