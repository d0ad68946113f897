"""Small Pibulix configurations with random (and crafted) weights for the tests.

Every comparison is between the engine (with a kernel table: the CUDA one on a GPU, the plain
PyTorch statements on the CPU) and the plain NumPy model of `tests/plain/pibulix_plain.py`, which
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
from tests.plain import pibulix_plain as plain
from tests.tolerances import assert_logits_close as check_close  # noqa: F401


def attention(heads=4, kv_heads=2, dim=16, vdim=16, window=12, keep_first=3, conv=3, dims=8, base=500.0, softcap=8.0,
              scale=0.3):
  m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
  if conv is not None:
    m["conv"] = conv
  if window is not None:
    m["mask"] = {"size": window, "keep_first": keep_first}
  if dims:
    m["rot"] = {"dims": dims, "base": base}
  if softcap:
    m["softcap"] = softcap
  return {"type": "attention", "mixer": m}


def gla(heads=2, dim=12, vdim=20, tau=8.0):
  return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff=56):
  return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=8, top=3, scale=1.5, groups=(4, 2), shared=40):
  d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
  if groups is not None:
    d["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
  if shared:
    d["shared"] = {"ff": shared}
  return d


def config(layers, mlps, width=40, vocab=83, eps=1e-5, alpha=1.7, rank=5, max_context=512):
  """An entry of `layers` that is a number repeats that layer with its tensors (`mlps`: ignored there)."""
  out = []
  for layer, mlp in zip(layers, mlps):
    if isinstance(layer, int):
      out.append({**copy.deepcopy(out[layer]), "weights_of": layer})
      continue
    out.append({**copy.deepcopy(layer), "mlp": copy.deepcopy(mlp)})
  return {"architecture": "Pibulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
          "layers": out, "max_context": max_context, "decay_rank": rank}


# Models that differ in every size and switch.  A: every mechanism, layers of both kinds run again with the
# tensors of earlier ones.  B: value heads larger than key heads, one kv head, two taps, a window of another size
# than A's beside one without kept tokens and one that keeps more than a page, one group open of two,
# no shared expert, a layer without a feed-forward, tau of 1.  C: sizes without whole 16-byte groups, five
# taps, as many groups as experts, a window of one token.  D: no groups, no cap, no window, one tap, no
# convolution, a whole head turned, one expert chosen of all, attention first and last.
CONFIG_A = config(
    [attention(), gla(), 0, attention(heads=6, kv_heads=3, window=7, keep_first=5, softcap=4.0, dims=4, conv=4),
     1, gla(heads=3, dim=8, vdim=8, tau=16.0)],
    [moe(), dense(64), None, dense(), None, moe(experts=12, top=4, groups=(3, 2), shared=16, scale=2.5)])
CONFIG_B = config(
    [gla(heads=1, dim=20, vdim=12, tau=1.0), attention(heads=6, kv_heads=1, dim=8, vdim=24, window=9, keep_first=0, conv=2),
     attention(heads=5, kv_heads=5, dim=16, vdim=8, window=20, keep_first=11, dims=16, base=3000.0), 2, 0],
    [dense(32), None, moe(experts=6, top=2, groups=(2, 1), shared=0), None, None], width=48, vocab=131, eps=1e-6,
    alpha=0.8, rank=3)
CONFIG_C = config(
    [attention(heads=3, kv_heads=3, dim=7, vdim=5, window=10, keep_first=2, conv=5, dims=6),
     gla(heads=3, dim=5, vdim=7, tau=3.5), attention(heads=2, kv_heads=1, dim=10, vdim=6, window=1, keep_first=1, dims=2),
     1], [moe(ff=10, experts=5, top=2, groups=(5, 3), shared=14), dense(22), dense(18), None],
    width=36, vocab=50, rank=2, alpha=2.2)
CONFIG_D = config(
    [attention(window=None, softcap=None, conv=1, dims=16), gla(heads=2, dim=16, vdim=16),
     attention(heads=4, kv_heads=4, dim=12, vdim=12, window=33, keep_first=4, conv=None, dims=0), 0],
    [moe(groups=None, top=1, experts=4), moe(top=8, groups=(2, 2)), dense(32), None], width=32, vocab=60, rank=8, alpha=3.0)


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
    elif name.endswith(".conv"):
      draw(name, 0.6)
    elif name.endswith(".a2.b"):
      draw(name, 1.0, 1.0)
    elif name.endswith(".a2"):
      draw(name, 0.5)
    elif name.endswith(".down"):
      draw(name, 0.7 / t[name].shape[1] ** 0.5)
    elif name.endswith(".router"):
      draw(name, 1.5 / cfg_dict["width"] ** 0.5)
    elif name.endswith(".correction"):
      draw(name, 0.5, -0.4)  # choice scores of both signs
  return cfg, t


def _margin(scores, correction, r):
  """How far one token's choice of experts is from another one: the smallest gap between what is chosen and
  what is not, among groups and among experts of open groups."""
  choice, gap = scores + correction, np.inf
  groups = r.get("groups")
  if groups and groups["keep"] < groups["count"]:
    parts = choice.reshape(groups["count"], -1)
    value = np.sort(parts, axis=1)[:, ::-1][:, :2].sum(axis=1)
    order = np.argsort(-value)
    gap = value[order[groups["keep"] - 1]] - value[order[groups["keep"]]]
    choice = parts[order[:groups["keep"]]].reshape(-1)
  if r["top"] < len(choice):
    best = np.sort(choice)[::-1]
    gap = min(gap, best[r["top"] - 1] - best[r["top"]])
  return gap


def tokens(cfg_dict, t, n, seed, margin=0.012, low=0, fixed=None):
  """n random tokens (from `low` on; `fixed`: {place: token}) none of which is a close call for a router: 16-bit
  rounding may turn such a choice, which says nothing about the engine."""
  w = as_numpy(t)
  rng = np.random.default_rng(seed)
  toks = rng.integers(low, cfg_dict["vocab"], n).tolist()
  for at, tok in (fixed or {}).items():
    toks[at] = tok
  real = plain.choose
  for _ in range(400):
    calls, bad = 0, n

    def watched(scores, correction, r):
      nonlocal calls, bad
      if _margin(scores, correction, r) < margin:
        bad = min(bad, calls % n)
      calls += 1
      return real(scores, correction, r)

    plain.choose = watched
    try:
      plain.forward(cfg_dict, w, toks)
    finally:
      plain.choose = real
    while bad < n and fixed and bad in fixed:
      bad -= 1  # (another token before it)
    if bad == n:
      return toks
    toks[bad] = int(rng.integers(low, cfg_dict["vocab"]))
  raise AssertionError("no sequence without close calls found")


def plant_needle(cfg_dict, t, layer, needle, asker, strength=7.0):
  """In a model whose layer `layer` (attention) is its first: makes the key of token `needle` and the query of
  token `asker` point the same way in the last (unturned) dim of every head, so that the score stands out
  however many other keys there are, and gives the needle a value of its own.  The last tap of every
  convolution is one and the others small, so that a token's neighbours hardly matter."""
  m = cfg_dict["layers"][layer]["mixer"]
  p, width = f"l{layer}.mix", cfg_dict["width"]
  gen = torch.Generator().manual_seed(77 + layer)
  h = {}
  for tok, sign in ((needle, 1.0), (asker, -1.0)):
    row = torch.zeros(width)
    row[(7 * tok + 3) % width] = 4.0 * sign
    row[(5 * tok + 1) % width] = 4.0
    t["embed"][tok] = row.to(torch.bfloat16)
    h[tok] = t["embed"][tok].double().numpy()
  for n in "qkv":
    if f"{p}.{n}.conv" in t:
      taps = 0.02 * torch.randn(t[f"{p}.{n}.conv"].shape, generator=gen)
      taps[:, -1] = 1.0
      t[f"{p}.{n}.conv"] = taps.to(torch.bfloat16)
  for n in "qk":
    t[f"{p}.{n}.norm"] = torch.ones_like(t[f"{p}.{n}.norm"])

  def bend(name, rows, by):
    v = t[name].float()
    v[rows] += torch.from_numpy(by).float()
    t[name] = v.to(torch.bfloat16)

  d = m["dim"]
  for g in range(m["kv_heads"]):
    bend(f"{p}.k", g * d + d - 1, strength * h[needle] / (h[needle] @ h[needle]))
  for a in range(m["heads"]):
    bend(f"{p}.q", a * d + d - 1, strength * h[asker] / (h[asker] @ h[asker]))
  v = t[f"{p}.v"].float()
  v += 2.0 * torch.randn(v.shape[0], generator=gen)[:, None] * torch.from_numpy(h[needle]).float()[None, :] / float(h[needle] @ h[needle])
  t[f"{p}.v"] = v.to(torch.bfloat16)
  return t
