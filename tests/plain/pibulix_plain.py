"""The Pibulix decoder, stated plainly in NumPy float64: whole sequences, one function per
mechanism, no code shared with the engine.  The yardstick of tests/test_pibulix*.py.

`cfg` is config.json as a dictionary, `w` maps tensor names to float64 arrays.  Linear weights are
[out, in].
"""

from __future__ import annotations

import math

import numpy as np


def unit_rms(x, eps):
  return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(x):
  return 1.0 / (1.0 + np.exp(-x))


def gelu_tanh(z):
  return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
  return z * sigmoid(z)


def normed_sum(x, branch, alpha, weight, eps):
  """The stream after a sublayer: the norm of the scaled stream plus the sublayer's result."""
  return unit_rms(alpha * x + branch, eps) * (1.0 + weight)


# ---- gated linear attention -------------------------------------------------------------------------
def key_decays(h, w, p, tau):
  z = (h @ w[p + ".a1"].T) @ w[p + ".a2"].T + w[p + ".a2.b"]
  return sigmoid(z) ** (1.0 / tau)


def gated_linear_attention(h, m, w, p, eps):
  """One token after the other, all heads at once: S <- diag(decay) S + k v^T, then o = S^T q."""
  t, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
  q = (h @ w[p + ".q"].T).reshape(t, heads, dim) / math.sqrt(dim)
  k = (h @ w[p + ".k"].T).reshape(t, heads, dim)
  v = (h @ w[p + ".v"].T).reshape(t, heads, vdim)
  keep = key_decays(h, w, p, m["tau"]).reshape(t, heads, dim)
  state = np.zeros((heads, dim, vdim))
  o = np.zeros((t, heads, vdim))
  for i in range(t):
    state = state * keep[i][:, :, None] + k[i][:, :, None] * v[i][:, None, :]
    o[i] = np.sum(state * q[i][:, :, None], axis=1)
  o = (unit_rms(o, eps) * w[p + ".norm"]).reshape(t, heads * vdim)
  return (o * silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


# ---- attention --------------------------------------------------------------------------------------
def short_convolution(u, taps):
  """u [T, channels], taps [channels, n]: the last tap weighs the token itself."""
  n = taps.shape[1]
  padded = np.concatenate([np.zeros((n - 1, u.shape[1])), u])
  return sum(padded[j:j + u.shape[0]] * taps[:, j] for j in range(n))


def turn_halves(x, positions, dims, base):
  """x [T, heads, D]: dim i turns together with dim i + dims / 2."""
  out, half = x.copy(), dims // 2
  for i in range(half):
    angle = (positions * base ** (-2.0 * i / dims))[:, None]
    c, s = np.cos(angle), np.sin(angle)
    u, v = x[..., i], x[..., i + half]
    out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
  return out


def sees(i, j, mask):
  """Whether the query at i sees the key at j."""
  if j > i:
    return False
  return mask is None or i - j < mask["size"] or j < mask.get("keep_first", 0)


def head_vectors(h, m, w, p, eps):
  """Queries and keys (convolved, normed per head, turned) and values (convolved)."""
  t = h.shape[0]
  heads = {"q": m["heads"], "k": m["kv_heads"], "v": m["kv_heads"]}
  size = {"q": m["dim"], "k": m["dim"], "v": m["vdim"]}
  out = {}
  for n in "qkv":
    u = h @ w[f"{p}.{n}"].T
    if m.get("conv"):
      u = short_convolution(u, w[f"{p}.{n}.conv"])
    out[n] = u.reshape(t, heads[n], size[n])
  rot = m.get("rot")
  for n in "qk":
    out[n] = unit_rms(out[n], eps) * w[f"{p}.{n}.norm"]
    if rot:
      out[n] = turn_halves(out[n], np.arange(t, dtype=np.float64), rot["dims"], rot["base"])
  return out["q"], out["k"], out["v"]


def attend(q, k, v, m, first=0):
  """q: the queries of positions first, first + 1, ...; k, v from position 0.  A one joins the
  denominator of every softmax."""
  per = m["heads"] // m["kv_heads"]
  cap, mask = m.get("softcap"), m.get("mask")
  out = np.zeros(q.shape[:2] + (v.shape[2],))
  for r in range(q.shape[0]):
    i = first + r
    seen = [j for j in range(i + 1) if sees(i, j, mask)]
    k_seen, v_seen = k[seen], v[seen]
    for a in range(m["heads"]):
      s = (k_seen[:, a // per] @ q[r, a]) * m["scale"]
      if cap:
        s = cap * np.tanh(s / cap)
      top = max(float(s.max()), 0.0)
      e = np.exp(s - top)
      out[r, a] = (e / (math.exp(-top) + e.sum())) @ v_seen[:, a // per]
  return out


def attention(h, m, w, p, eps):
  q, k, v = head_vectors(h, m, w, p, eps)
  return attend(q, k, v, m).reshape(h.shape[0], -1) @ w[p + ".o"].T


# ---- feed-forwards ------------------------------------------------------------------------------------
def gated_mlp(h, act, w, p):
  return (act(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def choose(scores, correction, r):
  """One token: the chosen experts (best first) and their weights."""
  choice = scores + correction
  n = len(scores)
  groups = r.get("groups")
  if groups:
    size = n // groups["count"]
    value = [np.sort(choice[g * size:(g + 1) * size])[::-1][:2].sum() for g in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda g: (-value[g], g))[:groups["keep"]]
    choice = np.array([choice[e] if e // size in kept else -np.inf for e in range(n)])
  best = sorted(range(n), key=lambda e: (-choice[e], e))[:r["top"]]
  s = scores[best]
  return best, s / (s.sum() + 1e-20) * r.get("scale", 1.0)


def expert_mlp(h, mlp, w, p):
  r = mlp["router"]
  scores = sigmoid(h @ w[p + ".router"].T)
  y = np.zeros_like(h)
  for t in range(h.shape[0]):
    for e, a in zip(*choose(scores[t], w[p + ".correction"], r)):
      y[t] += a * gated_mlp(h[t:t + 1], silu, w, f"{p}.e{e}")[0]
  if mlp.get("shared"):
    y += sigmoid(h @ w[p + ".shared.sg"].T) * gated_mlp(h, silu, w, p + ".shared")
  return y


# ---- the model ------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, layer_outputs=None):
  """Logits [T, vocab] of one sequence from its first token on."""
  eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
  x = w["embed"][np.asarray(tokens)]
  for i, layer in enumerate(cfg["layers"]):
    at = i
    while cfg["layers"][at].get("weights_of") is not None:
      at = cfg["layers"][at]["weights_of"]
    p, m, mlp = f"l{at}", layer["mixer"], layer.get("mlp")
    mixer = gated_linear_attention if layer["type"] == "gla" else attention
    x = normed_sum(x, mixer(x, m, w, f"{p}.mix", eps), alpha, w[f"{p}.norm1"], eps)
    if mlp is not None:
      y = gated_mlp(x, gelu_tanh, w, f"{p}.mlp") if mlp["kind"] == "dense" else expert_mlp(x, mlp, w, f"{p}.mlp")
      x = normed_sum(x, y, alpha, w[f"{p}.norm2"], eps)
    if layer_outputs is not None:
      layer_outputs.append(x.copy())
  return (unit_rms(x, eps) * (1.0 + w["final.norm"])) @ w["head"].T
