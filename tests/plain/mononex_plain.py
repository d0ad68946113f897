"""The Mononex decoder, stated plainly in NumPy float64: whole sequences, one function per
mechanism, no code shared with the engine.  The yardstick of tests/test_mononex*.py.

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


def zero_centred_norm(x, weight, eps):
  return unit_rms(x, eps) * (1.0 + weight)


def token_shift(h, weight):
  """Row t moves towards row t - 1 (zeros before the first), channel by channel."""
  before = np.zeros_like(h)
  before[1:] = h[:-1]
  return h + (before - h) * weight


# ---- rotary angles --------------------------------------------------------------------------------
def yarn_frequencies(dims, base, scaling):
  """Angles per position, and the factor on cos and sin."""
  n = dims // 2
  freq = np.array([base ** (-2.0 * i / dims) for i in range(n)])
  if not scaling:
    return freq, 1.0
  factor, original = scaling["factor"], scaling["original"]

  def turns_at(t):  # the (real) index whose frequency makes t turns over `original` positions
    return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

  lo = max(math.floor(turns_at(scaling["fast"])), 0)
  hi = min(math.ceil(turns_at(scaling["slow"])), dims - 1)
  out = np.zeros(n)
  for i in range(n):
    ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
    out[i] = freq[i] / factor * ramp + freq[i] * (1.0 - ramp)
  return out, 0.1 * math.log(factor) + 1.0


def turn_neighbours(x, positions, freq, amplitude):
  """x [T, ..., D]: the pairs (2i, 2i + 1) of the first 2 len(freq) dims turn by position * freq_i."""
  out = x.copy()
  for i, f in enumerate(freq):
    angle = positions * f
    while angle.ndim < x.ndim - 1:
      angle = angle[:, None]
    c, s = amplitude * np.cos(angle), amplitude * np.sin(angle)
    u, v = x[..., 2 * i], x[..., 2 * i + 1]
    out[..., 2 * i] = u * c - v * s
    out[..., 2 * i + 1] = v * c + u * s
  return out


# ---- mixers ---------------------------------------------------------------------------------------
def gated_linear_attention(h, m, w, p, eps):
  """Token by token: the state's rows decay by a number per key channel."""
  heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
  t = h.shape[0]
  q = (h @ w[p + ".q"].T).reshape(t, heads, dim) * dim ** -0.5
  k = (h @ w[p + ".k"].T).reshape(t, heads, dim)
  v = (h @ w[p + ".v"].T).reshape(t, heads, vdim)
  z = (h @ w[p + ".a1"].T) @ w[p + ".a2"].T + w[p + ".a2.b"]
  keep = np.power(sigmoid(z), 1.0 / m["tau"]).reshape(t, heads, dim)
  out = np.zeros((t, heads, vdim))
  for a in range(heads):
    state = np.zeros((dim, vdim))
    for i in range(t):
      state = keep[i, a][:, None] * state + np.outer(k[i, a], v[i, a])
      out[i, a] = state.T @ q[i, a]
  out = unit_rms(out, eps) * w[p + ".norm"]
  g = h @ w[p + ".g"].T
  return (out.reshape(t, heads * vdim) * (g * sigmoid(g))) @ w[p + ".o"].T


def latent_attention(h, m, w, p, eps):
  heads, dim, rdim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
  t = h.shape[0]
  positions = np.arange(t, dtype=np.float64)
  freq, amplitude = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
  cq = unit_rms(h @ w[p + ".dq"].T, eps) * w[p + ".dq.norm"]
  q = (cq @ w[p + ".uq"].T).reshape(t, heads, dim + rdim)
  q_turned = turn_neighbours(q[..., dim:], positions, freq, amplitude)
  down = h @ w[p + ".dkv"].T
  c = unit_rms(down[:, :rank], eps) * w[p + ".dkv.norm"]
  k_turned = turn_neighbours(down[:, rank:], positions, freq, amplitude)
  k = (c @ w[p + ".uk"].T).reshape(t, heads, dim)
  v = (c @ w[p + ".uv"].T).reshape(t, heads, vdim)
  out = np.zeros((t, heads, vdim))
  for i in range(t):
    for a in range(heads):
      s = (k[:i + 1, a] @ q[i, a, :dim] + k_turned[:i + 1] @ q_turned[i, a]) * m["scale"]
      e = np.exp(s - s.max())
      out[i, a] = (e / e.sum()) @ v[:i + 1, a]
  return (out.reshape(t, heads * vdim) * sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def keys_and_values(h, m, w, p):
  t = h.shape[0]
  return ((h @ w[p + ".k"].T).reshape(t, m["kv_heads"], m["dim"]),
          (h @ w[p + ".v"].T).reshape(t, m["kv_heads"], m["vdim"]))


def chunked_attention(h, k, v, m, w, p):
  """Scores lose slope * distance, keys of the query's own chunk only, a sink in the denominator."""
  heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
  per_kv = heads // m["kv_heads"]
  size = (m.get("mask") or {}).get("size")
  t = h.shape[0]
  q = (h @ w[p + ".q"].T).reshape(t, heads, dim)
  out = np.zeros((t, heads, vdim))
  for i in range(t):
    first = (i // size) * size if size else 0
    for a in range(heads):
      slope = 2.0 ** (-8.0 * (a + 1) / heads)
      j = np.arange(first, i + 1)
      s = (k[first:i + 1, a // per_kv] @ q[i, a]) * m["scale"] - slope * (i - j)
      sink = w[p + ".sink"][a]
      top = max(s.max(), sink)
      e = np.exp(s - top)
      out[i, a] = (e @ v[first:i + 1, a // per_kv]) / (e.sum() + math.exp(sink - top))
  return (out.reshape(t, heads * vdim) * sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def squared_relu_mlp(h, w, p):
  return np.maximum(h @ w[p + ".up"].T, 0.0) ** 2 @ w[p + ".down"].T


# ---- the model --------------------------------------------------------------------------------------
def forward(cfg, w, tokens, layer_outputs=None):
  """Logits [T, vocab] of one sequence from its first token on."""
  eps = cfg["norm"]["eps"]
  x = w["embed"][np.asarray(tokens)]
  kept = {}  # layer -> its keys and values
  for i, layer in enumerate(cfg["layers"]):
    p, m = f"l{i}", layer["mixer"]
    h = token_shift(zero_centred_norm(x, w[f"{p}.norm1"], eps), w[f"{p}.shift"])
    if layer["type"] == "gla":
      y = gated_linear_attention(h, m, w, f"{p}.mix", eps)
    elif layer["type"] == "latent_attention":
      y = latent_attention(h, m, w, f"{p}.mix", eps)
    else:
      source = m.get("kv_from")
      if source is None:
        kept[i] = keys_and_values(h, m, w, f"{p}.mix")
      k, v = kept[i if source is None else source]
      y = chunked_attention(h, k, v, m, w, f"{p}.mix")
    if layer.get("mlp") is not None:
      y = y + squared_relu_mlp(zero_centred_norm(x, w[f"{p}.norm2"], eps), w, f"{p}.mlp")
    x = x + y
    if layer_outputs is not None:
      layer_outputs.append(x.copy())
  return zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T
