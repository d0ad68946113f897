"""Configuration of the Mononex decoder, read from config.json.

config.json of this design:

  architecture     "Mononex"
  vocab, width     sizes of the embedding table and of the residual stream
  norm.eps         eps of every RMS norm
  layers           one entry per layer: `type` ("attention", "latent_attention" or "gla"), `mixer`
                   (its sizes) and `mlp` ({"kind": "dense", "ff"}, or null)
  max_context      (optional, this engine's own key) the longest sequence the engine will serve; the
                   design has no limit
  decay_rank       (optional, this engine's own key) rank of the a1 / a2 pairs where no folder of
                   tensors gives it (random-weights mode)

A layer is x <- x + mixer(shift(norm1(x))) + mlp(norm2(x)), both norms of the same x with scales kept
around zero (block `parallel_residual` with two norms and a token shift).  Tensor names: `embed`,
`l<i>.norm1|norm2|shift`, `l<i>.mix.*`, `l<i>.mlp.up|down`, `final.norm`, `head`.

"attention" (mixer `head_norm_attention` without its norm and rotation): heads, kv_heads, dim, vdim,
scale, mask.size (the chunk: a query sees its own chunk's keys), and optionally kv_from, an earlier
attention layer whose keys and values this one reads.  The scores lose 2^(-8 (h + 1) / heads) per
token of distance, the softmax has a sink, every element a gate.  Tensors q, k, v, sink, g, o.
"latent_attention": heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot.{dims, base, scaling:
{factor, original, fast, slow}} (neighbours pair up; YaRN).  Tensors dq, dq.norm, uq, dkv, dkv.norm, uk,
uv, g, o.
"gla" (mixer `gated_linear_attention`): heads, dim, vdim, tau.  Tensors q, k, v, g, a1, a2, a2.b, norm, o
(the rank of a1 / a2 is the tensors' own).
"""

from __future__ import annotations

import copy
import dataclasses
from typing import Any

from simply_b200.config.gemma2 import ConfigError
from simply_b200.config.model_spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from simply_b200.registry import ARCHITECTURES

_DEFAULT_MAX_CONTEXT = 1 << 17
_MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim"),
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"),
    "gla": ("heads", "dim", "vdim"),
}


def _need(d: dict, key: str, where: str):
  if not isinstance(d, dict) or key not in d or d[key] is None:
    raise ConfigError(f"config.json: {where} lacks {key!r}")
  return d[key]


def _chunk(mixer: dict) -> int | None:
  mask = mixer.get("mask") or {}
  return None if mask.get("size") is None else int(mask["size"])


@dataclasses.dataclass(frozen=True)
class MononexConfig:
  vocab: int
  width: int
  eps: float
  layers: tuple[dict, ...]
  max_context: int = _DEFAULT_MAX_CONTEXT
  decay_rank: int = -1
  bos_token_id: int | None = None
  eos_token_id: int | tuple[int, ...] | None = None

  architecture = "Mononex"

  # ---- reading and writing ------------------------------------------------------
  @classmethod
  def from_dict(cls, d: dict[str, Any]) -> "MononexConfig":
    eos = d.get("eos_token_id")
    if isinstance(eos, list):
      eos = tuple(int(e) for e in eos)
    cfg = cls(
        vocab=int(_need(d, "vocab", "the model")), width=int(_need(d, "width", "the model")),
        eps=float(_need(_need(d, "norm", "the model"), "eps", "norm")),
        layers=tuple(copy.deepcopy(l) for l in _need(d, "layers", "the model")),
        max_context=int(d.get("max_context") or _DEFAULT_MAX_CONTEXT), decay_rank=int(d.get("decay_rank") or -1),
        bos_token_id=d.get("bos_token_id"), eos_token_id=eos)
    cfg.validate()
    return cfg

  def to_dict(self) -> dict[str, Any]:
    d: dict[str, Any] = {
        "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
        "layers": [copy.deepcopy(l) for l in self.layers], "max_context": self.max_context}
    if self.decay_rank > 0:
      d["decay_rank"] = self.decay_rank
    if self.bos_token_id is not None:
      d["bos_token_id"] = self.bos_token_id
    if self.eos_token_id is not None:
      d["eos_token_id"] = list(self.eos_token_id) if isinstance(self.eos_token_id, tuple) else self.eos_token_id
    return d

  def replace(self, **changes: Any) -> "MononexConfig":
    cfg = dataclasses.replace(self, **changes)
    cfg.validate()
    return cfg

  # ---- checks -------------------------------------------------------------------
  def validate(self) -> None:
    if self.vocab <= 0 or self.width <= 0 or self.max_context <= 0:
      raise ConfigError("vocab, width and max_context must be positive")
    if not self.eps > 0:
      raise ConfigError("norm.eps must be positive")
    if not self.layers:
      raise ConfigError("the model has no layers")
    for i, layer in enumerate(self.layers):
      where = f"layer {i}"
      kind = _need(layer, "type", where)
      if kind not in _MIXER_KEYS:
        raise ConfigError(f"{where}: unknown type {kind!r} (known: {', '.join(sorted(_MIXER_KEYS))})")
      m = _need(layer, "mixer", where)
      for key in _MIXER_KEYS[kind]:
        if int(_need(m, key, where)) <= 0:
          raise ConfigError(f"{where}: {key} must be positive")
      if kind == "attention":
        self._check_attention(m, where, i)
      elif kind == "latent_attention":
        _need(m, "scale", where)
        rot = m.get("rot")
        if rot:
          dims = int(_need(rot, "dims", f"{where} (rot)"))
          _need(rot, "base", f"{where} (rot)")
          if dims % 2 or dims < 0 or dims > m["rot_dim"]:
            raise ConfigError(f"{where}: rot.dims must be even and at most rot_dim")
          if rot.get("scaling"):
            for key in ("factor", "original", "fast", "slow"):
              if not float(_need(rot["scaling"], key, f"{where} (rot.scaling)")) > 0:
                raise ConfigError(f"{where}: rot.scaling.{key} must be positive")
      elif not float(_need(m, "tau", where)) > 0:
        raise ConfigError(f"{where}: tau must be positive")
      mlp = layer.get("mlp")
      if mlp is not None:
        if mlp.get("kind") != "dense":
          raise ConfigError(f"{where}: unknown mlp kind {mlp.get('kind')!r} (known: dense)")
        if int(_need(mlp, "ff", f"{where} (mlp)")) <= 0:
          raise ConfigError(f"{where}: ff must be positive")

  def _check_attention(self, m: dict, where: str, index: int) -> None:
    _need(m, "scale", where)
    if m["heads"] % m["kv_heads"]:
      raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
    if _chunk(m) is not None and _chunk(m) <= 0:
      raise ConfigError(f"{where}: mask.size must be positive")
    source = m.get("kv_from")
    if source is None:
      return
    if not 0 <= int(source) < index:
      raise ConfigError(f"{where}: kv_from must name an earlier layer, got {source}")
    other = self.layers[int(source)]
    om = other.get("mixer", {})
    if other.get("type") != "attention" or om.get("kv_from") is not None:
      raise ConfigError(f"{where}: kv_from must name an attention layer with keys and values of its own")
    for key in ("kv_heads", "dim", "vdim"):
      if om.get(key) != m.get(key):
        raise ConfigError(f"{where}: {key} differs from layer {source}, whose cache it reads")

  # ---- derived --------------------------------------------------------------------
  def _mixer_spec(self, i: int, kind: str, m: dict) -> PartSpec:
    p = f"l{i}.mix"
    if kind == "attention":
      readers = tuple(_chunk(l["mixer"]) for l in self.layers
                      if l["type"] == "attention" and l["mixer"].get("kv_from") == i)
      return PartSpec("head_norm_attention", p, {
          "width": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
          "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "score_scale": float(m["scale"]), "eps": self.eps,
          "head_norm": False, "tie_values": False, "output_gate": True, "distance_slopes": True, "sink": True,
          "chunk": _chunk(m), "project_kv": m.get("kv_from") is None, "cache_chunks": readers})
    if kind == "latent_attention":
      rot = m.get("rot")
      rotary = None
      if rot and int(rot["dims"]) > 0:
        rotary = {"dims": int(rot["dims"]), "base": float(rot["base"]), "layout": "neighbours",
                  "scaling": rot.get("scaling")}
      return PartSpec("latent_attention", p, {
          "width": self.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]),
          "rotated_dim": int(m["rot_dim"]), "value_dim": int(m["vdim"]), "query_rank": int(m["q_rank"]),
          "kv_rank": int(m["kv_rank"]), "score_scale": float(m["scale"]), "rotary": rotary, "eps": self.eps,
          "sink": False, "output_gate": True, "gate_per_head": False})
    return PartSpec("gated_linear_attention", p, {
        "width": self.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
        "tau": float(m["tau"]), "eps": self.eps, "decay_rank": self.decay_rank})

  def _mlp_spec(self, i: int, mlp: dict | None) -> PartSpec:
    if mlp is None:
      return PartSpec("none", f"l{i}.mlp")
    return PartSpec("activated", f"l{i}.mlp", {
        "width": self.width, "hidden": int(mlp["ff"]), "activation": "relu_squared"})

  def model_spec(self) -> ModelSpec:
    norm = PartSpec("rms_norm", params={"eps": self.eps, "plus_one": True})
    layers, order = [], []
    for i, layer in enumerate(self.layers):
      p = f"l{i}"
      block = PartSpec("parallel_residual", p, {
          "width": self.width, "norm": norm, "names": {"norm": "norm1", "feed_forward_norm": "norm2"},
          "token_shift": "shift"})
      layers.append(LayerSpec(p, block, self._mixer_spec(i, layer["type"], layer["mixer"]),
                              self._mlp_spec(i, layer.get("mlp"))))
      source = layer["mixer"].get("kv_from") if layer["type"] == "attention" else None
      order.append(LayerCall(p, mixer_cache=None if source is None else f"l{int(source)}#{int(source)}"))
    spec = ModelSpec(
        architecture=self.architecture, vocab_size=self.vocab, width=self.width, max_context=self.max_context,
        embedding=PartSpec("token_embedding", "embed", {
            "vocab_size": self.vocab, "width": self.width, "scale": 1.0, "name": "embed"}),
        layers=tuple(layers), run_order=tuple(order),
        final_norm=PartSpec("rms_norm", "final", {"width": self.width, "eps": self.eps, "plus_one": True,
                                                  "name": "final.norm"}),
        head=PartSpec("linear_head", "head", {"logit_softcap": 0.0, "name": "head"}))
    spec.validate()
    return spec


ARCHITECTURES.register(MononexConfig.architecture, MononexConfig)
