"""Configuration of the Pibulix decoder, read from config.json.

config.json of this design:

  architecture     "Pibulix"
  vocab, width     sizes of the embedding table and of the residual stream
  norm.eps         eps of every RMS norm
  postln_alpha     a: the stream's factor in the sums below
  layers           one entry per layer: `type` ("attention" or "gla"), `mixer` (its sizes), `mlp` (a
                   feed-forward, or null) and optionally `weights_of`, an index of another layer whose
                   tensors this one uses (the rest of the entry repeats that layer's; the cache or
                   state is its own)
  max_context      (optional, this engine's own key) the longest sequence the engine will serve; the
                   design has no limit
  decay_rank       (optional, this engine's own key) rank of the a1 / a2 pairs where no folder of
                   tensors gives it (random-weights mode)

A layer is x <- norm1(a x + mixer(x)), then x <- norm2(a x + mlp(x)) (block `normed_sum`, scales kept
around zero).  Tensor names: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.

"gla" (mixer `gated_linear_attention`): heads, dim, vdim, tau.  Tensors q, k, v, g, a1, a2, a2.b, norm, o
(the rank of a1 / a2 is the tensors' own).
"attention" (mixer `head_norm_attention`): heads, kv_heads, dim, vdim, scale, and optionally conv (taps of
the convolutions on q, k and v), softcap, rot.{dims, base} (halves pair up), mask.{size, keep_first} (a
window, and the first tokens that stay visible behind it).  The softmax's denominator holds a one.
Tensors q, k, v, q.norm, k.norm, q.conv, k.conv, v.conv, o.
mlp {"kind": "dense", "ff"} (feed-forward `gated`, gelu): tensors gate, up, down.  {"kind": "moe", "expert":
{"ff"}, "router": {"experts", "top", "scale", "groups": {"count", "keep"} or absent}, "shared": {"ff"} or
absent} (feed-forward `routed_experts`, silu): tensors e<j>.{gate,up,down}, router, correction,
shared.{gate,up,down,sg}.
"""

from __future__ import annotations

import copy
import dataclasses
from typing import Any

from simply_b200.config.gemma2 import ConfigError
from simply_b200.config.model_spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from simply_b200.registry import ARCHITECTURES

_DEFAULT_MAX_CONTEXT = 1 << 17
_MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim"), "gla": ("heads", "dim", "vdim")}


def _need(d: dict, key: str, where: str):
  if not isinstance(d, dict) or key not in d or d[key] is None:
    raise ConfigError(f"config.json: {where} lacks {key!r}")
  return d[key]


def _positive(d: dict, key: str, where: str) -> int:
  if int(_need(d, key, where)) <= 0:
    raise ConfigError(f"{where}: {key} must be positive")
  return int(d[key])


@dataclasses.dataclass(frozen=True)
class PibulixConfig:
  vocab: int
  width: int
  eps: float
  alpha: float
  layers: tuple[dict, ...]
  max_context: int = _DEFAULT_MAX_CONTEXT
  decay_rank: int = -1
  bos_token_id: int | None = None
  eos_token_id: int | tuple[int, ...] | None = None

  architecture = "Pibulix"

  # ---- reading and writing ------------------------------------------------------
  @classmethod
  def from_dict(cls, d: dict[str, Any]) -> "PibulixConfig":
    eos = d.get("eos_token_id")
    if isinstance(eos, list):
      eos = tuple(int(e) for e in eos)
    cfg = cls(
        vocab=int(_need(d, "vocab", "the model")), width=int(_need(d, "width", "the model")),
        eps=float(_need(_need(d, "norm", "the model"), "eps", "norm")),
        alpha=float(_need(d, "postln_alpha", "the model")),
        layers=tuple(copy.deepcopy(l) for l in _need(d, "layers", "the model")),
        max_context=int(d.get("max_context") or _DEFAULT_MAX_CONTEXT), decay_rank=int(d.get("decay_rank") or -1),
        bos_token_id=d.get("bos_token_id"), eos_token_id=eos)
    cfg.validate()
    return cfg

  def to_dict(self) -> dict[str, Any]:
    d: dict[str, Any] = {
        "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
        "postln_alpha": self.alpha, "layers": [copy.deepcopy(l) for l in self.layers],
        "max_context": self.max_context}
    if self.decay_rank > 0:
      d["decay_rank"] = self.decay_rank
    if self.bos_token_id is not None:
      d["bos_token_id"] = self.bos_token_id
    if self.eos_token_id is not None:
      d["eos_token_id"] = list(self.eos_token_id) if isinstance(self.eos_token_id, tuple) else self.eos_token_id
    return d

  def replace(self, **changes: Any) -> "PibulixConfig":
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
        _positive(m, key, where)
      if kind == "attention":
        self._check_attention(m, where)
      elif not float(_need(m, "tau", where)) > 0:
        raise ConfigError(f"{where}: tau must be positive")
      if layer.get("mlp") is not None:
        self._check_mlp(layer["mlp"], where)
    for i in range(len(self.layers)):
      self._owner(i)

  @staticmethod
  def _check_attention(m: dict, where: str) -> None:
    _need(m, "scale", where)
    if m["heads"] % m["kv_heads"]:
      raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
    if int(m.get("conv") or 0) < 0:
      raise ConfigError(f"{where}: conv must not be negative")
    rot = m.get("rot")
    if rot:
      dims = int(_need(rot, "dims", f"{where} (rot)"))
      _need(rot, "base", f"{where} (rot)")
      if dims % 2 or not 0 <= dims <= m["dim"]:
        raise ConfigError(f"{where}: rot.dims must be even and at most dim")
    mask = m.get("mask")
    if mask:
      _positive(mask, "size", f"{where} (mask)")
      if int(mask.get("keep_first") or 0) < 0:
        raise ConfigError(f"{where} (mask): keep_first must not be negative")

  @staticmethod
  def _check_mlp(mlp: dict, where: str) -> None:
    if mlp.get("kind") == "dense":
      _positive(mlp, "ff", f"{where} (mlp)")
      return
    if mlp.get("kind") != "moe":
      raise ConfigError(f"{where}: unknown mlp kind {mlp.get('kind')!r} (known: dense, moe)")
    _positive(_need(mlp, "expert", f"{where} (mlp)"), "ff", f"{where} (expert)")
    r = _need(mlp, "router", f"{where} (mlp)")
    experts, top = _positive(r, "experts", f"{where} (router)"), _positive(r, "top", f"{where} (router)")
    groups = r.get("groups") or {"count": 1, "keep": 1}
    count, keep = _positive(groups, "count", f"{where} (groups)"), _positive(groups, "keep", f"{where} (groups)")
    if experts % count or keep > count:
      raise ConfigError(f"{where}: groups.count must divide the experts, and groups.keep be at most the count")
    if top > experts // count * keep:
      raise ConfigError(f"{where}: the kept groups have fewer experts than each token uses")
    if mlp.get("shared"):
      _positive(mlp["shared"], "ff", f"{where} (shared)")

  def _owner(self, index: int) -> int:
    """The layer whose tensors layer `index` uses (itself, as a rule)."""
    at, steps = index, 0
    while self.layers[at].get("weights_of") is not None:
      source = int(self.layers[at]["weights_of"])
      if not 0 <= source < len(self.layers) or steps == len(self.layers):
        raise ConfigError(f"layer {index}: weights_of must lead to a layer with tensors of its own")
      for key in ("type", "mixer", "mlp"):
        if self.layers[source].get(key) != self.layers[at].get(key):
          raise ConfigError(f"layer {at}: {key} differs from layer {source}, whose tensors it uses")
      at, steps = source, steps + 1
    return at

  # ---- derived --------------------------------------------------------------------
  def _mixer_spec(self, p: str, kind: str, m: dict) -> PartSpec:
    if kind == "gla":
      return PartSpec("gated_linear_attention", f"{p}.mix", {
          "width": self.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
          "tau": float(m["tau"]), "eps": self.eps, "decay_rank": self.decay_rank})
    rot, mask = m.get("rot"), m.get("mask") or {}
    rotary = None
    if rot and int(rot["dims"]) > 0:
      rotary = {"dims": int(rot["dims"]), "base": float(rot["base"]), "layout": "halves"}
    return PartSpec("head_norm_attention", f"{p}.mix", {
        "width": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
        "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "score_scale": float(m["scale"]), "eps": self.eps,
        "score_softcap": float(m.get("softcap") or 0.0), "rotary": rotary, "head_norm": True, "head_norm_scale": True,
        "tie_values": False, "output_gate": False, "unit_sink": True, "conv_taps": int(m.get("conv") or 0),
        "window": int(mask["size"]) if mask else None, "keep_first": int(mask.get("keep_first") or 0)})

  def _mlp_spec(self, p: str, mlp: dict | None) -> PartSpec:
    if mlp is None:
      return PartSpec("none", f"{p}.mlp")
    if mlp["kind"] == "dense":
      return PartSpec("gated", f"{p}.mlp", {
          "width": self.width, "hidden": int(mlp["ff"]), "activation": "gelu_tanh",
          "names": {"gate": "gate", "up": "up", "down": "down"}})
    r, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups")
    return PartSpec("routed_experts", f"{p}.mlp", {
        "width": self.width, "hidden": int(mlp["expert"]["ff"]), "num_experts": int(r["experts"]), "top": int(r["top"]),
        "weight_scale": float(r.get("scale", 1.0)), "activation": "silu", "score": "sigmoid", "correction": True,
        "renormalize": True, "shared_hidden": int(shared["ff"]) if shared else 0, "shared_gate": bool(shared),
        "groups": (int(groups["count"]), int(groups["keep"])) if groups else None})

  def model_spec(self) -> ModelSpec:
    norm = PartSpec("rms_norm", params={"eps": self.eps, "plus_one": True})
    layers = []
    for i, layer in enumerate(self.layers):
      if self._owner(i) != i:
        continue
      p = f"l{i}"
      block = PartSpec("normed_sum", p, {
          "width": self.width, "norm": norm, "stream_scale": self.alpha,
          "names": {"mixer_norm": "norm1", "feed_forward_norm": "norm2"}})
      layers.append(LayerSpec(p, block, self._mixer_spec(p, layer["type"], layer["mixer"]),
                              self._mlp_spec(p, layer.get("mlp"))))
    spec = ModelSpec(
        architecture=self.architecture, vocab_size=self.vocab, width=self.width, max_context=self.max_context,
        embedding=PartSpec("token_embedding", "embed", {
            "vocab_size": self.vocab, "width": self.width, "scale": 1.0, "name": "embed"}),
        layers=tuple(layers), run_order=tuple(LayerCall(f"l{self._owner(i)}") for i in range(len(self.layers))),
        final_norm=PartSpec("rms_norm", "final", {"width": self.width, "eps": self.eps, "plus_one": True,
                                                  "name": "final.norm"}),
        head=PartSpec("linear_head", "head", {"logit_softcap": 0.0, "name": "head"}))
    spec.validate()
    return spec


ARCHITECTURES.register(PibulixConfig.architecture, PibulixConfig)
