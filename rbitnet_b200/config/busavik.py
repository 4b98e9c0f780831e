"""BusavikConfig: the hyper-parameters of the Busavik decoder, by config.json key.

config.json names the design under "architecture" and gives

  vocab, width          sizes of the embedding table and of the residual stream
  norm.eps              eps of the RMS norms on the attention's latents (the norms over the width have none)
  logit_scale           multiplies the logits
  layers                a list, one entry per layer, in order:
      type              "latent_attention"
      mixer             heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims, optional scaling {factor,
                        original, fast, slow}}; rot.dims is rot_dim
      mlp               null, {"kind": "dense", "ff"}, or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"},
                        and optionally "shared": {"ff"}}
  loop                  optional {"start", "stop", "times"}: layers start .. stop-1 run `times` times in a row
  max_positions         optional: the longest sequence an engine may be asked to hold (default 131072; nothing in the
                        design depends on it)

Sizes that a model's files also give as a tensor's shape may be left out of config.json: mixer.q_rank ("mix.dq.norm"),
mixer.kv_rank ("mix.dkv.norm"), mixer.vdim ("mix.g"), mlp.ff ("mlp.gate"), mlp.expert.ff ("mlp.e0.gate"),
mlp.router.experts ("mlp.router") and mlp.shared.ff ("mlp.shared.gate"); ``sizes_from_tensors`` fills them in before the
model is built.  A configuration from which random weights are to be made names them all.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import ClassVar, List, Optional

from .base import ModelConfig, ConfigError
from .safuvik import _positive_int, _need
from .gozotar import _size


@dataclass
class BusavikConfig(ModelConfig):
    architecture: ClassVar[str] = "Busavik"
    required: ClassVar[tuple] = ("vocab", "width", "layers", "norm", "logit_scale")

    vocab: int = 0
    width: int = 0
    layers: List[dict] = field(default_factory=list)
    norm: dict = field(default_factory=dict)
    logit_scale: float = 1.0
    loop: Optional[dict] = None
    max_positions: int = 131072

    def validate(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _positive_int(self.max_positions, "max_positions")
        _need(self.norm, ("eps",), "norm")
        if not float(self.norm["eps"]) > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        float(self.logit_scale)
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            if layer["type"] != "latent_attention":
                raise ConfigError(f"config.json: {where}.type {layer['type']!r} is not a layer of this design ('latent_attention')")
            self._mixer(layer["mixer"], f"{where}.mixer")
            if layer.get("mlp") is not None:
                self._mlp(layer["mlp"], f"{where}.mlp")
        if self.loop:
            _need(self.loop, ("start", "stop", "times"), "loop")
            a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
            _positive_int(times, "loop.times")
            if not (isinstance(a, int) and isinstance(b, int) and 0 <= a < b <= len(self.layers)):
                raise ConfigError(f"config.json: loop {a}..{b} does not name layers of the {len(self.layers)}")

    @staticmethod
    def _mixer(m, where):
        _need(m, ("heads", "dim", "rot_dim", "scale", "rot"), where)
        for k in ("heads", "dim", "rot_dim"):
            _positive_int(m[k], f"{where}.{k}")
        for k in ("vdim", "q_rank", "kv_rank"):
            _size(m, k, where)
        if m["rot_dim"] % 2:
            raise ConfigError(f"config.json: {where}.rot_dim must be even")
        rot = m["rot"]
        _need(rot, ("base",), f"{where}.rot")
        if rot.get("dims", m["rot_dim"]) != m["rot_dim"]:
            raise ConfigError(f"config.json: {where}.rot.dims must equal rot_dim")
        if not float(rot["base"]) > 0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive")
        sc = rot.get("scaling")
        if sc is not None:
            _need(sc, ("factor", "original", "fast", "slow"), f"{where}.rot.scaling")
            if not min(float(sc[k]) for k in ("factor", "original", "fast", "slow")) > 0:
                raise ConfigError(f"config.json: {where}.rot.scaling: factor, original, fast and slow must be positive")

    @staticmethod
    def _mlp(mlp, where):
        _need(mlp, ("kind",), where)
        if mlp["kind"] == "dense":
            _size(mlp, "ff", where)
        elif mlp["kind"] == "moe":
            _need(mlp, ("router",), where)
            _need(mlp["router"], ("top",), f"{where}.router")
            _size(mlp.get("expert") or {}, "ff", f"{where}.expert")
            _size(mlp["router"], "experts", f"{where}.router")
            _positive_int(mlp["router"]["top"], f"{where}.router.top")
            if mlp["router"].get("experts") is not None and mlp["router"]["top"] > mlp["router"]["experts"]:
                raise ConfigError(f"config.json: {where}.router: top {mlp['router']['top']} of {mlp['router']['experts']} experts")
            if mlp.get("shared") is not None:
                if not isinstance(mlp["shared"], dict):
                    raise ConfigError(f"config.json: {where}.shared must be an object")
                _size(mlp["shared"], "ff", f"{where}.shared")
        else:
            raise ConfigError(f"config.json: {where}.kind {mlp['kind']!r} is not built ('dense', 'moe')")

    def sizes_from_tensors(self, shapes) -> None:
        """Takes from the shapes of a model's tensors (name -> shape) the sizes that config.json does not name."""
        self.layers = copy.deepcopy(self.layers)                  # the caller's dictionaries stay as they are

        def fill(d, key, name, parts=1):
            shape = shapes.get(name)
            if d.get(key) is None and shape is not None and len(shape) >= 1:
                d[key] = int(shape[0]) // parts
        for i, layer in enumerate(self.layers):
            m, mlp = layer["mixer"], layer.get("mlp")
            fill(m, "q_rank", f"l{i}.mix.dq.norm")
            fill(m, "kv_rank", f"l{i}.mix.dkv.norm")
            fill(m, "vdim", f"l{i}.mix.g", m["heads"])
            if mlp is not None and mlp["kind"] == "dense":
                fill(mlp, "ff", f"l{i}.mlp.gate")
            elif mlp is not None:
                mlp["expert"] = dict(mlp.get("expert") or {})
                fill(mlp["expert"], "ff", f"l{i}.mlp.e0.gate")
                fill(mlp["router"], "experts", f"l{i}.mlp.router")
                if mlp.get("shared") is not None:
                    fill(mlp["shared"], "ff", f"l{i}.mlp.shared.gate")
        self.validate()

    def missing_sizes(self):
        """Names of the sizes that neither config.json nor a tensor has given."""
        out = []
        for i, layer in enumerate(self.layers):
            where, m, mlp = f"layers[{i}]", layer["mixer"], layer.get("mlp")
            out += [f"{where}.mixer.{k}" for k in ("vdim", "q_rank", "kv_rank") if m.get(k) is None]
            if mlp is not None and mlp["kind"] == "dense" and mlp.get("ff") is None:
                out.append(f"{where}.mlp.ff")
            if mlp is not None and mlp["kind"] == "moe":
                out += [f"{where}.mlp.{part}.{k}" for part, k in (("expert", "ff"), ("router", "experts"))
                        if (mlp.get(part) or {}).get(k) is None]
                if mlp.get("shared") is not None and mlp["shared"].get("ff") is None:
                    out.append(f"{where}.mlp.shared.ff")
        return out

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": self.norm,
             "logit_scale": self.logit_scale, "layers": self.layers, "max_positions": self.max_positions}
        if self.loop:
            d["loop"] = self.loop
        return d
