"""BafulornConfig: the hyper-parameters of the Bafulorn decoder, by config.json key.

config.json names the design under "architecture" and gives

  vocab, width          sizes of the embedding table and of the residual stream
  norm.eps              eps of every norm, inside the mixers too
  residual_mult         multiplies every sublayer's normed result where it is added to the residual stream
  layers                a list, one entry per layer, in order:
      type              "latent_attention", "attention" or "mamba2"
      mixer             "latent_attention": heads, dim, vdim, kv_rank, scale, optional mask {size}
                        "attention": heads, kv_heads, dim, vdim (the keys are the values: vdim is dim), scale, optional rot
                        {base, dims, optional scaling {factor, low, high, original}}, optional mask {size, optional keep_first}
                        "mamba2": heads, vdim, state, groups, conv (taps), norm_groups
      mlp               null, {"kind": "dense", "ff"}, or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top",
                        optional "scale" (1)}, and optionally "shared": {"ff"}}
  max_positions         optional: the longest sequence an engine may be asked to hold (default 131072; nothing in the
                        design depends on it)

Sizes that a model's files also give as a tensor's shape may be left out of config.json: dim ("mix.q"), kv_rank
("mix.dkv.norm"), vdim ("mix.uv" or "mix.norm"), kv_heads ("mix.k"), a mamba2 layer's heads ("mix.A_log"), state and conv
("mix.conv"), mlp.ff ("mlp.gate"), mlp.expert.ff ("mlp.e0.gate"), mlp.router.experts ("mlp.router") and mlp.shared.ff
("mlp.shared.gate"); ``sizes_from_tensors`` fills them in before the model is built.  A configuration from which random
weights are to be made names them all.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import ClassVar, List

from .base import ModelConfig, ConfigError
from .safuvik import _positive_int, _need
from .gozotar import _size, _rot

#: per layer type, the sizes its mixer has (each may also come from a tensor) and the keys it must have besides
_SIZES = {"latent_attention": ("dim", "vdim", "kv_rank"), "attention": ("dim", "vdim", "kv_heads"),
          "mamba2": ("heads", "vdim", "state", "conv")}
_KEYS = {"latent_attention": ("heads", "scale"), "attention": ("heads", "scale"), "mamba2": ("groups", "norm_groups")}


@dataclass
class BafulornConfig(ModelConfig):
    architecture: ClassVar[str] = "Bafulorn"
    required: ClassVar[tuple] = ("vocab", "width", "layers", "norm", "residual_mult")

    vocab: int = 0
    width: int = 0
    layers: List[dict] = field(default_factory=list)
    norm: dict = field(default_factory=dict)
    residual_mult: float = 1.0
    max_positions: int = 131072

    def validate(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _positive_int(self.max_positions, "max_positions")
        _need(self.norm, ("eps",), "norm")
        if not float(self.norm["eps"]) > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        float(self.residual_mult)
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            if layer["type"] not in _SIZES:
                raise ConfigError(f"config.json: {where}.type {layer['type']!r} is not a layer of this design "
                                  f"({', '.join(repr(k) for k in _SIZES)})")
            self._mixer(layer["type"], layer["mixer"], f"{where}.mixer")
            if layer.get("mlp") is not None:
                self._mlp(layer["mlp"], f"{where}.mlp")

    @staticmethod
    def _mixer(kind, m, where):
        _need(m, _KEYS[kind], where)
        for k in _SIZES[kind] + tuple(k for k in _KEYS[kind] if k != "scale"):
            _size(m, k, where)
        mask = m.get("mask")
        if mask is not None and kind != "mamba2":
            _need(mask, ("size",), f"{where}.mask")
            _positive_int(mask["size"], f"{where}.mask.size")
            keep = mask.get("keep_first") or 0
            if kind == "attention" and (not isinstance(keep, int) or isinstance(keep, bool) or keep < 0):
                raise ConfigError(f"config.json: {where}.mask.keep_first must be a whole number, not negative")
        if kind == "attention":
            if m.get("dim") is not None and m.get("vdim") is not None and m["vdim"] != m["dim"]:
                raise ConfigError(f"config.json: {where}: the values are the keys, so vdim equals dim")
            if m.get("kv_heads") is not None and m["heads"] % m["kv_heads"]:
                raise ConfigError(f"config.json: {where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
            rot = m.get("rot")
            if rot is not None:
                _rot(rot, f"{where}.rot", m["dim"] if m.get("dim") is not None else rot.get("dims", 0))
        if kind == "mamba2" and m.get("heads") is not None:
            if m["heads"] % m["groups"]:
                raise ConfigError(f"config.json: {where}: {m['heads']} heads are not a multiple of {m['groups']} groups")
            if m.get("vdim") is not None and (m["heads"] * m["vdim"]) % m["norm_groups"]:
                raise ConfigError(f"config.json: {where}: {m['heads']} heads of {m['vdim']} values are not {m['norm_groups']} "
                                  "equal parts")

    @staticmethod
    def _mlp(mlp, where):
        _need(mlp, ("kind",), where)
        if mlp["kind"] == "dense":
            _size(mlp, "ff", where)
        elif mlp["kind"] == "moe":
            _need(mlp, ("router",), where)
            r = mlp["router"]
            _need(r, ("top",), f"{where}.router")
            _size(mlp.get("expert") or {}, "ff", f"{where}.expert")
            _size(r, "experts", f"{where}.router")
            _positive_int(r["top"], f"{where}.router.top")
            if r.get("experts") is not None and r["top"] > r["experts"]:
                raise ConfigError(f"config.json: {where}.router: top {r['top']} of {r['experts']} experts")
            float(r.get("scale", 1.0))
            if mlp.get("shared") is not None:
                if not isinstance(mlp["shared"], dict):
                    raise ConfigError(f"config.json: {where}.shared must be an object")
                _size(mlp["shared"], "ff", f"{where}.shared")
        else:
            raise ConfigError(f"config.json: {where}.kind {mlp['kind']!r} is not built ('dense', 'moe')")

    def sizes_from_tensors(self, shapes) -> None:
        """Takes from the shapes of a model's tensors (name -> shape) the sizes that config.json does not name."""
        self.layers = copy.deepcopy(self.layers)                  # the caller's dictionaries stay as they are

        def fill(d, key, name, axis=0, parts=1, less=0):
            shape = shapes.get(name)
            if d.get(key) is None and shape is not None and len(shape) > axis and parts:
                d[key] = (int(shape[axis]) - less) // parts
        for i, layer in enumerate(self.layers):
            m, mlp, mix = layer["mixer"], layer.get("mlp"), f"l{i}.mix"
            if layer["type"] == "latent_attention":
                fill(m, "dim", f"{mix}.q", parts=m["heads"])
                fill(m, "vdim", f"{mix}.uv", parts=m["heads"])
                fill(m, "kv_rank", f"{mix}.dkv.norm")
            elif layer["type"] == "attention":
                fill(m, "dim", f"{mix}.q", parts=m["heads"])
                fill(m, "kv_heads", f"{mix}.k", parts=m.get("dim") or 0)
                if m.get("vdim") is None and m.get("dim") is not None:
                    m["vdim"] = m["dim"]
            else:
                fill(m, "heads", f"{mix}.A_log")
                fill(m, "vdim", f"{mix}.norm", parts=m.get("heads") or 0)
                if m.get("heads") is not None and m.get("vdim") is not None:
                    fill(m, "state", f"{mix}.conv", parts=2 * m["groups"], less=m["heads"] * m["vdim"])
                fill(m, "conv", f"{mix}.conv", axis=1)
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
            where, mlp = f"layers[{i}]", layer.get("mlp")
            out += [f"{where}.mixer.{k}" for k in _SIZES[layer["type"]] if layer["mixer"].get(k) is None]
            if mlp is not None and mlp["kind"] == "dense" and mlp.get("ff") is None:
                out.append(f"{where}.mlp.ff")
            if mlp is not None and mlp["kind"] == "moe":
                out += [f"{where}.mlp.{part}.{k}" for part, k in (("expert", "ff"), ("router", "experts"))
                        if (mlp.get(part) or {}).get(k) is None]
                if mlp.get("shared") is not None and mlp["shared"].get("ff") is None:
                    out.append(f"{where}.mlp.shared.ff")
        return out

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": self.norm,
                "residual_mult": self.residual_mult, "layers": self.layers, "max_positions": self.max_positions}
