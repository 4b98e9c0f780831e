"""The Bafulorn decoder as data: which parts its layers are made of, in which order they run, and its tensor names.

The embedded row goes through a norm before the first layer.  Every sublayer has a norm before it and one after it,
x += residual_mult * norm1b(mixer(norm1(x))), then (unless "mlp" is null) x += residual_mult * norm2b(ff(norm2(x))); every
norm over the width is an RMS norm whose stored weight lies around zero (1 + w).  After the last layer that norm once more
and a linear head.

Layer types:
  "latent_attention"  windowed softmax attention without positions whose keys and values come from one cached latent per
                      position, a sigmoid gate per head
  "attention"         grouped attention whose values are its keys before the rotation, projections with biases, a turned
                      prefix with slow frequencies stretched by their wavelength, a window beside which the first positions
                      of the sequence stay visible
  "mamba2"            a state per head with one decay per head and token, behind a short convolution; the gated result under
                      an RMS norm in equal parts
Feed-forwards: "dense" (down(relu(gate h) * up h)) and "moe" (experts down(silu(gate h) * up h); sigmoid scores chosen with a
correction, the chosen scores divided by their sum and scaled; a shared expert without a gate).

Tensor names: "embed", "embed.norm", "final.norm", "head"; layer i: "l<i>.norm1", "l<i>.norm1b", "l<i>.norm2",
"l<i>.norm2b", "l<i>.mix.<key>", "l<i>.mlp.<key>", where <key> is the part's weight key ("q", "q.b", "dkv.norm", "g", "in",
"conv.b", "A_log", "router", "e3.gate", "shared.up", ...).
"""
from __future__ import annotations

from ..config.base import ConfigError
from ..config.registry import register_architecture
from ..config.bafulorn import BafulornConfig
from ..parts import PartSpec, BlockSpec, ScheduleEntry, ModelSpec, build_part
from .gozotar import _rotary

#: added to the sum that the chosen experts' scores are divided by, fixed by the design
_SCORE_FLOOR = 1e-20


def _latent(cfg: BafulornConfig, m: dict) -> PartSpec:
    return PartSpec("latent_attention", {
        "width": cfg.width, "n_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"], "q_rank": 0,
        "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "norm_eps": float(cfg.norm["eps"]), "head_gate": True,
        "window": (m.get("mask") or {}).get("size")})


def _attention(cfg: BafulornConfig, m: dict) -> PartSpec:
    mask = m.get("mask") or {}
    return PartSpec("attention", {
        "width": cfg.width, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
        "scale": float(m["scale"]), "values": "keys", "bias": True, "window": mask.get("size"),
        "keep_first": int(mask.get("keep_first") or 0),
        "position": _rotary(m["rot"], m["dim"], "half", cfg.max_positions) if m.get("rot") else None})


def _state_space(cfg: BafulornConfig, m: dict) -> PartSpec:
    return PartSpec("state_space", {
        "width": cfg.width, "n_heads": m["heads"], "value_dim": m["vdim"], "state_dim": m["state"], "n_groups": m["groups"],
        "taps": m["conv"], "norm_groups": m["norm_groups"], "norm_eps": float(cfg.norm["eps"])})


_MIXERS = {"latent_attention": _latent, "attention": _attention, "mamba2": _state_space}


def _feed_forward(cfg: BafulornConfig, mlp: dict) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("gated_dense", {"width": cfg.width, "inner": mlp["ff"], "activation": "relu"})
    r, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", {
        "width": cfg.width, "inner": mlp["expert"]["ff"], "n_experts": r["experts"], "top": r["top"], "correction": True,
        "activation": "silu", "scoring": "sigmoid", "normalize": _SCORE_FLOOR, "weight_scale": float(r.get("scale", 1.0)),
        "shared": {"inner": shared["ff"], "gate": False} if shared else None})


def build_bafulorn_spec(cfg: BafulornConfig) -> ModelSpec:
    missing = cfg.missing_sizes()
    if missing:
        raise ConfigError("config.json: " + ", ".join(missing) + ": neither named nor given by a tensor's shape")
    base = {"width": cfg.width, "eps": float(cfg.norm["eps"]), "one_plus": True}
    norm, result_norm = PartSpec("rmsnorm", base, role="norm"), \
        PartSpec("rmsnorm", dict(base, multiplier=float(cfg.residual_mult)), role="norm")
    layers, ignorable = [], []
    for i, layer in enumerate(cfg.layers):
        parts = {"mixer": _MIXERS[layer["type"]](cfg, layer["mixer"]), "mixer_norm": norm, "mixer_result_norm": result_norm}
        names = {"mixer_norm.weight": f"l{i}.norm1", "mixer_result_norm.weight": f"l{i}.norm1b"}
        if layer.get("mlp") is not None:
            parts.update({"feed_forward": _feed_forward(cfg, layer["mlp"]), "ffn_norm": norm, "ffn_result_norm": result_norm})
            names.update({"ffn_norm.weight": f"l{i}.norm2", "ffn_result_norm.weight": f"l{i}.norm2b"})
        else:
            ignorable += [f"l{i}.norm2", f"l{i}.norm2b"]
        for part_name, prefix in (("mixer", "mix"), ("feed_forward", "mlp")):
            if part_name in parts:
                for key in build_part(part_name, parts[part_name]).weight_shapes():
                    names[f"{part_name}.{key}"] = f"l{i}.{prefix}.{key}"
        layers.append(BlockSpec(parts=parts, names=names, arrangement="two_norm"))
    return ModelSpec(
        width=cfg.width, vocab_size=cfg.vocab, embedding_name="embed", layers=layers,
        schedule=[ScheduleEntry(i) for i in range(len(layers))],
        final_norm=norm, final_norm_names={"weight": "final.norm"}, head_name="head", max_positions=cfg.max_positions,
        stop_ids=[], ignorable=ignorable, embedding_norm=norm, embedding_norm_names={"weight": "embed.norm"})


register_architecture("Bafulorn", BafulornConfig, build_bafulorn_spec)
