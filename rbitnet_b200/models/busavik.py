"""The Busavik decoder as data: which parts its layers are made of, in which order they run, and its tensor names.

Pre-norm layers, x += mixer(norm1(x)), then (unless "mlp" is null) x += ff(norm2(x)); every norm over the width is
w * tanh(alpha x) + b with a stored number alpha and stored vectors w and b.  After the last layer that norm once more
and a linear head, whose logits are multiplied by logit_scale.  A span of layers ("loop") runs several times in a row with
the same weights; every run has its own cache.

Layer type:
  "latent_attention"  causal softmax attention whose queries come through a latent and whose keys and values come from one
                      cached latent per position, plus a turned key part that all heads share (pairs (i, i + dims/2), slow
                      frequencies stretched), a sigmoid gate per value on the joined heads
Feed-forwards: "dense" (down(gelu(gate h) * up h), gelu in its tanh form, all three with biases) and "moe" (experts
down(silu(gate h) * up h), the chosen experts weighed by the softmax over their logits alone, and a shared expert under a
gate of one number per token).

Tensor names: "embed", "head", "final.norm", "final.norm.b", "final.norm.alpha"; layer i: "l<i>.norm1", "l<i>.norm1.b",
"l<i>.norm1.alpha", the same of "l<i>.norm2", "l<i>.mix.<key>", "l<i>.mlp.<key>", where <key> is the part's weight key
("dq", "dq.norm", "uq", "dkv", "g", "gate.b", "router", "e3.gate", "shared.sg", ...).
"""
from __future__ import annotations

from ..config.base import ConfigError
from ..config.registry import register_architecture
from ..config.busavik import BusavikConfig
from ..parts import PartSpec, BlockSpec, ScheduleEntry, ModelSpec, build_part
from .vaderax import layer_schedule


def _latent(cfg: BusavikConfig, m: dict) -> PartSpec:
    rot = m["rot"]
    return PartSpec("latent_attention", {
        "width": cfg.width, "n_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"], "q_rank": m["q_rank"],
        "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "norm_eps": float(cfg.norm["eps"]), "rot_dim": m["rot_dim"],
        "value_gate": True, "position": {"kind": "rotary", "params": {
            "head_dim": m["rot_dim"], "theta": float(rot["base"]), "pairing": "half", "rot_dim": m["rot_dim"],
            "max_positions": cfg.max_positions, "scaling": rot.get("scaling")}}})


def _feed_forward(cfg: BusavikConfig, mlp: dict) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("gated_dense", {"width": cfg.width, "inner": mlp["ff"], "activation": "gelu_tanh", "bias": True})
    shared = mlp.get("shared")
    return PartSpec("routed_experts", {
        "width": cfg.width, "inner": mlp["expert"]["ff"], "n_experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
        "correction": False, "activation": "silu", "scoring": "softmax_chosen",
        "shared": {"inner": shared["ff"]} if shared else None})


def _norm_names(part: str, prefix: str) -> dict:
    return {f"{part}weight": prefix, f"{part}bias": f"{prefix}.b", f"{part}alpha": f"{prefix}.alpha"}


def build_busavik_spec(cfg: BusavikConfig) -> ModelSpec:
    missing = cfg.missing_sizes()
    if missing:
        raise ConfigError("config.json: " + ", ".join(missing) + ": neither named nor given by a tensor's shape")
    norm = PartSpec("tanh", {"width": cfg.width})
    layers, ignorable = [], []
    for i, layer in enumerate(cfg.layers):
        parts = {"mixer": _latent(cfg, layer["mixer"]), "mixer_norm": norm}
        names = _norm_names("mixer_norm.", f"l{i}.norm1")
        if layer.get("mlp") is not None:
            parts["feed_forward"], parts["ffn_norm"] = _feed_forward(cfg, layer["mlp"]), norm
            names.update(_norm_names("ffn_norm.", f"l{i}.norm2"))
        else:
            ignorable += list(_norm_names("", f"l{i}.norm2").values())
        for part_name, prefix in (("mixer", "mix"), ("feed_forward", "mlp")):
            if part_name in parts:
                for key in build_part(part_name, parts[part_name]).weight_shapes():
                    names[f"{part_name}.{key}"] = f"l{i}.{prefix}.{key}"
        layers.append(BlockSpec(parts=parts, names=names, arrangement="pre_norm"))
    return ModelSpec(
        width=cfg.width, vocab_size=cfg.vocab, embedding_name="embed", layers=layers,
        schedule=[ScheduleEntry(i) for i, _ in layer_schedule(len(layers), cfg.loop)],
        final_norm=norm, final_norm_names=_norm_names("", "final.norm"), head_name="head",
        max_positions=cfg.max_positions, stop_ids=[], logit_scale=float(cfg.logit_scale), ignorable=ignorable)


register_architecture("Busavik", BusavikConfig, build_busavik_spec)
