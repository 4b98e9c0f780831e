"""Small Bafulorn configurations for the tests and random weights for them.

The configurations differ from one another in every size and option: layer order, layers without feed-forward, windows of one
position, shorter and longer than a page and none, kept first positions (none, a few, more than a page, more than the
window), grouped and single key heads, whole heads and a prefix turned, with and without stretched frequencies, latents smaller
and larger than a head, one and several groups, heads per group, norm parts and taps, states smaller and larger than a
head, one and several choices among the experts, every expert chosen, with and without a shared expert, sizes that the
tensor-core kernels take and refuse.
"""
from __future__ import annotations

import torch

from rbitnet_b200.config import config_from_dict
from rbitnet_b200.config.registry import get_architecture
from rbitnet_b200.weights import random_tensors


def latent_layer(heads, dim, vdim, kv_rank, window, scale, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def attention_layer(heads, kv, dim, window, keep, scale, rot_dims, mlp=None, base=1000.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mamba_layer(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                                    "norm_groups": norm_groups}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None, scale=1.0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def model(vocab, width, layers, mult=0.5, eps=1e-5):
    return {"architecture": "Bafulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": layers}


#: every mixer, dense and routed feed-forwards and none; windows and kept positions inside one page
CFG_A = model(96, 64, [
    attention_layer(4, 2, 24, 21, 5, 0.3, 16, dense(48), base=100.0, scaling=(4.0, 1.0, 4.0, 40)),
    mamba_layer(4, 16, 8, 2, 4, 2, moe(6, 2, 24, shared=40, scale=1.7)),
    latent_layer(3, 16, 24, 40, 33, 0.35, None),
    mamba_layer(2, 24, 20, 1, 3, 1, dense(72))], mult=0.4)

#: sizes that the tensor-core kernels refuse; one expert chosen and all of them; a window of one position, kept positions
#: beyond the window, one tap, five taps; one norm part per head
CFG_B = model(70, 50, [
    mamba_layer(3, 7, 5, 3, 5, 3, moe(3, 1, 18)),
    latent_layer(2, 10, 7, 13, 70, 0.4, moe(4, 4, 10, shared=6, scale=0.5)),
    attention_layer(2, 2, 10, 6, 11, 0.4, 10, dense(30), base=20.0),
    mamba_layer(5, 6, 11, 1, 1, 5, None),
    attention_layer(3, 1, 6, 1, 3, 0.5, 2, moe(5, 3, 14))], mult=1.0, eps=1e-6)

#: sizes the tensor-core kernels take; kept positions over more than one page; no window at all
CFG_C = model(128, 128, [
    mamba_layer(8, 32, 64, 2, 4, 4, dense(160)),
    latent_layer(4, 32, 64, 128, 65, 0.17, moe(8, 3, 32, shared=64, scale=2.5)),
    attention_layer(8, 2, 64, 64, 70, 0.12, 64, moe(16, 4, 48, scale=1.5), base=50000.0, scaling=(8.0, 1.0, 4.0, 64)),
    latent_layer(8, 16, 16, 64, None, 0.25, dense(96)),
    attention_layer(4, 4, 16, None, 0, 0.25, 8, None)], mult=0.3)

#: a state larger than a chunk's tile of rows and heads wider than a tile of columns; no rotation; windows of whole pages
CFG_D = model(60, 48, [
    mamba_layer(2, 72, 80, 1, 2, 2, None),
    attention_layer(2, 1, 32, 128, 64, 0.2, 0, dense(40)),
    mamba_layer(4, 8, 130, 4, 4, 1, moe(5, 2, 16, shared=8)),
    latent_layer(1, 64, 8, 16, 128, 0.15, None)], mult=0.7)

CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}


def random_config(seed):
    """A configuration whose every size, option and layer order is drawn from ``seed``."""
    import random
    r = random.Random(seed)
    pick = r.choice

    def ff():
        kind = r.random()
        if kind < 0.2:
            return None
        if kind < 0.5:
            return dense(pick([24, 72, 128, 200]))
        experts = pick([2, 5, 8, 12, 33])
        return moe(experts, r.randint(1, min(experts, 6)), pick([8, 24, 40, 64]), shared=pick([None, 16, 72]), scale=pick([1.0, 0.5, 3.0]))

    def layer():
        kind, window = pick(["mamba2", "latent_attention", "attention"]), pick([None, 1, 2, 7, 30, 63, 64, 65, 90])
        if kind == "mamba2":
            groups = pick([1, 2, 3])
            heads = groups * pick([1, 2, 4])
            return mamba_layer(heads, pick([5, 8, 16, 24, 64, 80]), pick([4, 12, 16, 32, 64, 96, 128]), groups, pick([1, 2, 3, 4, 5]),
                               pick([1, heads, groups]), ff())
        if kind == "latent_attention":
            dim = pick([8, 16, 32, 40, 64])
            return latent_layer(pick([1, 2, 3, 4, 8, 16]), dim, pick([8, 16, 24, 64, 128]), pick([8, 24, 48, 64, 96, 128, 192]), window,
                                dim ** -0.5 * pick([1.0, 1.5]), ff())
        dim, kv = pick([8, 16, 20, 32, 64, 128]), pick([1, 2, 3])
        sc = (pick([2.0, 4.0, 16.0]), pick([1.0, 2.0]), 4.0, pick([16, 64, 256])) if r.random() < 0.6 else None
        return attention_layer(kv * pick([1, 2, 4]), kv, dim, window, pick([0, 1, 6, 40, 64, 65]), dim ** -0.5 * pick([1.0, 1.5]),
                               pick([dim, dim // 2, 0]), ff(), base=pick([50.0, 10000.0, 500000.0]), scaling=sc)
    return model(pick([64, 100, 257]), pick([48, 64, 100, 128, 192]), [layer() for _ in range(r.randint(1, 5))],
                 pick([0.2, 0.5, 1.0]), pick([1e-5, 1e-6]))


def spec_of(cfg_dict):
    cfg = config_from_dict(cfg_dict)
    return get_architecture(cfg.architecture).build_spec(cfg)


def make_tensors(cfg_dict, seed, spread=8.0):
    """Random weights, then made so that faults show: matrices are scaled up (random weights of deviation 0.02 give nearly
    uniform attention, gates stuck at one half and a router without preferences); norm weights are spread around zero; biases
    matter; the states forget slowly in some heads and fast in others, so that a token far back still moves the logits."""
    t = random_tensors(spec_of(cfg_dict), seed)
    g = torch.Generator().manual_seed(seed + 1000)
    out = {}
    for name in sorted(t):
        v = t[name].clone()
        if name.endswith(".router"):
            v = v * (2.0 / (0.02 * v.shape[-1] ** 0.5))
        elif name.endswith(".correction"):
            v = v * 10.0
        elif name.endswith(".conv"):
            v = v + 0.3 * torch.randn(v.shape, generator=g)
        elif name.endswith(".A_log"):
            v = torch.linspace(-4.0, 0.5, v.shape[0]) + v
        elif name.endswith(".dt_bias"):
            v = torch.randn(v.shape, generator=g) * 0.5 - 0.5
        elif name.endswith(".b"):
            v = v * 20.0
        elif v.dim() >= 2 and name != "embed":
            v = v * (spread / 8.0 * 1.15 / (0.02 * v.shape[-1] ** 0.5))      # rows of deviation one come out a little larger
        elif v.dim() == 1:
            v = float(v.mean() > 0.5) + 0.3 * torch.randn(v.shape, generator=g)     # around one, or around zero
        out[name] = v.to(torch.bfloat16).to(torch.float32)        # values both dtypes of the engine can hold
    return out
