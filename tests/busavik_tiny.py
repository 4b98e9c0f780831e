"""Small Busavik configurations for the tests and random weights for them.

The configurations differ from one another in every size and option: layer order, layers without feed-forward, a loop over
a part of the layers, over all of them and none, query and key latents smaller and larger than a head and than one
another, turned parts of two values and of a whole head, with and without stretched frequencies, values narrower and
wider than keys, one and several heads, one and several choices among the experts, every expert chosen, with and without a
shared expert, sizes that the tensor-core kernels take and refuse.
"""
from __future__ import annotations

import torch

from rbitnet_b200.config import config_from_dict
from rbitnet_b200.config.registry import get_architecture
from rbitnet_b200.weights import random_tensors


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mlp=None, base=10000.0, scaling=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": rot}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def model(vocab, width, layers, loop=None, logit_scale=0.5, eps=1e-5):
    cfg = {"architecture": "Busavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
           "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


#: a dense layer, one of experts and one without feed-forward, the last two run twice; sequences longer than `original`
CFG_A = model(96, 64, [
    latent_layer(3, 16, 8, 24, 20, 40, 0.3, dense(48), base=1000.0, scaling=(4.0, 16, 8.0, 1.0)),
    latent_layer(3, 16, 8, 24, 24, 16, 0.35, moe(6, 2, 24, shared=40), base=300.0, scaling=(8.0, 32, 4.0, 0.5)),
    latent_layer(2, 8, 8, 8, 12, 24, 0.4, None, base=50.0)], loop=(1, 3, 2))

#: sizes that the tensor-core products refuse; one expert chosen, and all of them; no shared expert; no loop
CFG_B = model(70, 50, [
    latent_layer(2, 10, 6, 7, 9, 13, 0.4, moe(3, 1, 18), base=77.0),
    latent_layer(1, 6, 2, 12, 15, 5, 0.5, moe(4, 4, 10), base=20.0, scaling=(2.0, 8, 2.0, 1.0)),
    latent_layer(5, 4, 4, 3, 7, 11, 0.6, dense(30))], logit_scale=2.0, eps=1e-6)

#: sizes the tensor-core kernels take (cached rows of 128 and of 64); everything runs three times
CFG_C = model(128, 128, [
    latent_layer(4, 32, 16, 32, 48, 112, 0.15, moe(8, 3, 32, shared=64), base=50000.0, scaling=(4.0, 32, 16.0, 1.0)),
    latent_layer(4, 32, 32, 128, 64, 32, 0.12, dense(160), base=10000.0)], loop=(0, 2, 3), logit_scale=0.25)

#: one layer that runs twice between two that do not; no feed-forward but one; cached rows of 80 and 144 values
CFG_D = model(60, 48, [
    latent_layer(2, 16, 16, 16, 32, 64, 0.2, None, base=500.0, scaling=(16.0, 64, 32.0, 2.0)),
    latent_layer(4, 24, 16, 40, 8, 128, 0.15, moe(5, 2, 16, shared=8)),
    latent_layer(1, 64, 64, 8, 16, 16, 0.1, None, base=100.0)], loop=(1, 2, 2), logit_scale=1.0)

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
        return moe(experts, r.randint(1, min(experts, 6)), pick([8, 24, 40, 64]), shared=pick([None, 16, 72]))

    def layer():
        dim, rd = pick([8, 16, 32, 40, 64]), pick([2, 4, 8, 16, 32, 64])
        sc = (pick([2.0, 4.0, 16.0]), pick([16, 64, 256]), pick([8.0, 32.0]), pick([0.5, 1.0, 2.0])) if r.random() < 0.6 else None
        return latent_layer(pick([1, 2, 3, 4, 8, 16]), dim, rd, pick([8, 16, 24, 64, 128]), pick([8, 20, 64, 96]),
                            pick([8, 24, 48, 64, 96, 112, 192]), (dim + rd) ** -0.5 * pick([1.0, 1.5]), ff(),
                            base=pick([50.0, 1000.0, 10000.0, 500000.0]), scaling=sc)
    layers = [layer() for _ in range(r.randint(1, 4))]
    loop = None
    if r.random() < 0.6:
        a = r.randrange(len(layers))
        loop = (a, r.randint(a + 1, len(layers)), pick([1, 2, 3]))
    return model(pick([64, 100, 257]), pick([48, 64, 100, 128, 192]), layers, loop, pick([0.25, 1.0, 3.0]), pick([1e-5, 1e-6]))


def spec_of(cfg_dict):
    cfg = config_from_dict(cfg_dict)
    return get_architecture(cfg.architecture).build_spec(cfg)


def make_tensors(cfg_dict, seed, spread=8.0):
    """Random weights, then made so that faults show: matrices are scaled up (random weights of deviation 0.02 give
    nearly uniform attention, gates stuck at one half and a router without preferences); every norm's curve gets a slope
    of its own between one and four, so that the residual rows reach into its bend, its weights and biases are spread, and
    so are the projections' biases."""
    t = random_tensors(spec_of(cfg_dict), seed)
    g = torch.Generator().manual_seed(seed + 1000)
    out = {}
    for name in sorted(t):
        v = t[name].clone()
        if name.endswith(".alpha"):
            v = 1.0 + 3.0 * torch.rand((), generator=g)
        elif name == "embed":
            v = v * 3.0 * spread
        elif name.endswith(".router") or name.endswith(".shared.sg"):
            v = v * (2.0 / (0.02 * v.shape[-1] ** 0.5))           # sums of deviation 2 or less whatever the width
        elif name.endswith(".norm1.b") or name.endswith(".norm2.b") or name.endswith("final.norm.b"):
            v = v * 10.0
        elif name.endswith(".b"):
            v = v * 20.0
        elif v.dim() >= 2:
            v = v * (spread / 8.0 * 1.15 / (0.02 * v.shape[-1] ** 0.5))      # rows of deviation one come out a little larger
        elif v.dim() == 1:
            v = 1.0 + 0.3 * torch.randn(v.shape, generator=g)
        out[name] = v.to(torch.bfloat16).to(torch.float32)        # values both dtypes of the engine can hold
    return out
