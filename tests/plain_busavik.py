"""A plain, slow implementation of the Busavik decoder, for tests only: one function per
mechanism, whole sequences, no cache, no batching, any float type.  It shares no code with
the package: it reads config.json's dictionary and the stored tensors by name.

Notation: x [T, E] is a sequence's residual stream, positions 0..T-1; weights are stored [out, in].

  norm              n(x) = w * tanh(a x) + b, value by value, a one number
  layer             x += mixer(n1(x));  x += ff(n2(x)), the second only where the layer has a feed-forward
  schedule          layers 0 .. start-1, then the span start .. stop-1 `times` times over, then the rest
  latent attention  q = U (rms(D_q h) * w_q), per head [q_c, q_r]; [c', k_r] = D_k h, c = rms(c') * w_k;
                    score_ij = (q_c,i . K_h c_j + rot_i(q_r,i) . rot_j(k_r,j)) * scale for j <= i; the joined heads' mixes of
                    V_h c_j are multiplied by sigmoid(G h) before the output matrix
  rotation          pairs (i, i + n/2); slow frequencies stretched by a ramp, cosines and sines magnified
  dense ff          W_d (gelu_tanh(W_g h + b_g) * (W_u h + b_u)) + b_d
  experts           the `top` largest of z = R h, weights softmax over those z alone; sum of weight * W_d (silu(W_g h) * W_u h);
                    a shared expert of the same form times sigmoid(s . h) is added
"""
from __future__ import annotations

import math

import torch


def tanh_norm(x, w, b, alpha):
    return w * torch.tanh(alpha * x) + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def turns(rot):
    """(the dims/2 frequencies, the magnitude of cosines and sines) of a rotary description, as Python floats."""
    n, base = int(rot["dims"]), float(rot["base"])
    freqs = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freqs, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def at(t):
        return n * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(at(float(sc["fast"]))), 0)
    hi = min(math.ceil(at(float(sc["slow"]))), n - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, rot):
    """x [T, H, D]: the first rot["dims"] values of every head turned by the row's position, pairs (i, i + dims/2)."""
    T, n = x.shape[0], int(rot["dims"])
    freqs, magnitude = turns(rot)
    a = torch.arange(T, dtype=x.dtype)[:, None] * torch.tensor(freqs, dtype=x.dtype)[None, :]
    cos, sin = (torch.cos(a) * magnitude)[:, None, :], (torch.sin(a) * magnitude)[:, None, :]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., n:]], dim=-1)


def causal_attention(q, k, v, scale):
    """q, k [T, H, D], v [T, H, Dv] -> [T, H, Dv]; one head at a time."""
    T, H, _ = q.shape
    later = torch.triu(torch.ones(T, T, dtype=torch.bool), diagonal=1)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = ((q[:, h] @ k[:, h].T) * scale).masked_fill(later, float("-inf"))
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, h]
    return out


def latent_attention(h, m, w, eps):
    T = h.shape[0]
    H, D, R, Dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
    q = (cq @ w["uq"].T).view(T, H, D + R)
    down = h @ w["dkv"].T
    c = rms(down[:, :C], eps) * w["dkv.norm"]
    k_r = rotate(down[:, C:].view(T, 1, R), m["rot"]).expand(T, H, R)
    k_c = (c @ w["uk"].T).view(T, H, D)
    v = (c @ w["uv"].T).view(T, H, Dv)
    o = causal_attention(torch.cat([q[..., :D], rotate(q[..., D:], m["rot"])], dim=-1), torch.cat([k_c, k_r], dim=-1), v,
                         float(m["scale"]))
    return (o.reshape(T, H * Dv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def dense_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def gated_expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose(z, top):
    """(indices of the ``top`` largest of z, the softmax over those alone)."""
    best, ids = torch.sort(z, descending=True)
    return ids[:top], torch.softmax(best[:top], dim=-1)


def routed_ff(h, mlp, w):
    out = torch.zeros_like(h)
    z = h @ w["router"].T
    for t in range(h.shape[0]):
        ids, weights = choose(z[t], int(mlp["router"]["top"]))
        for e, p in zip(ids.tolist(), weights):
            out[t] += p * gated_expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    if mlp.get("shared"):
        y = gated_expert(h, w["shared.gate"], w["shared.up"], w["shared.down"])
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * y
    return out


def runs(cfg):
    """The layers' indices in the order they run."""
    order = list(range(len(cfg["layers"])))
    loop = cfg.get("loop")
    if not loop:
        return order
    a, b, n = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return order[:a] + order[a:b] * n + order[b:]


def _sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg: dict, tensors: dict, tokens, dt=torch.float64, layer_outputs=None):
    """Logits [T, vocab] of one sequence; ``layer_outputs`` (a list) receives x after every layer run."""
    t = {k: (v.to(dt) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])

    def norm(x, name):
        return tanh_norm(x, t[name], t[name + ".b"], t[name + ".alpha"])
    x = t["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    for i in runs(cfg):
        layer = cfg["layers"][i]
        x = x + latent_attention(norm(x, f"l{i}.norm1"), layer["mixer"], _sub(t, f"l{i}.mix."), eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm(x, f"l{i}.norm2")
            w = _sub(t, f"l{i}.mlp.")
            x = x + (dense_ff(h, w) if mlp["kind"] == "dense" else routed_ff(h, mlp, w))
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return norm(x, "final.norm") @ t["head"].T * float(cfg["logit_scale"])
