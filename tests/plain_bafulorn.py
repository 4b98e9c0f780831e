"""A plain, slow implementation of the Bafulorn decoder, for tests only: one function per
mechanism, whole sequences, no cache, no batching, any float type.  It shares no code with
the package: it reads config.json's dictionary and the stored tensors by name.

Notation: x [T, E] is a sequence's residual stream, positions 0..T-1; weights are stored [out, in].

  N(x; w)           x / sqrt(mean x^2 + eps) * (1 + w)
  start             x = N(embed[token])
  layer             x += m N(mixer(N(x)));  x += m N(ff(N(x)))     (four norms with weights of their own)
  latent attention  per head q = Q h; c = rms(D h) * w cached; k = U_k c, v = U_v c; softmax of q . k scale over the last
                    `size` positions; head h's result times sigmoid(G h)_h
  attention         grouped; q = Q h + b, k = K h + b, values are k before the rotation; a rotated prefix with stretched
                    slow frequencies; a position sees the last `size` positions and the first `keep_first`
  state space       [z | x | B | C | dt] = W h; x, B, C convolved over time (with a bias) and silu; per head, with
                    dt = softplus(dt + bias): S_t = exp(-exp(A) dt) S_(t-1) + dt B_t x_t^T, y_t = S_t^T C_t + D x_t;
                    (y * silu(z)) / rms over each of `norm_groups` equal parts * w
  feed-forward      W_down (relu(W_gate h) * W_up h), or experts with silu in relu's place: s = sigmoid(R h), the largest
                    s + correction are chosen, weighed by s / (sum of the chosen s + 1e-20) * router scale; one more
                    expert that every token uses is added as it is
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def relu(z):
    return torch.clamp(z, min=0.0)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def frequencies(rot, dt=torch.float64):
    """The dims/2 frequencies of a rotary description {"base", "dims", optional "scaling"}."""
    n = int(rot["dims"])
    sc = rot.get("scaling")
    out = []
    for i in range(n // 2):
        f = float(rot["base"]) ** (-2.0 * i / n)
        if sc:
            length = 2.0 * math.pi / f
            if length > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif length >= sc["original"] / sc["high"]:
                s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=dt)


def rotate(x, rot):
    """x [T, H, D]: of every head the first rot["dims"] values turned by the row's position, in pairs (i, i + dims/2)."""
    T, half = x.shape[0], int(rot["dims"]) // 2
    a = torch.arange(T, dtype=x.dtype)[:, None] * frequencies(rot, x.dtype)[None, :]
    cos, sin = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], dim=-1)


def visible(T, mask):
    """[T, T] bool: whether row i sees column j, for a mask {"size", optional "keep_first"} (None: causal only)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    size = (mask or {}).get("size")
    if size:
        see = see & ((i - j < size) | (j < int(mask.get("keep_first") or 0)))
    return see


def softmax_attention(q, k, v, scale, see):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]; query head h reads key head h // (H/G)."""
    H, G = q.shape[1], k.shape[1]
    heads = []
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~see, float("-inf"))
        heads.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.stack(heads, dim=1)


def latent_attention(h, m, w, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    c = rms(h @ w["dkv"].T, eps) * w["dkv.norm"]
    q = (h @ w["q"].T).view(T, H, D)
    k, v = (c @ w["uk"].T).view(T, H, D), (c @ w["uv"].T).view(T, H, -1)
    o = softmax_attention(q, k, v, float(m["scale"]), visible(T, m.get("mask")))
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, -1) @ w["o"].T


def attention(h, m, w):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, D)
    k = (h @ w["k"].T + w["k.b"]).view(T, G, D)
    turned = [rotate(x, m["rot"]) if m.get("rot") else x for x in (q, k)]
    o = softmax_attention(*turned, k, float(m["scale"]), visible(T, m.get("mask")))
    return o.reshape(T, -1) @ w["o"].T + w["o.b"]


def causal_convolution(x, taps, bias):
    """y_t = bias + sum_d taps[:, K-1-d] x_(t-d) per channel, with zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = bias[None, :].expand(T, -1).clone()
    for d in range(min(K, T)):
        y[d:] += taps[:, K - 1 - d] * x[:T - d]
    return y


def state_space(x, B, C, dt, A_log, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (positive): the recurrence and its read-out, y [T, H, P]."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    group = torch.arange(H) // (H // G)
    S = x.new_zeros(H, N, P)
    ys = []
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][group][:, :, None] * x[t][:, None, :]
        ys.append((S * C[t][group][:, :, None]).sum(1) + D[:, None] * x[t])
    return torch.stack(ys)


def gated_group_norm(y, z, w, groups, eps):
    """(y silu(z)), cut into equal parts, each divided by its own root mean square, times w."""
    v = y * silu(z)
    return rms(v.view(v.shape[0], groups, -1), eps).reshape(v.shape) * w


def mamba2(h, m, w, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = h @ w["in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_convolution(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :inner].view(T, H, P), xbc[:, inner:inner + G * N].view(T, G, N), xbc[:, inner + G * N:].view(T, G, N)
    y = state_space(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return gated_group_norm(y.reshape(T, inner), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


def gated_ff(h, gate, up, down, act):
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


def choose(z, correction, top, scale):
    """(chosen outputs, their weights) for one row of router sums."""
    s = torch.sigmoid(z)
    ids = torch.argsort(s + correction, descending=True, stable=True)[:top]
    return ids, s[ids] / (s[ids].sum() + 1e-20) * scale


def routed_ff(h, mlp, w):
    r = mlp["router"]
    rows = []
    for t in range(h.shape[0]):
        ids, weights = choose(w["router"] @ h[t], w["correction"], r["top"], float(r["scale"]))
        y = torch.zeros_like(h[t])
        for e, a in zip(ids.tolist(), weights):
            y = y + a * gated_ff(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], silu)
        if mlp.get("shared"):
            y = y + gated_ff(h[t], w["shared.gate"], w["shared.up"], w["shared.down"], silu)
        rows.append(y)
    return torch.stack(rows)


def forward(cfg, tensors, tokens, dt=torch.float64, layer_outputs=None):
    """Logits [T, vocab] of one sequence; ``layer_outputs`` (a list) receives x after every layer."""
    t = {k: v.to(dt) for k, v in tensors.items()}
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = norm(t["embed"][torch.tensor(list(tokens))], t["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        def of(part):
            pre = f"l{i}.{part}."
            return {k[len(pre):]: v for k, v in t.items() if k.startswith(pre)}
        w = of("mix")
        h = norm(x, t[f"l{i}.norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, layer["mixer"], w, eps)
        elif layer["type"] == "attention":
            y = attention(h, layer["mixer"], w)
        else:
            y = mamba2(h, layer["mixer"], w, eps)
        x = x + m * norm(y, t[f"l{i}.norm1b"], eps)
        if layer.get("mlp"):
            w = of("mlp")
            h = norm(x, t[f"l{i}.norm2"], eps)
            if layer["mlp"]["kind"] == "dense":
                y = gated_ff(h, w["gate"], w["up"], w["down"], relu)
            else:
                y = routed_ff(h, layer["mlp"], w)
            x = x + m * norm(y, t[f"l{i}.norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return norm(x, t["final.norm"], eps) @ t["head"].T
