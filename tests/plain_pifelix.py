"""A plain, slow restatement of the Pifelix design in float64, one function per mechanism.

It shares nothing with the package: it reads a configuration as a plain dict (the keys of config.json)
and weights as a dict of tensors by checkpoint name, and runs one request's tokens at once on the CPU.

Notation.  ``x``: the residual ``[T, width]``, which the sublayers read as it is; ``p``: positions ``0 .. T-1``.
"""

from __future__ import annotations

import math

import torch

F = torch.float64
GATE_SLOPE = 1.702


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def rms(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


# ---------------------------------------------------------------- convolution over time
def causal_conv(u, weight):
    """``y_t = sum_j weight[:, j] u_{t - taps + 1 + j}``, one filter per channel; zeros before the first token."""
    taps = weight.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += weight[:, j] * u[s]
    return y


def convolved_projection(x, w, name):
    return causal_conv(x @ w[name].T + w[name + ".b"], w[name + ".conv"])


# ---------------------------------------------------------------- rotation
def yarn_frequencies(rot: dict) -> list[float]:
    """``base^(-2i/dims)``; with ``scaling`` pairs before ``lo`` keep it, pairs from ``hi`` on have it divided by
    ``factor``, a linear ramp in between; ``lo`` and ``hi`` are where ``fast`` and ``slow`` turns fit ``original``."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return f

    def pair_with(turns):
        return dims * math.log(float(s["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_with(float(s["fast"]))), 0)
    hi = min(math.ceil(pair_with(float(s["slow"]))), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / float(s["factor"]) * r + v * (1.0 - r))
    return out


def yarn_magnitude(rot: dict) -> float:
    s = rot.get("scaling")
    return 0.1 * math.log(float(s["factor"])) + 1.0 if s else 1.0


def rotate_pairs(x, p, rot):
    """``x [T, heads, dim]``: columns (2i, 2i+1) of the first ``dims`` turn by ``p f_i`` and grow by the magnitude."""
    dims = int(rot["dims"]) if rot else 0
    if dims == 0:
        return x
    a = p.to(F)[:, None] * torch.tensor(yarn_frequencies(rot), dtype=F)[None, :]
    mag = yarn_magnitude(rot)
    c, s = (a.cos() * mag)[:, None, :], (a.sin() * mag)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ---------------------------------------------------------------- attention inside chunks
def queries(x, p, m, w, pre, eps):
    q = convolved_projection(x, w, pre + ".q").view(x.shape[0], m["heads"], m["dim"])
    return rotate_pairs(rms(q, w[pre + ".q.norm"], eps), p, m.get("rot"))


def keys_values(x, p, m, w, pre, eps):
    """Normed and rotated keys ``[T, G, dim]``, convolved values ``[T, G, vdim]``."""
    T = x.shape[0]
    k = convolved_projection(x, w, pre + ".k").view(T, m["kv_heads"], m["dim"])
    v = convolved_projection(x, w, pre + ".v").view(T, m["kv_heads"], m["vdim"])
    return rotate_pairs(rms(k, w[pre + ".k.norm"], eps), p, m.get("rot")), v


def attend(q, k, v, q_pos, k_pos, scale, chunk):
    """``q [Tq, H, dim]``, ``k [Tk, G, dim]``, ``v [Tk, G, vdim]``: softmax over the keys up to the query's position
    in the query's own chunk of ``chunk`` positions (None: no chunks).  Returns ``[Tq, H * vdim]``."""
    H, G = q.shape[1], k.shape[1]
    visible = k_pos[None, :] <= q_pos[:, None]
    if chunk:
        visible &= (k_pos[None, :] // chunk) == (q_pos[:, None] // chunk)
    heads = []
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * float(scale)
        heads.append(torch.softmax(s.masked_fill(~visible, -math.inf), -1) @ v[:, g])
    return torch.cat(heads, -1)


# ---------------------------------------------------------------- routed experts
def route(x, w, pre, top):
    """(chosen experts ``[T, top]``, their scores): the largest sigmoids of the router's logits."""
    s = sigmoid(x @ w[pre + ".router"].T)
    scores, ids = torch.sort(s, dim=-1, descending=True, stable=True)
    return ids[:, :top], scores[:, :top]


def expert(h, w, pre, limit):
    g = torch.clamp(h @ w[pre + ".gate"].T, max=limit)
    u = torch.clamp(h @ w[pre + ".up"].T, min=-limit, max=limit)
    return (g * sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ w[pre + ".down"].T


def routed_experts(x, w, pre, mlp):
    """Every chosen expert gets the token's row multiplied by its score; their results are added."""
    ids, scores = route(x, w, pre, int(mlp["router"]["top"]))
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e, s in zip(ids[t].tolist(), scores[t]):
            out[t] += expert((s * x[t])[None], w, f"{pre}.e{e}", float(mlp["expert"]["limit"]))[0]
    return out


# ---------------------------------------------------------------- the model
def forward(cfg: dict, weights: dict, tokens, layers_out: list | None = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one request's tokens from position 0; ``layers_out`` collects the residual after
    every layer."""
    w = {k: v.to(F) for k, v in weights.items()}
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    T = len(tokens)
    p = torch.arange(T)
    x = w["embed"][torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        m, pre = layer["mixer"], f"l{i}.mix"
        source = m.get("kv_from")
        if source is None:
            kept[i] = keys_values(x, p, m, w, pre, eps)
            source = i
        k, v = kept[source]
        chunk = int(m["mask"]["size"]) if m.get("mask") else None
        o = attend(queries(x, p, m, w, pre, eps), k, v, p, p, m["scale"], chunk) @ w[pre + ".o"].T
        x = x + mult * rms(o, w[f"l{i}.norm1"], eps)
        if layer.get("mlp"):
            x = x + mult * rms(routed_experts(x, w, f"l{i}.mlp", layer["mlp"]), w[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, w["final.norm"], eps) @ w["head"].T
