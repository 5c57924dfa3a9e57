"""A plain, slow restatement of the Vonedra design in float64, one function per mechanism.

It shares nothing with the package: it reads a configuration as a plain dict (the keys of config.json) and weights as
a dict of tensors by checkpoint name, and runs one request's tokens at once (or portion after portion through
``PlainState``) on the CPU.

Notation.  ``x``: the residual ``[T, width]``; ``h``: what a sublayer reads; ``p``: positions;
``rms(x) = x / sqrt(mean(x^2) + eps)``.
"""

from __future__ import annotations

import math
from fractions import Fraction

import torch

F = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


# ---------------------------------------------------------------- convolutions over time
def causal_conv(x: torch.Tensor, w: torch.Tensor, before: torch.Tensor):
    """``y_t = sum_j w[:, j] x_(t - taps + 1 + j)`` per channel; ``before [taps-1, C]``: the inputs before the first
    row.  Returns y and the inputs to keep."""
    taps, T = w.shape[1], x.shape[0]
    full = torch.cat([before, x], 0)
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + full[j:j + T] * w[:, j]
    return y, full[T:]


def sublayer_input(x, w, state, key):
    """``x + conv(x)``."""
    y, state[key] = causal_conv(x, w, state[key])
    return x + y


# ---------------------------------------------------------------- what attention sees and how far it is
def visible(q_pos, k_pos, size=None, keep_first=0):
    d = q_pos[:, None] - k_pos[None, :]
    ok = d >= 0
    if size is not None:
        ok = ok & ((d < size) | (k_pos[None, :] < keep_first))
    return ok


def distance_bucket(n: int, rows: int, distance_max) -> int:
    """``n`` below half the rows; above: logarithmic steps up to ``distance_max`` (exact arithmetic: the step is the
    largest k with (n / half)^m >= (distance_max / half)^k, m the number of logarithmic rows)."""
    half = rows // 2
    if n < half:
        return n
    m = rows - half
    ratio, span = Fraction(n, half), Fraction(distance_max) / half
    k = 0
    while k < m - 1 and ratio ** m >= span ** (k + 1):
        k += 1
    return min(rows - 1, half + k)


def attend(q, k, v, q_pos, k_pos, scale, size, keep_first=0, bias=None, sink=None):
    """``q [T, H, d]``, ``k [S, G, d]``, ``v [S, G, dv]``; ``bias`` a function (distance, head) -> number; ``sink
    [H]`` adds exp(sink) to every denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    ok = visible(q_pos, k_pos, size, keep_first)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias(q_pos[:, None] - k_pos[None, :], hd)
        s = s.masked_fill(~ok, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink[hd].expand(T, 1)], 1)
        a = torch.softmax(s, -1)
        out[:, hd] = a[:, :k.shape[0]] @ v[:, g]
    return out.reshape(T, -1)


# ---------------------------------------------------------------- mixers
def rotate_pairs(x: torch.Tensor, p: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """``x [T, heads, d]``: neighbours (2i, 2i+1) of the first ``dims`` columns turn by ``p * base^(-2i/dims)``."""
    if dims == 0:
        return x
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=F) / dims)
    a = p.to(F)[:, None] * f[None, :]
    c, s = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def latent_attention(h, p, m, w, pre, eps, state):
    T, H, d, r, dv, c_n = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    cq = rms(h @ w[pre + ".dq"].T, eps) * w[pre + ".dq.norm"]
    q = (cq @ w[pre + ".uq"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], p, float(rot["base"]), int(rot["dims"]))], -1)
    down = h @ w[pre + ".dkv"].T
    c = rms(down[:, :c_n], eps) * w[pre + ".dkv.norm"]
    kr = rotate_pairs(down[:, None, c_n:], p, float(rot["base"]), int(rot["dims"]))[:, 0]
    state["c"], state["kr"] = torch.cat([state["c"], c]), torch.cat([state["kr"], kr])
    S = state["c"].shape[0]
    k = torch.cat([(state["c"] @ w[pre + ".uk"].T).view(S, H, d), state["kr"][:, None].expand(S, H, r)], -1)
    v = (state["c"] @ w[pre + ".uv"].T).view(S, H, dv)
    mask = m.get("mask")
    o = attend(q, k, v, p, torch.arange(S), float(m["scale"]), mask["size"] if mask else None)
    return o @ w[pre + ".o"].T


def attention(h, p, m, w, pre, eps, state, first_values):
    """``first_values``: None in the first layer that mixes values (its own are then returned), else that layer's
    values of the same tokens."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[pre + ".q"].T + w[pre + ".q.b"]).view(T, H, d), eps)
    k = rms((h @ w[pre + ".k"].T + w[pre + ".k.b"]).view(T, G, d), eps)
    v = (h @ w[pre + ".v"].T + w[pre + ".v.b"]).view(T, G, dv)
    if m.get("v_mix"):
        if first_values is None:
            first_values = v
        else:
            lam = w[pre + ".vmix"].reshape(())
            v = (1 - lam) * v + lam * first_values.reshape(v.shape)
    state["k"], state["v"] = torch.cat([state["k"], k]), torch.cat([state["v"], v])
    S, table = state["k"].shape[0], w[pre + ".rel"]
    buckets = torch.tensor([distance_bucket(n, table.shape[0], m["bias_max"]) for n in range(S)])
    mask = m.get("mask") or {}
    o = attend(q, state["k"], state["v"], p, torch.arange(S), float(m["scale"]), mask.get("size"),
               mask.get("keep_first", 0), bias=lambda n, hd: table[buckets[n.clamp(min=0)], hd], sink=w[pre + ".sink"])
    return o @ w[pre + ".o"].T + w[pre + ".o.b"], first_values


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta, S):
    """Per head, token after token: ``S <- g S``, ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q``.
    ``q, k [T, H, dk]``, ``v [T, H, dv]``, ``g, beta [T, H]``, ``S [H, dk, dv]`` (changed in place)."""
    o = torch.zeros_like(v)
    for t in range(v.shape[0]):
        for hd in range(v.shape[1]):
            S[hd] *= g[t, hd]
            u = beta[t, hd] * (v[t, hd] - S[hd].T @ k[t, hd])
            S[hd] += torch.outer(k[t, hd], u)
            o[t, hd] = S[hd].T @ q[t, hd]
    return o


def delta(h, m, w, pre, eps, state):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    x = {}
    for n in ("q", "k", "v"):
        y, state["conv_" + n] = causal_conv(h @ w[f"{pre}.{n}"].T, w[f"{pre}.{n}.conv"], state["conv_" + n])
        x[n] = silu(y)
    q = (unit(x["q"].view(T, G, dk)) * dk ** -0.5).repeat_interleave(H // G, 1)
    k = unit(x["k"].view(T, G, dk)).repeat_interleave(H // G, 1)
    v = x["v"].view(T, H, dv)
    beta = torch.sigmoid(h @ w[pre + ".b"].T)
    g = torch.exp(-torch.exp(w[pre + ".A_log"]) * softplus(h @ w[pre + ".a"].T + w[pre + ".dt_bias"]))
    o = delta_rule(q, k, v, g, beta, state["S"])
    o = rms(o, eps) * w[pre + ".norm"] * silu(h @ w[pre + ".g"].T).view(T, H, dv)
    return o.reshape(T, -1) @ w[pre + ".o"].T


def feed_forward(h, w, pre):
    return (silu(h @ w[pre + ".gate"].T) * (h @ w[pre + ".up"].T)) @ w[pre + ".down"].T


# ---------------------------------------------------------------- the model
class PlainState:
    """What one request carries from token to token, per layer."""

    def __init__(self, cfg):
        taps, width = int(cfg["canon"]["taps"]), int(cfg["width"])
        self.layers, self.length = [], 0
        zeros = lambda *s: torch.zeros(*s, dtype=F)
        for layer in cfg["layers"]:
            m = layer["mixer"]
            s = {"in1": zeros(taps - 1, width), "in2": zeros(taps - 1, width)}
            if layer["type"] == "latent_attention":
                s.update(c=zeros(0, m["kv_rank"]), kr=zeros(0, m["rot_dim"]))
            elif layer["type"] == "attention":
                s.update(k=zeros(0, m["kv_heads"], m["dim"]), v=zeros(0, m["kv_heads"], m["vdim"]))
            else:
                c, qk = m["conv"] - 1, m["kv_heads"] * m["dim"]
                s.update(S=zeros(m["heads"], m["dim"], m["vdim"]), conv_q=zeros(c, qk), conv_k=zeros(c, qk),
                         conv_v=zeros(c, m["heads"] * m["vdim"]))
            self.layers.append(s)


def forward(cfg, weights, tokens, state: PlainState | None = None, layers_out: list | None = None):
    """Logits ``[T, vocab]`` (float64) of ``tokens`` continuing ``state`` (a fresh one if None); ``layers_out``
    collects the residual after every layer."""
    w = {k: v.to(F) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    state = state or PlainState(cfg)
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    p = torch.arange(state.length, state.length + tokens.numel())
    x = w["embed"][tokens] * float(cfg["embedding"]["scale"])
    results, first_values = [x], None
    for i, layer in enumerate(cfg["layers"]):
        pre, m, s = f"l{i}", layer["mixer"], state.layers[i]
        h = sublayer_input(x, w[pre + ".canon1"], s, "in1")
        if layer["type"] == "latent_attention":
            y = latent_attention(h, p, m, w, pre + ".mix", eps, s)
        elif layer["type"] == "attention":
            y, first_values = attention(h, p, m, w, pre + ".mix", eps, s, first_values)
        else:
            y = delta(h, m, w, pre + ".mix", eps, s)
        x = x + rms(y, eps) * w[pre + ".norm1"]
        if layer.get("mlp"):
            h = sublayer_input(x, w[pre + ".canon2"], s, "in2")
            x = x + rms(feed_forward(h, w, pre + ".mlp"), eps) * w[pre + ".norm2"]
        results.append(x)
        x = sum(a * r for a, r in zip(w[pre + ".dwa"], results))
        if layers_out is not None:
            layers_out.append(x.clone())
    state.length += tokens.numel()
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
