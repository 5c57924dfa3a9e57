"""Small Vonedra configurations for the tests, as raw config.json dicts, and a writer that draws their weights here (not
through the engine's random-weights mode), tensor by tensor under the names the design gives them.

The configurations differ in every size and option: grouped / multi-query / one head per key head and groups that are no
power of two, key and value widths that differ both ways and are no multiple of 8, windows of one token to more than the
longest request, with and without kept first tokens (fewer and more than a page, more than the window) and none at all,
bias tables with even and odd numbers of rows, layers that mix values and ones that do not, latents and rotated parts
that fill a kernel's tile and ones that do not, partly rotated parts, convolutions of 1 to 6 taps on the sublayers'
inputs and of 1 to 4 in the delta rule, layers without a feed-forward, every order of mixers."""

from __future__ import annotations

import copy
import json
import math
import os

import torch
from safetensors.torch import save_file

BIAS_ROWS = 12            # where the configuration does not name them (the tensor's shape gives them)


def _att(heads, kv_heads, dim, vdim, scale, bias_max, size=None, keep=None, v_mix=True, rows=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
         "v_mix": v_mix}
    if size is not None:
        m["mask"] = {"size": size} | ({} if keep is None else {"keep_first": keep})
    if rows is not None:
        m["bias_rows"] = rows
    return {"type": "attention", "mixer": m}


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, size=None, base=10000.0, dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim if dims is None else dims}}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def _model(layers, width, vocab, taps, scale=2.0, eps=1e-5):
    """``layers``: pairs (mixer entry, feed-forward width or None)."""
    return {"architecture": "Vonedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "canon": {"taps": taps},
            "layers": [{**copy.deepcopy(m), "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for m, ff in layers]}


# all three mixers; a layer that does not mix values between two that do; a layer without a feed-forward
VONEDRA_A = _model([
    (_att(4, 2, 16, 24, 0.4, 50, size=20, keep=5, rows=12), 96),
    (_latent(4, 16, 8, 24, 40, 32, 0.3, size=33), 64),
    (_att(3, 3, 32, 16, 0.25, 64, size=9, keep=0, v_mix=False, rows=7), None),
    (_delta(4, 2, 16, 24, 4), 80),
    (_att(6, 1, 8, 48, 0.5, 40, size=48, keep=3, rows=16), 64),
], width=64, vocab=200, taps=3, scale=5.0)
# sizes that are no multiple of 8; no window in two layers; a window of one token; one tap
VONEDRA_B = _model([
    (_delta(3, 1, 10, 6, 1), 36),
    (_latent(3, 10, 6, 14, 22, 18, 0.35, base=300.0, dims=4), None),
    (_att(3, 1, 20, 12, 0.3, 30.5), 44),
    (_att(2, 2, 12, 6, 0.4, 90, size=1, keep=17), 20),
], width=44, vocab=131, taps=1, scale=1.0, eps=3e-6)
# head widths the tensor-core kernels fill; more kept tokens than the window; long convolutions
VONEDRA_C = _model([
    (_latent(8, 32, 32, 32, 64, 64, 0.2, size=70, base=50000.0), 192),
    (_att(8, 2, 64, 64, 0.15, 128, size=37, keep=50), 128),
    (_att(8, 4, 64, 32, 0.15, 100, size=100, keep=16), None),
    (_delta(4, 4, 32, 32, 2), 128),
], width=128, vocab=160, taps=6, scale=3.0, eps=1e-6)
# every layer without a feed-forward but one; four taps
VONEDRA_D = _model([
    (_att(2, 1, 8, 8, 0.6, 20, size=12, keep=2), None),
    (_delta(2, 2, 8, 16, 3), None),
    (_latent(2, 8, 4, 8, 12, 16, 0.4, size=5), 40),
], width=32, vocab=150, taps=4)
VONEDRA = {"A": VONEDRA_A, "B": VONEDRA_B, "C": VONEDRA_C, "D": VONEDRA_D}


def one_layer(mixer, ff=None, width=64, vocab=120, taps=3, **kw) -> dict:
    return _model([(mixer, ff)], width, vocab, taps, **kw)


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    w, taps = cfg["width"], cfg["canon"]["taps"]
    out = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "final.norm": (w,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, x = f"l{i}", layer["mixer"], f"l{i}.mix"
        out.update({f"{p}.norm1": (w,), f"{p}.canon1": (w, taps), f"{p}.dwa": (i + 2,)})
        h, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            g = m["kv_heads"]
            for n, rows in (("q", h * d), ("k", g * d), ("v", g * dv)):
                out.update({f"{x}.{n}": (rows, w), f"{x}.{n}.b": (rows,)})
            out.update({f"{x}.o": (w, h * dv), f"{x}.o.b": (w,), f"{x}.sink": (h,),
                        f"{x}.rel": (m.get("bias_rows", BIAS_ROWS), h)})
            if m["v_mix"]:
                out[f"{x}.vmix"] = ()
        elif layer["type"] == "latent_attention":
            r, qr, c = m["rot_dim"], m["q_rank"], m["kv_rank"]
            out.update({f"{x}.dq": (qr, w), f"{x}.dq.norm": (qr,), f"{x}.uq": (h * (d + r), qr), f"{x}.dkv": (c + r, w),
                        f"{x}.dkv.norm": (c,), f"{x}.uk": (h * d, c), f"{x}.uv": (h * dv, c), f"{x}.o": (w, h * dv)})
        else:
            g, t = m["kv_heads"], m["conv"]
            for n, rows in (("q", g * d), ("k", g * d), ("v", h * dv)):
                out.update({f"{x}.{n}": (rows, w), f"{x}.{n}.conv": (rows, t)})
            out.update({f"{x}.b": (h, w), f"{x}.a": (h, w), f"{x}.A_log": (h,), f"{x}.dt_bias": (h,), f"{x}.norm": (dv,),
                        f"{x}.g": (h * dv, w), f"{x}.o": (w, h * dv)})
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({f"{p}.norm2": (w,), f"{p}.canon2": (w, taps), f"{p}.mlp.gate": (ff, w), f"{p}.mlp.up": (ff, w),
                        f"{p}.mlp.down": (w, ff)})
    return out


def draw_weights(cfg: dict, seed: int, sharp: float = 1.0) -> dict[str, torch.Tensor]:
    """float32 tensors whose values are bfloat16 numbers.  ``sharp`` multiplies the latent queries, so that the softmax
    has a few large weights and a key that is lost or one too many shows (elsewhere queries and keys have unit size)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        draw = torch.randn(shape, generator=g)
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + draw * 0.15
        elif name == "embed":
            t = draw
        elif last in ("canon1", "canon2"):
            t = draw * 0.3
        elif last == "dwa":
            t = 0.3 * draw + torch.eye(shape[0])[-1]
        elif last == "conv":
            t = draw * 0.6
        elif last == "vmix":
            t = torch.tensor(0.35 + 0.1 * float(torch.rand((), generator=g)))
        elif last in ("rel", "sink"):
            t = draw
        elif len(shape) == 1:                          # biases, A_log, dt_bias
            t = draw * 0.5
        else:
            t = draw / math.sqrt(shape[1])
            if last == "uq":
                t = t * sharp
            if last in ("a", "b") and len(shape) == 2:
                t = t * 0.7
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def write_model(cfg: dict, weights: dict, folder: str) -> str:
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f, indent=1)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights.items()},
              os.path.join(folder, "model.safetensors"))
    return folder
