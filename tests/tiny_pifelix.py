"""Small Pifelix configurations for the tests, as raw config.json dicts, and a writer that draws their weights here
(not through the engine's random-weights mode), tensor by tensor under the names the design gives them.

The configurations differ in every size and option: layers that read the keys and values of an earlier layer (one
reader, two readers, with chunks and filters of their own), layers without a feed-forward, grouped / multi-query / one
query head per key head, key and value widths that differ both ways, rotations over the whole head, a part of it and
none, with and without frequency scaling, convolutions of 1 to 6 taps, chunks that are smaller than a page, no multiple
of one, larger than one, and none, one expert per token, several and all of them, sizes that are no multiple of 8 and
sizes the tensor-core kernels take."""

from __future__ import annotations

import json
import math
import os

import torch
from safetensors.torch import save_file


def _att(heads, kv_heads, dim, vdim, scale, chunk, conv, dims, base=10000.0, scaling=None, kv_from=None):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "rot": rot}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _moe(ff, experts, top, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _model(vocab, width, layers, eps=1e-5, scale=4.0, mult=0.6):
    return {"architecture": "Pifelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "layers": layers}


_YARN = (4.0, 64, 16.0, 1.0)

# values wider than keys, a partial scaled rotation; two readers of layer 0, one with larger chunks, one with smaller
PIFELIX_A = _model(200, 64, [
    _layer(_att(4, 2, 16, 24, 0.2, 20, 3, 8, scaling=_YARN), _moe(32, 8, 2, 0.7)),
    _layer(_att(4, 2, 16, 24, 0.25, 33, 4, 8, scaling=_YARN, kv_from=0), _moe(24, 5, 3, 1.5)),
    _layer(_att(2, 1, 24, 16, 0.3, 16, 2, 24, base=300.0), None),
    _layer(_att(4, 2, 16, 24, 0.15, 12, 2, 8, scaling=_YARN, kv_from=0), _moe(40, 4, 4, 0.4)),
])

# sizes that are no multiple of 8, one key head for all query heads, one expert per token, a filter of one tap (no
# state) and of six, a head without a rotation, a layer without chunks
PIFELIX_B = _model(131, 44, [
    _layer(_att(3, 1, 10, 7, 0.35, 50, 1, 10, base=500.0), _moe(20, 6, 1, 2.0)),
    _layer(_att(1, 1, 12, 21, 0.3, 7, 6, 0), _moe(28, 3, 1, 0.5)),
    _layer(_att(2, 2, 9, 5, 0.4, None, 5, 4, scaling=(8.0, 32, 8.0, 0.5)), None),
], eps=1e-6, scale=9.0, mult=1.3)

# sizes the tensor-core products and attention kernels take
PIFELIX_C = _model(256, 128, [
    _layer(_att(4, 2, 64, 64, 0.125, 40, 4, 32, scaling=_YARN), _moe(64, 4, 2, 1.0)),
    _layer(_att(6, 3, 40, 56, 0.2, 64, 2, 40, scaling=(16.0, 48, 4.0, 0.25)), _moe(128, 6, 1, 0.8)),
    _layer(_att(4, 2, 64, 64, 0.1, 96, 3, 32, scaling=_YARN, kv_from=0), _moe(64, 3, 3, 3.0)),
    _layer(_att(2, 1, 128, 96, 0.09, 150, 4, 64), None),
], scale=2.0, mult=0.8)

PIFELIX = {"A": PIFELIX_A, "B": PIFELIX_B, "C": PIFELIX_C}


def one_layer(mixer, mlp=None, width=64, vocab=150, **more):
    """A model of one layer: the mechanism alone between the embedding and the head."""
    return _model(vocab, width, [_layer(mixer, mlp)], **more)


def tensor_shapes(cfg: dict) -> dict[str, tuple]:
    """Names and shapes of a configuration's tensors, as the design lays them out."""
    w, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        rows = {"q": m["heads"] * m["dim"]}
        if m.get("kv_from") is None:
            rows |= {"k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
        for n, r in rows.items():
            out[f"{p}.{n}"], out[f"{p}.{n}.b"], out[f"{p}.{n}.conv"] = (r, w), (r,), (r, m["conv"])
            if n != "v":
                out[f"{p}.{n}.norm"] = (m["dim"],)
        out[p + ".o"], out[f"l{i}.norm1"] = (w, m["heads"] * m["vdim"]), (w,)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        q, ff = f"l{i}.mlp", mlp["expert"]["ff"]
        out[q + ".router"], out[f"l{i}.norm2"] = (mlp["router"]["experts"], w), (w,)
        for e in range(mlp["router"]["experts"]):
            out[f"{q}.e{e}.gate"], out[f"{q}.e{e}.up"], out[f"{q}.e{e}.down"] = (ff, w), (ff, w), (w, ff)
    out["final.norm"], out["head"] = (w,), (cfg["vocab"], w)
    return out


def draw_weights(cfg: dict, seed: int = 0, sharp: float = 1.0) -> dict[str, torch.Tensor]:
    """Weights as bfloat16-representable fp32 tensors.  ``sharp`` multiplies the query norms (peaked attention)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + torch.randn(shape, generator=g) * 0.2
            if name.endswith(".q.norm"):
                t = t * sharp
        elif last == "b":
            t = torch.randn(shape, generator=g) * 0.3
        elif last == "conv":
            t = torch.randn(shape, generator=g) * 0.5
            t[:, -1] += 0.5
        elif name == "embed":
            t = torch.randn(shape, generator=g) / cfg["embedding"]["scale"]
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


ROUTE_COLUMNS = 4


def decisive_routing(cfg: dict, weights: dict, seed: int = 3, gap: float = 0.4) -> dict:
    """Make every router's choice robust against rounding without making it the same for all tokens.  The last
    ``ROUTE_COLUMNS`` columns of the residual carry a code of +-2 per token (exact in bfloat16) that no layer changes
    (their norm weights are zero there); the routers read only these columns, and their rows are drawn again until, for
    every code, the last chosen expert's logit lies at least ``gap`` above the next one's."""
    g = torch.Generator().manual_seed(seed)
    w, cols = cfg["width"], list(range(cfg["width"] - ROUTE_COLUMNS, cfg["width"]))
    out = {k: v.clone() for k, v in weights.items()}
    codes = (torch.randint(0, 2, (cfg["vocab"], ROUTE_COLUMNS), generator=g) * 2 - 1).float() * 2.0
    out["embed"][:, cols] = codes
    for name in out:
        if name.endswith((".norm1", ".norm2")):
            out[name][cols] = 0.0
    seen = torch.tensor([[1.0 if (c >> j) & 1 else -1.0 for j in range(ROUTE_COLUMNS)]
                         for c in range(2 ** ROUTE_COLUMNS)]) * 2.0 * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        mlp = layer.get("mlp")
        if not mlp:
            continue
        E, top = mlp["router"]["experts"], mlp["router"]["top"]
        for _ in range(20000):
            rows = torch.randn(E, ROUTE_COLUMNS, generator=g) / (2.0 * cfg["embedding"]["scale"])
            rows = rows.to(torch.bfloat16).to(torch.float32)
            order = (seen @ rows.T).sort(-1, descending=True).values
            if top == E or bool((order[:, top - 1] - order[:, top] >= gap * (1.0 if E < 8 else 0.25)).all()):
                break
        else:
            raise RuntimeError("no decisive router found")
        t = torch.zeros(E, w)
        t[:, cols] = rows
        out[f"l{i}.mlp.router"] = t
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in out.items()}


def write_model(cfg: dict, weights: dict, folder: str) -> str:
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f, indent=1)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights.items()},
              os.path.join(folder, "model.safetensors"))
    return folder
