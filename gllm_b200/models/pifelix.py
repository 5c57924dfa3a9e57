"""``Pifelix`` as a ModelSpec: a scaled token embedding; layers of the ``result_only_norm`` block (the sublayers read the
residual as it is, their results are RMS-normed and added with a constant factor); the mixer is ``conv_attention`` (biased
projections convolved over time, normed query and key heads, neighbouring rotary pairs with wavelength-dependent
frequency scaling, attention within chunks; a layer may read an earlier layer's keys and values); the feed-forward is
``routed_experts`` (sigmoid scores that are not renormalized and multiply the experts' inputs, clamped gated experts); the
output head has a matrix of its own.

Tensor names: ``embed``, ``head``, ``final.norm``; layer ``i``: ``l<i>.norm1|norm2``, ``l<i>.mix.*``,
``l<i>.mlp.router``, ``l<i>.mlp.e<j>.gate|up|down``.
"""

from __future__ import annotations

from gllm_b200.config.pifelix_config import PifelixConfig
from gllm_b200.config.registry import register_architecture
from gllm_b200.models.spec import LayerSpec, ModelSpec, PartSpec, PlanEntry

# the design's fixed constants: the slope of the gate's sigmoid and what is added to the up product
GATE_SLOPE = 1.702
UP_OFFSET = 1.0


def _rotary(rot: dict | None, dim: int) -> PartSpec | None:
    if rot is None or int(rot["dims"]) == 0:
        return None
    scaling = rot.get("scaling")
    if scaling is not None:
        scaling = {"rope_type": "yarn", "factor": scaling["factor"], "beta_fast": scaling["fast"],
                   "beta_slow": scaling["slow"], "original_max_position_embeddings": scaling["original"]}
    return PartSpec("rotary", dict(head_dim=dim, rotary_dim=int(rot["dims"]), theta=float(rot["base"]),
                                   scaling=scaling, interleaved=True))


def _attention(width: int, eps: float, m: dict, p: str) -> PartSpec:
    own = m.get("kv_from") is None
    names = {"o": f"{p}.o"}
    for n in ("q", "k", "v") if own else ("q",):
        names |= {n: f"{p}.{n}", f"{n}_bias": f"{p}.{n}.b", f"{n}_conv": f"{p}.{n}.conv"}
    names |= {f"{n}_norm": f"{p}.{n}.norm" for n in (("q", "k") if own else ("q",))}
    mask = m.get("mask")
    return PartSpec(
        "conv_attention",
        dict(hidden_size=width, heads=m["heads"], kv_heads=m["kv_heads"], dk=m["dim"], dv=m["vdim"], taps=m["conv"],
             scale=float(m["scale"]), eps=eps, position=_rotary(m.get("rot"), int(m["dim"])),
             chunk=None if mask is None else int(mask["size"]), own_kv=own),
        names,
    )


def _experts(width: int, mlp: dict, p: str) -> PartSpec:
    router, expert = mlp["router"], mlp["expert"]
    return PartSpec(
        "routed_experts",
        dict(hidden_size=width, intermediate_size=expert["ff"], experts=router["experts"], top=router["top"],
             score="sigmoid", renormalize=False, gate_slope=GATE_SLOPE, gate_limit=float(expert["limit"]),
             up_offset=UP_OFFSET, weight_on_input=True),
        {"router": f"{p}.router", "expert": p + ".e{index}.{part}"},
    )


def build_pifelix_spec(cfg: PifelixConfig) -> ModelSpec:
    width, eps = cfg.hidden_size, cfg.norm_eps

    def norm(weight: str, multiplier: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", dict(size=width, eps=eps, multiplier=multiplier), {"weight": weight})

    layers, plan, ignorable = [], [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer.mixer
        parts = {"mixer": _attention(width, eps, m, f"{p}.mix"), "mixer_norm": norm(f"{p}.norm1", cfg.residual_mult)}
        if layer.mlp is not None:
            parts["feed_forward"] = _experts(width, layer.mlp, f"{p}.mlp")
            parts["feed_forward_norm"] = norm(f"{p}.norm2", cfg.residual_mult)
        else:                                   # a checkpoint may hold it all the same
            ignorable.append(f"{p}.norm2")
        layers.append(LayerSpec("result_only_norm", parts))
        # (plan entries and layers run one to one here, so a layer index is a plan index)
        reads = m.get("kv_from")
        plan.append(PlanEntry(i, reads_cache_of=None if reads is None else int(reads)))
    return ModelSpec(
        hidden_size=width,
        vocab_size=cfg.vocab_size,
        layers=tuple(layers),
        plan=tuple(plan),
        final_norm=norm("final.norm"),
        embedding_name="embed",
        head_name="head",
        eos_token_ids=cfg.eos_token_ids,
        embedding_scale=cfg.embedding_scale,
        ignorable_names=tuple(ignorable),
    )


register_architecture("Pifelix", PifelixConfig, build_pifelix_spec)
