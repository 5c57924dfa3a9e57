"""``Vonedra`` as a ModelSpec: a scaled token embedding; layers of the ``result_norm`` block (every sublayer reads the
residual plus a causal convolution of it and has its result RMS-normed before it is added; at a layer's end the residual
becomes a weighted sum over the embedding output and all layers' results); the mixer is ``distance_attention``
(grouped-query attention with unit-size queries and keys, a learned bias by distance, a window that keeps the first
tokens, a sink, values mixed with the first such layer's), ``latent_attention`` (queries through a latent of their own,
one cached latent and rotated key part per token, a window) or ``gated_delta_rule`` in its plain form (one decay per
head, a SiLU gate); the feed-forward is ``swiglu``; the output head has a matrix of its own.

Tensor names: ``embed``, ``head``, ``final.norm``; layer ``i``: ``l<i>.norm1|norm2``, ``l<i>.canon1|canon2``,
``l<i>.dwa``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down``.
"""

from __future__ import annotations

from gllm_b200.config.registry import register_architecture
from gllm_b200.config.vonedra_config import VonedraConfig
from gllm_b200.models.spec import LayerSpec, ModelSpec, PartSpec, PlanEntry

# the design's fixed constant: what is added under the root when queries and keys of the delta rule are made unit
# vectors
UNIT_NORM_EPS = 1e-6


def _distance_attention(width: int, eps: float, m: dict, p: str, value_mix: str | None) -> PartSpec:
    mask = m.get("mask") or {}
    names = {n: f"{p}.{n}" for n in ("q", "k", "v", "o", "rel", "sink")}
    names.update({f"{n}_bias": f"{p}.{n}.b" for n in ("q", "k", "v", "o")})
    if value_mix is not None:
        names["mix"] = f"{p}.vmix"
    return PartSpec(
        "distance_attention",
        dict(hidden_size=width, heads=m["heads"], kv_heads=m["kv_heads"], dk=m["dim"], dv=m["vdim"],
             scale=float(m["scale"]), eps=eps, distance_max=m["bias_max"], window=mask.get("size"),
             keep_first=int(mask.get("keep_first", 0)), value_mix=value_mix, bias_rows=m.get("bias_rows")),
        names,
    )


def _latent_attention(width: int, eps: float, m: dict, p: str) -> PartSpec:
    rot, mask = m["rot"], m.get("mask") or {}
    return PartSpec(
        "latent_attention",
        dict(hidden_size=width, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
             kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=float(m["scale"]), eps=eps, window=mask.get("size"),
             position=PartSpec("rotary", dict(head_dim=int(m["rot_dim"]), rotary_dim=int(rot["dims"]),
                                              theta=float(rot["base"]), interleaved=True))),
        {**{n: f"{p}.{n}" for n in ("dq", "uq", "dkv", "uk", "uv", "o")},
         "dq_norm": f"{p}.dq.norm", "dkv_norm": f"{p}.dkv.norm"},
    )


def _delta(width: int, eps: float, m: dict, p: str) -> PartSpec:
    names = {n: f"{p}.{n}" for n in ("q", "k", "v", "b", "a", "A_log", "dt_bias", "norm", "g", "o")}
    names.update({f"{n}_conv": f"{p}.{n}.conv" for n in ("q", "k", "v")})
    return PartSpec(
        "gated_delta_rule",
        dict(hidden_size=width, heads=m["heads"], kv_heads=m["kv_heads"], dk=m["dim"], dv=m["vdim"], taps=m["conv"],
             eps=eps, unit_eps=UNIT_NORM_EPS, q_scale=float(m["dim"]) ** -0.5, head_decay=True),
        names,
    )


def build_vonedra_spec(cfg: VonedraConfig) -> ModelSpec:
    width, eps = cfg.hidden_size, cfg.norm_eps
    mixing = cfg.value_mixing_layers()

    def norm(weight: str) -> PartSpec:
        return PartSpec("rmsnorm", dict(size=width, eps=eps), {"weight": weight})

    def conv(weight: str) -> PartSpec:
        return PartSpec("causal_conv", dict(width=width, taps=cfg.conv_taps), {"weight": weight})

    layers, ignorable = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer.mixer
        if layer.type == "attention":
            value_mix = None if i not in mixing else ("first" if i == mixing[0] else "mixed")
            mixer = _distance_attention(width, eps, m, f"{p}.mix", value_mix)
            if value_mix is None:
                ignorable.append(f"{p}.mix.vmix")
        elif layer.type == "latent_attention":
            mixer = _latent_attention(width, eps, m, f"{p}.mix")
        else:
            mixer = _delta(width, eps, m, f"{p}.mix")
        parts = {"mixer_conv": conv(f"{p}.canon1"), "mixer": mixer, "mixer_norm": norm(f"{p}.norm1")}
        if layer.mlp is not None:
            parts["feed_forward_conv"] = conv(f"{p}.canon2")
            parts["feed_forward"] = PartSpec("swiglu", dict(hidden_size=width, intermediate_size=layer.mlp["ff"]),
                                             {n: f"{p}.mlp.{n}" for n in ("gate", "up", "down")})
            parts["feed_forward_norm"] = norm(f"{p}.norm2")
        else:                                   # a checkpoint may hold them all the same
            ignorable += [f"{p}.norm2", f"{p}.canon2"]
        # the embedding output, the layers before this one, and this one
        parts["depth_average"] = PartSpec("depth_average", dict(streams=i + 2), {"weight": f"{p}.dwa"})
        layers.append(LayerSpec("result_norm", parts))
    return ModelSpec(
        hidden_size=width,
        vocab_size=cfg.vocab_size,
        layers=tuple(layers),
        plan=tuple(PlanEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        embedding_name="embed",
        head_name="head",
        eos_token_ids=cfg.eos_token_ids,
        embedding_scale=cfg.embedding_scale,
        depth_streams=True,
        ignorable_names=tuple(ignorable),
    )


register_architecture("Vonedra", VonedraConfig, build_vonedra_spec)
