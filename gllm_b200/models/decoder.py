"""The generic decoder: builds whatever a ModelSpec describes and runs it.

``forward`` is the model half of the step function: embedding lookup, the
layer plan, the final norm at the wanted rows only, and the output head in
fp32.  The reference computes logits at every position and slices afterwards
(gllm/llm/llm.py:335-340); here the final norm and the head see only the rows
whose logits were asked for.
"""

from __future__ import annotations

import torch

from gllm_b200 import ops
from gllm_b200.models.spec import ModelSpec
from gllm_b200.parts import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, build_part
from gllm_b200.parts.base import (DEPTH_AVERAGES, INPUT_CONVS, Block, MixerCache, Norm, StateRequirement, StepContext,
                                  TensorExpectation)


_TABLE_OF_KIND = {"mixer": MIXERS, "feed_forward": FEED_FORWARDS, "norm": NORMS, "input_conv": INPUT_CONVS,
                  "depth_average": DEPTH_AVERAGES}


def _build_layer(layer_spec) -> Block:
    """The registered block of ``layer_spec.block`` with the parts it declares, each built from the
    spec of the same name."""
    try:
        block_cls = BLOCKS[layer_spec.block]
    except KeyError:
        raise KeyError(f"no block of kind {layer_spec.block!r} is registered; known: {sorted(BLOCKS)}") from None
    declared = block_cls.part_kinds
    missing = [n for n in declared if n not in layer_spec.parts and n not in block_cls.optional_parts]
    extra = [n for n in layer_spec.parts if n not in declared]
    if missing or extra:
        raise ValueError(f"block {layer_spec.block!r} declares parts {list(declared)}: the layer lacks {missing} "
                         f"and names {extra} beyond them")
    return block_cls(**{name: build_part(_TABLE_OF_KIND[kind], layer_spec.parts[name])
                        for name, kind in declared.items() if name in layer_spec.parts})


def expected_tensors_of_spec(spec: ModelSpec) -> dict[str, TensorExpectation]:
    """Every checkpoint tensor the model will read, in declaration order."""
    spec.validate()
    exp: dict[str, TensorExpectation] = {
        spec.embedding_name: TensorExpectation((spec.vocab_size, spec.hidden_size), "matrix")
    }
    for layer_spec in spec.layers:
        for part in _build_layer(layer_spec).parts():
            exp.update(part.expected_tensors())
    if spec.rejoin_name is not None:
        exp[spec.rejoin_name] = TensorExpectation((spec.hidden_size, 2 * spec.hidden_size), "matrix")
    exp.update(build_part(NORMS, spec.final_norm).expected_tensors())
    if spec.head_name is not None:
        exp[spec.head_name] = TensorExpectation((spec.vocab_size, spec.hidden_size), "matrix")
    return exp


class DecoderModel:
    """A stack of blocks between an embedding table and an output head."""

    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device: torch.device | str):
        spec.validate()
        self.spec = spec
        self.dtype = dtype
        self.device = torch.device(device)
        self.layers: list[Block] = [_build_layer(s) for s in spec.layers]
        self.final_norm: Norm = build_part(NORMS, spec.final_norm)
        self.embedding: torch.Tensor | None = None
        self.head: torch.Tensor | None = None
        self.rejoin: torch.Tensor | None = None
        self._frequencies: torch.Tensor | None = None

    @property
    def graph_safe_portions(self) -> bool:
        """True when every part (the mixers' position encodings included) may have its prompt portions
        captured in a CUDA graph (``Part.graph_safe_portions``)."""
        parts = [self.final_norm] + [p for block in self.layers for p in [block] + block.parts()]
        parts += [p.position for p in list(parts) if getattr(p, "position", None) is not None]
        return all(getattr(p, "graph_safe_portions", False) for p in parts)

    # ---------------------------------------------------------------- weights
    def expected_tensors(self) -> dict[str, TensorExpectation]:
        exp = {self.spec.embedding_name: TensorExpectation((self.spec.vocab_size, self.spec.hidden_size), "matrix")}
        for block in self.layers:
            for part in block.parts():
                exp.update(part.expected_tensors())
        if self.spec.rejoin_name is not None:
            exp[self.spec.rejoin_name] = TensorExpectation((self.spec.hidden_size, 2 * self.spec.hidden_size), "matrix")
        exp.update(self.final_norm.expected_tensors())
        if self.spec.head_name is not None:
            exp[self.spec.head_name] = TensorExpectation((self.spec.vocab_size, self.spec.hidden_size), "matrix")
        return exp

    def load(self, checkpoint) -> None:
        checkpoint.validate(self.expected_tensors(), self.spec.ignorable_names)
        get = checkpoint.getter(self.dtype, self.device)
        self.embedding = get(self.spec.embedding_name, "matrix")
        for block in self.layers:
            for part in block.parts():
                part.load(get, self.dtype, self.device)
        if self.spec.rejoin_name is not None:
            self.rejoin = get(self.spec.rejoin_name, "matrix").contiguous()
        self.final_norm.load(get, self.dtype, self.device)
        self.head = self.embedding if self.spec.head_name is None else get(self.spec.head_name, "matrix")
        self._sinusoid_frequencies()

    # ------------------------------------------------------------------ cache
    def cache_requirements(self):
        """Per plan entry: (kv requirement | None, state requirement | None,
        reads_cache_of | None).  The state of an entry that reads another's cache is None unless its mixer keeps its
        states itself (``Mixer.keeps_own_states``)."""
        out = []
        for entry in self.spec.plan:
            block = self.layers[entry.layer]
            mixer, extra = block.cache_mixer(), tuple(block.block_states())
            if extra and entry.reads_cache_of is not None:
                raise ValueError("an entry that reads another's cache cannot keep states of its own")
            kv, state = (None, None) if mixer is None else (mixer.kv_requirement(), mixer.state_requirement())
            if extra:
                own = () if state is None else (state,) if isinstance(state, StateRequirement) else tuple(state)
                state = own + extra
            if entry.reads_cache_of is not None:
                if not (mixer is not None and mixer.keeps_own_states):
                    state = None
                owner_kv, owner_state, _ = out[entry.reads_cache_of]
                if kv is not None and owner_kv is not None and kv != owner_kv:
                    # the pages keep what every entry that attends over them needs
                    out[entry.reads_cache_of] = (owner_kv.shared_with(kv), owner_state, None)
            out.append((kv, state, entry.reads_cache_of))
        return out

    def kernel_needs(self) -> dict:
        """Union of what the parts will ask of the kernel modules (``Part.kernel_needs``)."""
        needs: dict = {}
        parts = [self.final_norm] + [p for block in self.layers for p in [block] + block.parts()]
        for part in parts:
            for key, values in part.kernel_needs().items():
                needs.setdefault(key, set()).update(values)
        return needs

    def _sinusoid_frequencies(self):
        """fp32 ``[ceil(width / 2)]``: ``base ** (-2i / width)``, formed in float64 and rounded once."""
        base = self.spec.position_sinusoid_base
        if base is None:
            return None
        if self._frequencies is None:
            i = torch.arange((self.spec.hidden_size + 1) // 2, dtype=torch.float64)
            freq = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / self.spec.hidden_size)
            self._frequencies = freq.to(torch.float32).to(self.device)
        return self._frequencies

    # ---------------------------------------------------------------- forward
    def forward(
        self,
        tokens: torch.Tensor,
        ctx: StepContext,
        caches: list[MixerCache],
        logit_rows: torch.Tensor,
        logits_out: torch.Tensor | None = None,
    ) -> torch.Tensor:
        """Logits ``[len(logit_rows), vocab]`` fp32 of the flat batch ``tokens``."""
        scale = 1.0 if self.spec.embedding_scale is None else self.spec.embedding_scale
        if self.spec.position_sinusoid_base is not None or self.spec.residual_streams > 1:
            from gllm_b200.ops import stateful

            resid = stateful.embed_streams(tokens, self.embedding, ctx.positions, self._sinusoid_frequencies(),
                                           streams=self.spec.residual_streams, sampled=ctx.sampled,
                                           token_row=ctx.token_row, scale=scale)
        elif self.spec.depth_streams:
            # every layer's result is kept beside the embedding output until the step is over
            ctx.depth_streams = torch.empty((len(self.spec.plan) + 1, tokens.numel(), self.spec.hidden_size),
                                            dtype=torch.float32, device=self.device)
            resid = ops.embedding(tokens, self.embedding, out=ctx.depth_streams[0], sampled=ctx.sampled,
                                  token_row=ctx.token_row, scale=scale)
        else:
            resid = ops.embedding(tokens, self.embedding, sampled=ctx.sampled, token_row=ctx.token_row, scale=scale)
        ctx.shared = {}
        branch = None
        first = None
        if any(entry.rejoins_embedding or entry.adds_embedding for entry in self.spec.plan):
            # the embedding output is kept: the residual itself is updated in place by the layers
            first = ops.embedding(tokens, self.embedding, sampled=ctx.sampled, token_row=ctx.token_row, scale=scale)
        for entry_idx, entry in enumerate(self.spec.plan):
            if entry.rejoins_embedding:
                joined = ops.join_rows(None if branch is ops.ADDED else branch, resid, first, self.dtype)
                resid = ops.linear(joined, self.rejoin, out_dtype=torch.float32)
                branch = None
            if entry.adds_embedding:
                # the entry's first norm adds the embedding output together with the branch that is still pending
                branch = ops.Pending.of(branch).with_extra(first)
            branch, resid = self.layers[entry.layer].forward(branch, resid, ctx, caches[entry_idx])
        if logit_rows.numel() == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=self.device)
        final = self.final_norm.forward(None if branch is ops.ADDED else branch, resid, self.dtype, rows=logit_rows)
        logits = ops.linear(final, self.head, out_dtype=torch.float32, out=logits_out)
        if self.spec.logit_scale is not None or self.spec.logit_softcap is not None:
            ops.scale_softcap(logits, 1.0 if self.spec.logit_scale is None else self.spec.logit_scale,
                              self.spec.logit_softcap)
        return logits
