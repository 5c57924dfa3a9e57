"""Pifelix without a GPU: its configuration, the tensors its spec expects, what its layers ask of the cache, what the
cache manager makes of chunks and of layers that read another's pages, the random-weights mode, and the plain
implementation's own consistency."""

import copy
import math

import pytest
import torch

import plain_pifelix as plain
from tiny_pifelix import PIFELIX, _att, _moe, decisive_routing, draw_weights, one_layer, tensor_shapes

F = plain.F


@pytest.mark.parametrize("name", sorted(PIFELIX))
def test_the_spec_expects_exactly_the_tensors_the_design_names(name):
    from gllm_b200.config import load_config
    from gllm_b200.weights.random_init import expected_tensors_of

    shapes = tensor_shapes(PIFELIX[name])
    expected = expected_tensors_of(load_config(copy.deepcopy(PIFELIX[name])))
    assert {k: e.shape for k, e in expected.items()} == shapes


def test_config_round_trip_and_errors():
    from gllm_b200.config import ConfigError, load_config
    from gllm_b200.config.pifelix_config import PifelixConfig

    cfg = load_config(copy.deepcopy(PIFELIX["A"]))
    assert isinstance(cfg, PifelixConfig) and (cfg.hidden_size, cfg.vocab_size, cfg.norm_eps) == (64, 200, 1e-5)
    assert (cfg.embedding_scale, cfg.residual_mult) == (4.0, 0.6)
    assert load_config(cfg.to_dict()) == cfg
    assert load_config(load_config(copy.deepcopy(PIFELIX["B"])).to_dict()).norm_eps == 1e-6

    def broken(change):
        bad = copy.deepcopy(PIFELIX["A"])
        change(bad)
        with pytest.raises(ConfigError):
            load_config(bad)

    mixer = lambda c, i: c["layers"][i]["mixer"]
    broken(lambda c: c["layers"][1].update(type="other"))
    broken(lambda c: mixer(c, 0).update(kv_heads=3))
    broken(lambda c: mixer(c, 0).pop("scale"))
    broken(lambda c: mixer(c, 0).update(conv=0))
    broken(lambda c: mixer(c, 0)["mask"].update(size=0))
    broken(lambda c: mixer(c, 0)["rot"].update(dims=9))
    broken(lambda c: mixer(c, 0)["rot"].update(dims=18))
    broken(lambda c: mixer(c, 0)["rot"]["scaling"].pop("slow"))
    broken(lambda c: mixer(c, 1).update(kv_from=1))
    broken(lambda c: mixer(c, 3).update(kv_from=1))                 # layer 1 has no keys of its own
    broken(lambda c: mixer(c, 1).update(vdim=16))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=9))
    broken(lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.0))
    broken(lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"))
    broken(lambda c: c.pop("residual_mult"))
    broken(lambda c: c.pop("embedding"))
    broken(lambda c: c.update(layers=[]))


def test_spec_parts_and_what_they_ask_of_the_cache():
    from gllm_b200.config import load_config
    from gllm_b200.config.registry import architecture_for
    from gllm_b200.models.decoder import DecoderModel

    spec = architecture_for("Pifelix").build_spec(load_config(copy.deepcopy(PIFELIX["A"])))
    assert spec.head_name == "head" and spec.embedding_scale == 4.0 and spec.ignorable_names == ("l2.norm2",)
    assert [e.reads_cache_of for e in spec.plan] == [None, 0, None, 0]
    assert "feed_forward" not in spec.layers[2].parts
    assert spec.layers[0].mixer_norm.params["multiplier"] == 0.6 and "multiplier" in spec.final_norm.params
    assert spec.final_norm.params["multiplier"] == 1.0
    ff = spec.layers[1].feed_forward.params
    assert (ff["gate_slope"], ff["gate_limit"], ff["up_offset"], ff["weight_on_input"]) == (1.702, 1.5, 1.0, True)
    model = DecoderModel(spec, torch.float32, "cpu")
    assert model.graph_safe_portions
    assert {"conv_qkv", "moe", "postnorm"} <= model.kernel_needs()["modules"]
    needs = model.cache_requirements()
    # the pages of layer 0 keep what its readers' chunks need as well; the readers keep convolution states of their own
    assert needs[0][0].tensors == ((2, 32), (2, 32)) and needs[0][0].chunks == (12, 20, 33)
    assert needs[2][0].chunks == (16,)
    assert [r[1].shape for r in needs] == [(2, 64 + 32 + 48), (3, 64), (1, 48 + 24 + 16), (1, 64)]
    spec = architecture_for("Pifelix").build_spec(load_config(copy.deepcopy(PIFELIX["B"])))
    needs = DecoderModel(spec, torch.float32, "cpu").cache_requirements()
    assert needs[0][1] is None                                       # one tap: no state
    assert not needs[2][0].bounded and needs[2][0].tensors == ((2, 32), (2, 32))


def test_what_a_page_requirement_keeps():
    from gllm_b200.parts.base import KVPageRequirement

    t = ((1, 8), (1, 8))
    chunked = KVPageRequirement(t, chunks=(20,))
    assert chunked.bounded and [chunked.first_needed(p) for p in (0, 19, 20, 39, 40)] == [0, 0, 20, 20, 40]
    both = chunked.shared_with(KVPageRequirement(t, chunks=(33,)))
    assert both.chunks == (20, 33)
    for p in range(200):
        assert both.first_needed(p) == min(p // 20 * 20, p // 33 * 33)
        assert both.first_needed(p) <= both.first_needed(p + 1)
    mixed = chunked.shared_with(KVPageRequirement(t, window=7, keep_first=3))
    assert (mixed.window, mixed.keep_first, mixed.chunks) == (7, 3, (20,))
    assert mixed.first_needed(21) == 15 and mixed.first_needed(35) == 20
    assert not chunked.shared_with(KVPageRequirement(t)).bounded
    assert KVPageRequirement(t).first_needed(50) == 0 and not KVPageRequirement(t).bounded
    with pytest.raises(ValueError):
        chunked.shared_with(KVPageRequirement(((2, 8), (2, 8))))
    with pytest.raises(ValueError):
        KVPageRequirement(t, chunks=(0,))


@pytest.mark.parametrize("block_size,chunks", [(4, (10,)), (4, (8,)), (8, (3,)), (4, (6, 10))])
def test_chunks_give_their_pages_back_when_they_end(block_size, chunks):
    from gllm_b200.cache import CacheManager
    from gllm_b200.parts.base import KVPageRequirement

    req = KVPageRequirement(((1, 4), (1, 4)), chunks=chunks)
    m = CacheManager([(req, None, None)], block_size=block_size, num_blocks=16, max_batch_size=2, max_seq_len=100,
                     dtype=torch.float32, device="cpu")
    m.add_request("a")
    for n_new in (3, 1, 7, 1, 1, 12, 2, 30, 1, 5):
        slots = m.append("a", n_new)[0]
        assert (slots >= 0).all()
        m.commit("a", n_new)
        n, blocks = m.requests["a"].num_tokens, m.requests["a"].blocks[0]
        need = min(n // c * c for c in chunks) // block_size
        assert [b >= 0 for b in blocks] == [i >= need for i in range(len(blocks))], n
        m.check_invariants()
    assert m.groups[0].allocator.total_reused > 0
    m.free_request("a")
    assert m.num_free_pages() == 16


def test_a_reader_of_anothers_pages_keeps_its_own_states_when_it_names_some():
    from gllm_b200.cache import CacheManager
    from gllm_b200.parts.base import KVPageRequirement, StateRequirement

    kv = KVPageRequirement.keys_and_values(1, 16)
    reqs = [(kv, StateRequirement((2, 3)), None), (kv, StateRequirement((5,)), 0), (kv, None, 0)]
    m = CacheManager(reqs, 4, 8, 2, 32, torch.float32, "cpu")
    owner, reader, sharing = m.mixer_caches()
    assert owner.writes and not reader.writes and not sharing.writes
    assert reader.pages.data_ptr() == owner.pages.data_ptr() and reader.group == owner.group
    assert tuple(reader.state.shape) == (3, 5) and sharing.state is owner.state
    rc = m.add_request("a")
    owner.state[rc.slot], reader.state[rc.slot] = 1.0, 2.0
    other = m.add_request("b")
    assert float(reader.state[rc.slot].min()) == 2.0 and float(reader.state[other.slot].abs().max()) == 0.0
    m.free_request("a")
    again = m.add_request("c")
    assert again.slot == rc.slot
    assert float(owner.state[again.slot].abs().max()) == 0.0 and float(reader.state[again.slot].abs().max()) == 0.0


def test_a_reader_with_other_heads_is_refused():
    from gllm_b200.models.decoder import DecoderModel
    from gllm_b200.models.pifelix import build_pifelix_spec
    from gllm_b200.config import load_config
    from gllm_b200.models.spec import ModelSpec
    import dataclasses

    spec = build_pifelix_spec(load_config(copy.deepcopy(PIFELIX["A"])))
    plan = list(spec.plan)
    plan[2] = dataclasses.replace(plan[2], reads_cache_of=0)          # layer 2 has heads of other widths
    with pytest.raises(ValueError):
        DecoderModel(dataclasses.replace(spec, plan=tuple(plan)), torch.float32, "cpu").cache_requirements()
    assert isinstance(spec, ModelSpec)


def test_how_many_spans_a_decoded_token_reads():
    from gllm_b200.ops.attention_bf16 import visible_spans

    for span in (128, 256):
        for window in (0, 1, 5, 128, 129, 300, 1000, -1, -3, -64, -100, -128, -256, -300, -512, -1000):
            worst = 0
            for p in range(3000):
                first = max(0, p - window + 1) if window > 0 else (p // -window * -window if window < 0 else 0)
                worst = max(worst, p // span - first // span + 1)
            got = visible_spans(3000, span, window)
            assert worst <= got <= worst + (0 if window <= 0 and window % span == 0 else 1), (span, window)


def test_yarn_frequencies_of_the_part_match_the_plain_ones():
    from gllm_b200.parts.rotary import rotary_magnitude, scaled_inverse_frequencies

    for dims, base, s in ((24, 10000.0, (4.0, 64, 16.0, 1.0)), (40, 300.0, (16.0, 48, 4.0, 0.25)), (8, 5e5, (2.0, 4096, 32.0, 1.0)),
                          (16, 10000.0, (8.0, 8, 1.0, 0.9)), (12, 50.0, None)):
        rot = {"base": base, "dims": dims}
        if s:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), s))
        part = s and {"rope_type": "yarn", "factor": s[0], "original_max_position_embeddings": s[1], "beta_fast": s[2],
                      "beta_slow": s[3]}
        assert scaled_inverse_frequencies(dims, base, part or None) == pytest.approx(plain.yarn_frequencies(rot), rel=1e-12)
        assert rotary_magnitude(part or None) == pytest.approx(plain.yarn_magnitude(rot), rel=1e-12)


def test_random_weights_cover_the_spec():
    from gllm_b200.config import load_config
    from gllm_b200.weights.random_init import random_tensors

    t = random_tensors(load_config(copy.deepcopy(PIFELIX["A"])), seed=1)
    assert {k: tuple(v.shape) for k, v in t.items()} == tensor_shapes(PIFELIX["A"])


# ------------------------------------------------------------------ the plain implementation against itself
def test_plain_convolution_is_a_filter_over_time():
    g = torch.Generator().manual_seed(1)
    u, w = torch.randn(11, 5, generator=g, dtype=F), torch.randn(5, 4, generator=g, dtype=F)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (3, 0)), w[:, None], groups=5)[0].T
    assert torch.allclose(plain.causal_conv(u, w), want)


def test_plain_chunks_are_separate_sequences_for_attention():
    g = torch.Generator().manual_seed(2)
    q, k, v = (torch.randn(25, h, 6, generator=g, dtype=F) for h in (4, 2, 2))
    p = torch.arange(25)
    whole = plain.attend(q, k, v, p, p, 0.3, 10)
    for lo in (0, 10, 20):
        hi = min(lo + 10, 25)
        part = plain.attend(q[lo:hi], k[lo:hi], v[lo:hi], p[lo:hi], p[lo:hi], 0.3, None)
        assert torch.allclose(whole[lo:hi], part)


def test_plain_expert_clamps_gate_above_only_and_up_on_both_sides():
    w = {"e.gate": torch.tensor([[1.0]], dtype=F), "e.up": torch.tensor([[2.0]], dtype=F), "e.down": torch.tensor([[1.0]], dtype=F)}
    for h in (-9.0, -0.4, 0.1, 5.0):
        g, u = min(h, 1.5), min(max(2 * h, -1.5), 1.5)
        want = g / (1 + math.exp(-1.702 * g)) * (u + 1)
        assert float(plain.expert(torch.tensor([[h]], dtype=F), w, "e", 1.5)) == pytest.approx(want)


def test_plain_weights_enter_ahead_of_the_activation():
    cfg = one_layer(_att(2, 1, 8, 8, 0.3, 9, 2, 8), _moe(12, 3, 3, 0.5), width=24, vocab=40)
    w = {k: v.to(F) for k, v in decisive_routing(cfg, draw_weights(cfg, seed=2)).items()}
    x = torch.randn(5, 24, generator=torch.Generator().manual_seed(3), dtype=F) * 3
    mlp = cfg["layers"][0]["mlp"]
    got = plain.routed_experts(x, w, "l0.mlp", mlp)
    s = plain.sigmoid(x @ w["l0.mlp.router"].T)
    on_input = sum(plain.expert(s[:, e:e + 1] * x, w, f"l0.mlp.e{e}", 0.5) for e in range(3))
    on_output = sum(s[:, e:e + 1] * plain.expert(x, w, f"l0.mlp.e{e}", 0.5) for e in range(3))
    assert torch.allclose(got, on_input) and float((on_input - on_output).abs().max()) > 0.05


def test_plain_prefix_does_not_depend_on_what_follows():
    cfg = PIFELIX["A"]
    w = decisive_routing(cfg, draw_weights(cfg, seed=4))
    toks = torch.randint(0, cfg["vocab"], (45,), generator=torch.Generator().manual_seed(5)).tolist()
    full = plain.forward(cfg, w, toks)
    for n in (1, 2, 19, 21, 34):
        assert torch.allclose(plain.forward(cfg, w, toks[:n]), full[:n], atol=1e-9)
