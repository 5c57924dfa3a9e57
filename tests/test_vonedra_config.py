"""Vonedra without a GPU: its configuration, the tensors its spec expects, what its layers ask of the cache and what the
cache manager makes of a window that keeps the first tokens, the buckets of distances, the random-weights mode, and the
plain implementation's own consistency (mechanisms against independent restatements, a prompt against its portions)."""

import copy
import math

import pytest
import torch

import plain_vonedra as plain
from tiny_vonedra import VONEDRA, _att, _delta, _latent, draw_weights, one_layer, tensor_shapes

F = plain.F


@pytest.mark.parametrize("name", sorted(VONEDRA))
def test_the_spec_expects_exactly_the_tensors_the_design_names(name):
    from gllm_b200.config import load_config
    from gllm_b200.weights.random_init import expected_tensors_of

    cfg = VONEDRA[name]
    shapes = tensor_shapes(cfg)
    expected = expected_tensors_of(load_config(copy.deepcopy(cfg)))
    assert set(expected) == set(shapes)
    for key, exp in expected.items():
        assert len(exp.shape) == len(shapes[key]), key
        assert all(a in (b, -1) for a, b in zip(exp.shape, shapes[key])), key
    unknown = {k for k, e in expected.items() if -1 in e.shape}
    assert unknown == {f"l{i}.mix.rel" for i, l in enumerate(cfg["layers"])
                       if l["type"] == "attention" and "bias_rows" not in l["mixer"]}


def test_config_round_trip_and_errors():
    from gllm_b200.config import ConfigError, load_config
    from gllm_b200.config.vonedra_config import VonedraConfig

    cfg = load_config(copy.deepcopy(VONEDRA["A"]))
    assert isinstance(cfg, VonedraConfig) and cfg.hidden_size == 64 and cfg.vocab_size == 200 and cfg.conv_taps == 3
    assert cfg.norm_eps == 1e-5 and cfg.embedding_scale == 5.0 and cfg.value_mixing_layers() == [0, 4]
    assert [l.type for l in cfg.layers] == ["attention", "latent_attention", "attention", "delta", "attention"]
    again = load_config(cfg.to_dict())
    assert again == cfg

    def broken(change):
        bad = copy.deepcopy(VONEDRA["A"])
        change(bad)
        with pytest.raises(ConfigError):
            load_config(bad)

    broken(lambda c: c["layers"][1].update(type="other"))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mixer"].pop("bias_max"))
    broken(lambda c: c["layers"][0]["mixer"].update(bias_max=0))
    broken(lambda c: c["layers"][0]["mixer"].update(bias_rows=100))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].pop("size"))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1))
    broken(lambda c: c["layers"][0]["mixer"].update(vdim=8))                   # layer 4 mixes values of another size
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3))
    broken(lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=2))     # latent attention keeps none
    broken(lambda c: c["layers"][1]["mixer"].pop("q_rank"))
    broken(lambda c: c["layers"][3]["mixer"].update(conv=0))
    broken(lambda c: c["layers"][0].update(mlp={"kind": "sparse", "ff": 8}))
    broken(lambda c: c["layers"][0].update(mlp={"kind": "dense", "ff": 0}))
    broken(lambda c: c["canon"].update(taps=0))
    broken(lambda c: c.pop("canon"))
    broken(lambda c: c["embedding"].pop("scale"))


def test_spec_parts_and_what_they_ask_of_the_cache():
    from gllm_b200.config import load_config
    from gllm_b200.config.registry import architecture_for
    from gllm_b200.models.decoder import DecoderModel

    spec = architecture_for("Vonedra").build_spec(load_config(copy.deepcopy(VONEDRA["A"])))
    assert spec.depth_streams and spec.head_name == "head" and spec.ignorable_names == ("l2.mix.vmix", "l2.norm2", "l2.canon2")
    assert [l.mixer.params.get("value_mix") for l in spec.layers] == ["first", None, None, None, "mixed"]
    assert [l.depth_average.params["streams"] for l in spec.layers] == [2, 3, 4, 5, 6]
    assert "feed_forward" not in spec.layers[2].parts
    model = DecoderModel(spec, torch.float32, "cpu")
    assert model.graph_safe_portions
    needs = model.cache_requirements()
    kv = [r[0] for r in needs]
    assert kv[0].tensors == ((2, 16), (2, 24)) and (kv[0].window, kv[0].keep_first) == (20, 5)
    assert kv[1].tensors == ((1, 40),) and (kv[1].window, kv[1].keep_first) == (33, 0)
    assert kv[3] is None
    states = [[s.shape for s in r[1]] for r in needs]
    assert states[0] == [(2, 64), (2, 64)] and states[2] == [(2, 64)]
    assert states[3] == [(4, 24, 16), (3, 2 * 2 * 16 + 4 * 24), (2, 64), (2, 64)]


def test_a_window_gives_pages_back_but_those_of_the_first_tokens():
    from gllm_b200.cache import CacheManager
    from gllm_b200.parts.base import KVPageRequirement

    plain_window, keeping = KVPageRequirement(((1, 4),), 10), KVPageRequirement(((1, 4),), 10, 5)
    cache = CacheManager([(plain_window, None, None), (keeping, None, None)], block_size=4, num_blocks=12, max_batch_size=2,
                         max_seq_len=48, dtype=torch.float32, device="cpu")
    assert len(cache.groups) == 2
    cache.add_request("a")
    for n in (7, 1, 12, 2, 20, 1):
        cache.append("a", n)
        cache.commit("a", n)
        total = cache.requests["a"].num_tokens
        for group, keep in zip(cache.groups, (0, 5)):
            blocks = cache.requests["a"].blocks[group.index]
            for b, page in enumerate(blocks):
                # the next token sees positions >= total - 9, and the kept ones
                needed = (b + 1) * 4 > total - 9 or b * 4 < keep
                assert (page >= 0) == needed, (total, b, keep)
                assert group.block_table_host[cache.requests["a"].slot, b] == page
    cache.check_invariants()
    assert cache.groups[0].allocator.num_held == 3 and cache.groups[1].allocator.num_held == 5
    cache.free_request("a")
    cache.check_invariants()
    assert all(g.allocator.num_held == 0 for g in cache.groups)


@pytest.mark.parametrize("rows,far", [(16, 240), (12, 50), (8, 64), (32, 128), (6, 100), (7, 50), (2, 30), (3, 12), (16, 9),
                                      (12, 30.5), (40, 5000)])
def test_buckets_of_distances(rows, far):
    """Against the formula with logarithms wherever those do not fall on a border, and against powers at borders."""
    from gllm_b200.ops.distance import distance_buckets

    n_max = int(far) + 300
    got = distance_buckets(rows, far, n_max)
    half = rows // 2
    assert got[:half] == list(range(min(half, n_max))) and got[-1] == rows - 1 and got == sorted(got)
    for n in range(half, n_max):
        x = math.log(n / half) / math.log(far / half) * (rows - half)
        if abs(x - round(x)) > 1e-9:
            assert got[n] == min(rows - 1, half + math.floor(x)), n
    if n_max < 1000:
        assert got == [plain.distance_bucket(n, rows, far) for n in range(n_max)]
    if (rows, far) == (8, 64):                             # 4 * 2^k: the borders are exact
        assert [got.index(b) for b in (4, 5, 6, 7)] == [4, 8, 16, 32]


def test_bias_table_holds_one_value_per_distance():
    from gllm_b200.ops.distance import DistanceBias

    rel = torch.arange(12.0).view(6, 2)
    b = DistanceBias.build(rel, 20, torch.tensor([0.5, -1.0]))
    assert b.table.shape == (2, 21)
    for n in range(21):
        assert b.table[0, n] == rel[plain.distance_bucket(n, 6, 20), 0]
    assert b.table[1, -1] == rel[5, 1] and torch.allclose(b.sink_log2, torch.tensor([0.5, -1.0]) * math.log2(math.e))


def test_random_weights_need_the_rows_of_the_bias_named():
    from gllm_b200.config import load_config
    from gllm_b200.weights.random_init import random_tensors

    drawn = random_tensors(load_config(copy.deepcopy(VONEDRA["A"])), seed=1)
    assert {k: tuple(v.shape) for k, v in drawn.items()} == tensor_shapes(VONEDRA["A"])
    with pytest.raises(ValueError, match="rel"):
        random_tensors(load_config(copy.deepcopy(VONEDRA["C"])), seed=1)


# ------------------------------------------------------------------ the plain implementation itself
@pytest.mark.parametrize("name", sorted(VONEDRA))
def test_plain_portions_equal_the_whole(name):
    cfg = VONEDRA[name]
    w = draw_weights(cfg, seed=2)
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = plain.forward(cfg, w, toks)
    state, got, p = plain.PlainState(cfg), [], 0
    for n in (1, 2, 30, 1, 1, 25):
        got.append(plain.forward(cfg, w, toks[p:p + n], state))
        p += n
    assert torch.allclose(torch.cat(got), whole, atol=1e-10)


def test_plain_convolution_and_delta_rule():
    g = torch.Generator().manual_seed(3)
    x, w = torch.randn(9, 5, generator=g, dtype=F), torch.randn(5, 4, generator=g, dtype=F)
    y, kept = plain.causal_conv(x, w, torch.zeros(3, 5, dtype=F))
    for t in range(9):
        for c in range(5):
            assert math.isclose(y[t, c], sum(w[c, j] * x[t - 3 + j, c] for j in range(4) if t - 3 + j >= 0), abs_tol=1e-12)
    assert torch.equal(kept, x[-3:])
    # the corrected write makes a unit key's read-out its value when beta is 1 and nothing decays
    k = plain.unit(torch.randn(1, 2, 6, generator=g, dtype=F) * 50)
    v = torch.randn(1, 2, 3, generator=g, dtype=F)
    S = torch.randn(2, 6, 3, generator=g, dtype=F)
    one = torch.ones(1, 2, dtype=F)
    o = plain.delta_rule(k, k, v, one, one, S)
    assert torch.allclose(o, v, atol=1e-6)


def test_plain_attention_edges():
    """What a query sees at the edges of the window and of the kept tokens; the sink takes its share."""
    pos = torch.arange(12)
    ok = plain.visible(pos, pos, size=4, keep_first=2)
    assert ok[9].nonzero().flatten().tolist() == [0, 1, 6, 7, 8, 9] and ok[0].sum() == 1
    assert plain.visible(pos, pos, size=4)[9].nonzero().flatten().tolist() == [6, 7, 8, 9]
    q = torch.zeros(1, 1, 2, dtype=F)
    k, v = torch.zeros(3, 1, 2, dtype=F), torch.ones(3, 1, 1, dtype=F)
    o = plain.attend(q, k, v, torch.tensor([2]), torch.arange(3), 1.0, None, sink=torch.tensor([math.log(2.0)], dtype=F))
    assert math.isclose(float(o), 3 / 5, rel_tol=1e-12)


@pytest.mark.parametrize("mixer", [_att(2, 1, 8, 8, 0.5, 20, size=6, keep=2), _latent(2, 8, 4, 8, 12, 8, 0.4, size=6),
                                   _delta(2, 1, 8, 8, 2)])
def test_plain_logits_do_not_look_ahead(mixer):
    cfg = one_layer(mixer, 24, width=32, vocab=50)
    w = draw_weights(cfg, seed=5)
    toks = torch.randint(0, 50, (20,), generator=torch.Generator().manual_seed(2)).tolist()
    a = plain.forward(cfg, w, toks)
    b = plain.forward(cfg, w, toks[:12] + [1] * 8)
    assert torch.equal(a[:12], b[:12]) and not torch.allclose(a[13], b[13])
