"""Pifelix on the GPU against the plain implementation: each kernel of its mechanisms alone, each mechanism alone in a
model of one layer, whole prompts against token by token decoding and portions of every size, mixed batches over a pool
so small that pages and state slots are used again, decisive keys just inside and just outside a chunk and at page
borders, the first tokens, long decoding through the decode graphs, sizes of every kind, layers that read another
layer's keys, and greedy generation through the engine."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_pifelix as plain
from replay_helpers import (BF16_TOL_MAX, BF16_TOL_MEAN, FP32_TOL, LENGTHS, compare, mixed_steps, replay, rounded,
                            run_steps, sequences, single_request_steps)
from tiny_pifelix import PIFELIX, _att, _moe, decisive_routing, draw_weights, one_layer, write_model

pytestmark = pytest.mark.gpu

PAGE = {"A": 4, "B": 8, "C": 16}
F = plain.F


def tolerance(dtype):
    return (FP32_TOL, None) if dtype == "float32" else (BF16_TOL_MAX, BF16_TOL_MEAN)


def make(cfg, tmp_path, dtype, seed=7, max_tokens=512, block_size=16, max_live=4, sharp=None, weights=None):
    from gllm_b200.engine.replay import build_runner

    sharp = (1.5 if dtype == "float32" else 1.0) if sharp is None else sharp
    if weights is None:
        weights = decisive_routing(cfg, draw_weights(cfg, seed=seed, sharp=sharp))
    folder = write_model(cfg, weights, str(tmp_path / "model"))
    _, runner = build_runner(folder, dtype, max_tokens, block_size=block_size, max_live=max_live)
    return weights, folder, runner


def steps_of(tokens, cuts, rid="r", first_step=0, end=True):
    """One request fed in portions of the given sizes; every logit is wanted."""
    steps, index, p = [], [], 0
    for i, n in enumerate(cuts):
        last = p + n == len(tokens)
        steps.append({"step": first_step + i, "entries": [{"id": rid, "tokens": tokens[p:p + n], "want": list(range(n))}],
                      "end": [rid] if (last and end) else []})
        index += [(first_step + i, k, rid, p + k) for k in range(n)]
        p += n
    assert p == len(tokens)
    return steps, index


class _Step:
    """What the kernels read of a step: requests that bring ``lengths`` tokens from positions ``starts`` on, on state
    slots that are not their numbers; portions first, single tokens after them."""

    def __init__(self, lengths, starts, slots):
        from gllm_b200.engine.step import Workspace

        dev = "cuda"
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        self.cu_q = i32([0] + list(np.cumsum(lengths)))
        self.context_lens, self.state_slots = i32(starts), i32(slots)
        self.positions = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lengths)]).to(torch.int32).to(dev)
        self.token_row = torch.cat([torch.full((n,), s) for s, n in zip(slots, lengths)]).to(torch.int32).to(dev)
        self.num_requests, self.max_q_len = len(lengths), max(lengths)
        self.max_seq_len = max(s + n for s, n in zip(starts, lengths))
        multi = [n for n in lengths if n > 1]
        assert list(lengths[:len(multi)]) == multi
        self.num_prefill_requests, self.num_prefill_tokens = len(multi), sum(multi)
        self.workspace = Workspace(dev)


def _tables(total, page, slot_of, seed=0):
    """Shuffled pages for requests of the given lengths: (block table, number of pages)."""
    g = torch.Generator().manual_seed(seed)
    per = {r: -(-n // page) for r, n in total.items()}
    n_pages = sum(per.values()) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((max(slot_of.values()) + 2, max(per.values())), -1, dtype=torch.int32)
    for r in total:
        for i in range(per[r]):
            table[slot_of[r], i] = order.pop()
    return table, n_pages


def _slots(table, row, start, n, page):
    return [int(table[row, t // page]) * page + t % page for t in range(start, start + n)]


# ------------------------------------------------------------------ the kernels of each mechanism alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dk,dv,taps,dims,own,splits", [
    (4, 2, 16, 24, 3, 8, True, 0), (3, 1, 10, 7, 6, 10, True, 0), (2, 2, 64, 64, 4, 64, True, 3), (6, 3, 40, 56, 2, 20, True, 0),
    (4, 2, 64, 48, 4, 32, False, 0), (1, 1, 128, 96, 4, 128, True, 5), (2, 1, 9, 5, 1, 4, True, 2), (8, 2, 24, 72, 9, 0, True, 0),
    (2, 1, 200, 130, 4, 50, True, 0), (3, 3, 12, 12, 16, 12, False, 2), (20, 4, 64, 64, 4, 64, True, 0)])
def test_bias_convolution_norm_rotation_and_store(dtype, heads, kv_heads, dk, dv, taps, dims, own, splits):
    """The kernel between the fused projection and the attention, for two requests in several steps (long portions that
    are cut into runs, portions beside single tokens, single tokens), against the plain functions; the projection as a
    slice of wider rows or as unsummed splits."""
    from gllm_b200 import ops
    from gllm_b200.ops.conv_qkv import conv_qkv
    from gllm_b200.parts.attention import stored_head_width

    g = torch.Generator().manual_seed(heads * 100 + dk)
    rot = {"base": 500.0, "dims": dims, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}}
    eps, page, dp = 1e-3, 8, stored_head_width(dk, dv)
    cols = [("q", heads * dk)] + ([("k", kv_heads * dk), ("v", kv_heads * dv)] if own else [])
    channels = sum(c for _, c in cols)
    total = {0: 150, 1: 41}
    n_parts = max(splits, 1)
    parts = {r: torch.randn(n_parts, n, channels, generator=g) / n_parts ** 0.5 for r, n in total.items()}
    proj = {r: p.sum(0).to(dtype).float() for r, p in parts.items()}
    bias, conv_w = torch.randn(channels, generator=g) * 0.5, torch.randn(channels, taps, generator=g) * 0.6
    qn, kn = 1 + torch.randn(dk, generator=g) * 0.3, 1 + torch.randn(dk, generator=g) * 0.3

    def plain_request(r):
        y = plain.causal_conv(proj[r].to(F) + bias.to(F), conv_w.to(F))
        p, T = torch.arange(total[r]), total[r]
        q = plain.rotate_pairs(plain.rms(y[:, :heads * dk].reshape(T, heads, dk), qn.to(F), eps), p, rot)
        if not own:
            return q, None, None
        k = y[:, heads * dk: (heads + kv_heads) * dk].reshape(T, kv_heads, dk)
        return q, plain.rotate_pairs(plain.rms(k, kn.to(F), eps), p, rot), y[:, -kv_heads * dv:].reshape(T, kv_heads, dv)

    want = {r: plain_request(r) for r in total}
    inv_freq = torch.tensor(plain.yarn_frequencies(rot), dtype=torch.float32).cuda() if dims else None
    slot_of = {0: 3, 1: 1}
    table, n_pages = _tables(total, page, slot_of)
    cache = torch.full((n_pages, 2, kv_heads, page, dp), 5.0, device="cuda", dtype=dtype)
    state = torch.full((5, taps - 1, channels), 7.0, device="cuda")
    for s in slot_of.values():
        state[s] = 0.0                                              # a request's slot starts at zero
    done, got = {0: 0, 1: 0}, {r: [] for r in total}
    for plan in ([(0, 9), (1, 2)], [(0, 2), (1, 1)], [(0, 1), (1, 1)], [(0, 90), (1, 17)], [(1, 20), (0, 1)], [(0, 47)]):
        lengths, starts = [n for _, n in plan], [done[r] for r, _ in plan]
        step = _Step(lengths, starts, [slot_of[r] for r, _ in plan])
        chunk = torch.cat([parts[r][:, done[r]:done[r] + n] for r, n in plan], 1).cuda()
        if splits:
            x = ops.SplitSum(chunk.contiguous(), dtype)
        else:
            x = torch.cat([torch.zeros(chunk.shape[1], 8, device="cuda"), chunk[0]], 1).to(dtype)[:, 8:]
        where = torch.tensor([v for r, n in plan for v in _slots(table, slot_of[r], done[r], n, page)], dtype=torch.int32)
        q = conv_qkv(x, bias.cuda(), conv_w.t().contiguous().cuda(), state, qn.cuda(), kn.cuda() if own else None, eps,
                     inv_freq, dims, plain.yarn_magnitude(rot), where.cuda(), cache, heads, kv_heads, dk, dv, dp, step,
                     own_kv=own)
        at = 0
        for r, n in plan:
            got[r].append(q[at:at + n].double().cpu().view(n, heads, dp))
            at += n
            done[r] += n
    ops.check_status()
    tol = dict(atol=2e-4, rtol=2e-4) if dtype == torch.float32 else dict(atol=3e-2, rtol=1e-2)
    pages = cache.double().cpu()
    for r in total:
        q = torch.cat(got[r])
        assert done[r] == q.shape[0] and torch.allclose(q[..., :dk], want[r][0][:done[r]], **tol), r
        assert float(q[..., dk:].abs().max() if dk < dp else 0.0) == 0.0
        last = (proj[r] + bias)[max(0, done[r] - taps + 1):done[r]]
        assert torch.allclose(state[slot_of[r]].cpu(), last, atol=1e-5)
        if own:
            for t in range(done[r]):
                k, v = pages[int(table[slot_of[r], t // page]), :, :, t % page]
                assert torch.allclose(k[:, :dk], want[r][1][t], **tol) and torch.allclose(v[:, :dv], want[r][2][t], **tol), t
                assert float(k[:, dk:].abs().sum() + v[:, dv:].abs().sum()) == 0.0
    if not own:
        assert float(cache.min()) == 5.0 == float(cache.max())      # a layer that reads another's keys stores nothing
    if taps > 1:
        assert float(state[0].min()) == 7.0 == float(state[4].min())   # the other slots are untouched


@pytest.mark.parametrize("heads,kv_heads,d,page,chunk", [
    (4, 2, 64, 16, 40), (8, 2, 64, 16, 64), (4, 4, 64, 16, 200), (2, 1, 128, 16, 150), (4, 1, 32, 8, 30), (6, 3, 64, 8, 128),
    (4, 2, 64, 32, 7), (3, 1, 48, 4, 25), (2, 2, 136, 16, 100), (4, 2, 64, 16, 256), (4, 2, 64, 16, 300)])
@pytest.mark.parametrize("kernel", ["float32", "bf16", "bf16_stream"])
def test_attention_within_chunks(kernel, heads, kv_heads, d, page, chunk, monkeypatch):
    """Every attention kernel of the paged cache with a chunk: two requests over shuffled pages in portions and single
    tokens, against the plain function.  A page is taken from its request (its entry in the block table becomes -1 and
    its contents enormous) as soon as the chunk has left it; a comparison with chunks one position off must fail."""
    from gllm_b200 import ops
    from gllm_b200.ops import attention_bf16

    dtype = torch.float32 if kernel == "float32" else torch.bfloat16
    if kernel == "bf16_stream":
        if d not in (64, 128) or page not in (16, 32):
            pytest.skip("sizes the persistent decode kernel does not take")
        monkeypatch.setattr(attention_bf16, "STREAM_MIN_ITEMS", 1)
    g = torch.Generator().manual_seed(heads * 100 + d + chunk)
    total, slot_of, scale = {0: 700, 1: 150}, {0: 2, 1: 0}, 2.0 * d ** -0.5
    rnd = lambda n, h: torch.randn(n, h, d, generator=g).to(dtype)
    q, k, v = ({r: rnd(n, h) for r, n in total.items()} for h in (heads, kv_heads, kv_heads))
    pos = {r: torch.arange(n) for r, n in total.items()}
    want = {r: plain.attend(q[r].to(F), k[r].to(F), v[r].to(F), pos[r], pos[r], scale, chunk) for r in total}
    table, n_pages = _tables(total, page, slot_of)
    cache = torch.zeros((n_pages, 2, kv_heads, page, d), device="cuda", dtype=dtype)
    done, got = {0: 0, 1: 0}, {r: [] for r in total}
    plans = [[(0, 190), (1, 38)], [(0, 2), (1, 1)], [(0, 7), (1, 3)], [(0, 1), (1, 1)], [(0, 1), (1, 1)], [(1, 90), (0, 1)],
             [(0, 64)], [(0, 130)], [(0, 2)]] + [[(0, 1), (1, 1)]] * 6 + [[(0, 250)]] + [[(0, 1)]] * 3
    for plan in plans:
        lengths, starts = [n for _, n in plan], [done[r] for r, _ in plan]
        step = _Step(lengths, starts, [slot_of[r] for r, _ in plan])
        for r, n in plan:
            for t in range(done[r], done[r] + n):
                p = int(table[slot_of[r], t // page])
                cache[p, 0, :, t % page], cache[p, 1, :, t % page] = k[r][t].cuda(), v[r][t].cuda()
            for b in range(done[r] // chunk * chunk // page):       # what this step's first token no longer needs
                if int(table[slot_of[r], b]) >= 0:
                    cache[int(table[slot_of[r], b])] = 1e30
                    table[slot_of[r], b] = -1
        qs = torch.cat([q[r][done[r]:done[r] + n].reshape(n, -1) for r, n in plan]).cuda()
        out = ops.paged_attention(qs, cache, table.cuda(), step.positions, step.token_row, heads, scale, batch=step, chunk=chunk)
        at = 0
        for r, n in plan:
            got[r].append(out[at:at + n].double().cpu())
            at += n
            done[r] += n
    ops.check_status()
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    for r in total:
        n = done[r]
        err = float((torch.cat(got[r]) - want[r][:n]).abs().max())
        assert err < tol, (r, err)
        for other in (chunk - 1, chunk + 1, None):
            off = plain.attend(q[r][:n].to(F), k[r][:n].to(F), v[r][:n].to(F), pos[r][:n], pos[r][:n], scale, other)
            assert n <= chunk or float((off - want[r][:n]).abs().max()) > 10 * tol


def test_window_of_a_decoded_token_over_compact_spans(monkeypatch):
    """Windows (not chunks) through both decode kernels, whose grids count spans from the window's first key."""
    from gllm_b200 import ops
    from gllm_b200.ops import attention_bf16

    g = torch.Generator().manual_seed(5)
    heads, kv_heads, d, page, n = 4, 2, 64, 16, 900
    k, v = (torch.randn(n, kv_heads, d, generator=g).to(torch.bfloat16) for _ in range(2))
    table, n_pages = _tables({0: n}, page, {0: 1})
    cache = torch.zeros((n_pages, 2, kv_heads, page, d), device="cuda", dtype=torch.bfloat16)
    for t in range(n):
        p = int(table[1, t // page])
        cache[p, 0, :, t % page], cache[p, 1, :, t % page] = k[t].cuda(), v[t].cuda()
    for stream in (1, 10 ** 9):
        monkeypatch.setattr(attention_bf16, "STREAM_MIN_ITEMS", stream)
        for window in (1, 2, 100, 128, 129, 256, 257, 600, 2000):
            for p in (0, 127, 128, 255, 256, 511, 640, 899):
                q = torch.randn(1, heads, d, generator=g).to(torch.bfloat16)
                step = _Step([1], [p], [1])
                out = ops.paged_attention(q.view(1, -1).cuda(), cache, table.cuda(), step.positions, step.token_row, heads, 0.2,
                                          window=window, batch=step)
                lo = max(0, p - window + 1)
                want = plain.attend(q.to(F), k[lo:p + 1].to(F), v[lo:p + 1].to(F), torch.tensor([p]), torch.arange(lo, p + 1), 0.2, None)
                assert float((out.double().cpu() - want).abs().max()) < 2e-2, (stream, window, p)
    ops.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width", [(5, 64), (3, 50), (70, 1024), (1, 7), (2, 2304)])
def test_norm_of_a_result_and_the_residual_as_it_is(dtype, rows, width):
    """``resid += rms(value) * w`` and the sum rounded: the value as a tensor, as unsummed splits, and none."""
    from gllm_b200 import ops

    g = torch.Generator().manual_seed(rows * width)
    resid, w = torch.randn(rows, width, generator=g) * 3, torch.randn(width, generator=g)
    parts = torch.randn(4, rows, width, generator=g)
    value = parts.sum(0).to(dtype)
    want = resid.double() + plain.rms(value.double(), w.double(), 1e-3)
    for branch in (value.cuda(), ops.SplitSum(parts.cuda(), dtype)):
        r = resid.cuda()
        got = ops.add_cast(ops.Pending(branch, w.cuda(), 1e-3), r, dtype)
        assert torch.allclose(r.double().cpu(), want, atol=1e-2 if isinstance(branch, ops.SplitSum) and dtype != torch.float32 else 1e-5)
        assert torch.equal(got, r.to(dtype))
    r = resid.cuda()
    assert torch.equal(ops.add_cast(None, r, dtype), resid.cuda().to(dtype)) and torch.equal(r.cpu(), resid)
    r = resid.cuda()
    assert torch.equal(ops.add_cast(value.cuda(), r, dtype), r.to(dtype))
    assert torch.allclose(r.cpu(), resid + value.float(), atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,width,ff,experts,top,limit", [(37, 64, 64, 8, 2, 0.5), (1, 44, 20, 4, 1, 1.0), (300, 128, 64, 16, 4, 0.3),
                                                         (9, 48, 24, 6, 6, 2.0), (1500, 256, 128, 4, 2, 0.7), (130, 64, 192, 3, 1, 0.4),
                                                         (3, 64, 1024, 4, 2, 0.6), (100, 128, 64, 8, 2, 0.5),
                                                         (60, 200, 320, 6, 2, 0.5), (2, 136, 576, 9, 3, 1.1)])
def test_experts_with_weights_on_their_inputs_and_a_clamped_gate(dtype, n, width, ff, experts, top, limit):
    """``sum_s expert(w_s x)``: bf16 sizes that the tensor-core kernel takes run there, the others (and float32) on the
    CUDA cores.  The clamps bite, and the weights on the output, or no clamps, would give another result."""
    from gllm_b200 import ops
    from gllm_b200.ops import moe

    g = torch.Generator().manual_seed(n + width)
    rnd = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
    x, wg, wu = rnd(n, width), rnd(experts, ff, width) / math.sqrt(width), rnd(experts, ff, width) / math.sqrt(width)
    wg, wu = wg.to(dtype).float(), wu.to(dtype).float()
    wd = (rnd(experts, width, ff) / math.sqrt(ff)).to(dtype).float()
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    wts = torch.rand(n, top, generator=g) + 0.05

    def reference(limit, on_input=True):
        gate, up = (torch.einsum("tw,efw->tef", x.to(F), w.to(F)) for w in (wg, wu))
        out = torch.zeros(n, width, dtype=F)
        for s in range(top):
            e, a = ids[:, s].long(), wts[:, s].to(F)[:, None]
            gs, us = (t[torch.arange(n), e] * (a if on_input else 1.0) for t in (gate, up))
            if limit is not None:
                gs, us = gs.clamp(max=limit), us.clamp(-limit, limit)
            y = torch.einsum("tf,twf->tw", gs * plain.sigmoid(1.702 * gs) * (us + 1.0), wd.to(F)[e])
            out += y if on_input else a * y
        return out

    want = reference(limit)
    cores = moe.tensor_cores_take(dtype, width, ff)
    assert cores == (dtype == torch.bfloat16 and width % 8 == 0 and ff % 64 == 0)
    stack = ops.interleave_gate_up if cores else (lambda a, b: torch.cat([a, b], 0))
    w_gu = torch.stack([stack(wg[e], wu[e]) for e in range(experts)]).to(dtype).cuda()
    got = moe.apply_experts(x.to(dtype).cuda(), ids.cuda(), wts.cuda(), w_gu, wd.to(dtype).cuda().contiguous(), None, cores,
                            act=(1.702, limit, 1.0), weight_on_input=True).double().cpu()
    tol = (1e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want.abs().max()))
    assert float((got - want).abs().max()) <= tol
    # the sum over the experts left to the kernel that norms and adds the result
    tile = moe.grouped_tile_rows(n * top, experts) if cores else moe.TILE_ROWS
    choice = moe.Choice(ids.cuda(), wts.cuda(), moe.align(ids.cuda(), experts, tile, want_rows=True), tile)
    rows = moe.apply_choice(x.to(dtype).cuda(), choice, w_gu, wd.to(dtype).cuda().contiguous(), None, cores,
                            act=(1.702, limit, 1.0), weight_on_input=True, defer_sum=True)
    assert isinstance(rows, ops.RowSum) and tuple(rows.shape) == (n, width)
    assert not (cores and n == 3) or rows.y.shape[0] > 1              # few tiles: the second product is cut along K
    assert float((ops.as_tensor(rows).double().cpu() - want).abs().max()) <= tol
    resid, w = torch.randn(n, width, generator=g) * 3, torch.randn(width, generator=g)
    for weights, value in ((None, got.cpu()), (wts, None)):
        if weights is not None:                                       # a sum with weights: the same rows, weighted
            rows = ops.RowSum(rows.y, rows.row_of_pair, wts.cuda(), n, top, dtype)
            value = ops.as_tensor(rows).double().cpu()
        r = resid.cuda()
        cast = ops.add_cast(ops.Pending(rows, w.cuda(), 1e-3), r, dtype)
        total = resid.double() + plain.rms(value, w.double(), 1e-3)
        assert torch.allclose(r.double().cpu(), total, atol=1e-4 if dtype == torch.float32 else 2e-2)
        assert torch.equal(cast, r.to(dtype))
        pick = torch.tensor([n - 1, 0], dtype=torch.int32)
        normed = ops.add_rmsnorm(ops.Pending(rows, w.cuda(), 1e-3), resid.cuda(), w.cuda(), 1e-5, dtype, rows=pick.cuda())
        want_rows = plain.rms(total, w.double(), 1e-5)[pick.long()]
        assert torch.allclose(normed.double().cpu(), want_rows, atol=1e-4 if dtype == torch.float32 else 5e-2, rtol=1e-2)
    for other in (reference(None), reference(limit, on_input=False)):
        assert n < 9 or float((other - want).abs().max()) > 5 * tol


@pytest.mark.parametrize("n,experts,top,splits", [(1, 8, 2, 0), (7, 3, 1, 4), (64, 40, 5, 2), (65, 16, 4, 3), (40, 5, 5, 0)])
def test_routing_and_sorting_in_one_launch(n, experts, top, splits):
    """Scores, choice, weights and the sort of the pairs by expert, the logits as a tensor or as unsummed splits of the
    router's product, for few tokens (one launch) and more (two)."""
    from gllm_b200 import ops
    from gllm_b200.ops import moe

    g = torch.Generator().manual_seed(n + experts)
    parts = torch.randn(max(splits, 1), n, experts, generator=g)
    z = parts.sum(0)
    logits = ops.SplitSum(parts.cuda(), torch.float32) if splits else z.cuda()
    for cores in (False, True):
        choice = moe.choose(logits, None, top, cores)
        order = torch.sort(z.double(), dim=-1, descending=True, stable=True).indices[:, :top]
        assert torch.equal(choice.ids.long().cpu(), order)
        want = plain.sigmoid(z.double()).gather(1, order)
        assert torch.allclose(choice.weights.double().cpu(), want, atol=1e-6)
        sorted_pairs, tile_expert, num_tiles, row_of_pair = (t if t is None else t.cpu() for t in choice.plan)
        ids, tile = choice.ids.reshape(-1).cpu(), choice.tile_rows
        counts = torch.bincount(ids.long(), minlength=experts)
        assert int(num_tiles) == int(((counts + tile - 1) // tile).sum())
        if cores:
            assert len(set(row_of_pair.tolist())) == n * top
            assert all(int(tile_expert[int(row) // tile]) == int(e) for row, e in zip(row_of_pair, ids))
        else:
            for row, p in enumerate(sorted_pairs[: int(num_tiles) * tile].tolist()):
                assert p < 0 or int(ids[p]) == int(tile_expert[row // tile])
            assert sorted(p for p in sorted_pairs.tolist() if p >= 0) == list(range(n * top))


# ------------------------------------------------------------------ each mechanism alone in a model of one layer
ALONE = {
    "attention": one_layer(_att(4, 2, 16, 24, 0.2, 20, 3, 8, scaling=(4.0, 64, 16.0, 1.0))),
    "attention_one_head": one_layer(_att(1, 1, 40, 8, 0.15, 33, 1, 40), width=40, scale=1.0, mult=1.0),
    "attention_without_chunks": one_layer(_att(2, 1, 12, 12, 0.3, None, 2, 0), width=36),
    "attention_chunks_of_one": one_layer(_att(2, 2, 16, 16, 0.3, 1, 4, 16), width=48),
    "wide_heads": one_layer(_att(2, 1, 160, 64, 0.05, 25, 2, 32), width=64),
    "experts": one_layer(_att(2, 1, 8, 8, 0.3, 16, 2, 8), _moe(24, 8, 2, 0.6)),
    "experts_all": one_layer(_att(2, 1, 8, 8, 0.3, 16, 2, 8), _moe(64, 5, 5, 0.8)),
    "experts_one_of_one": one_layer(_att(2, 1, 8, 8, 0.3, 16, 2, 8), _moe(16, 1, 1, 1e9)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", sorted(ALONE))
def test_each_mechanism_alone(kind, dtype, tmp_path):
    cfg = ALONE[kind]
    weights, _, runner = make(cfg, tmp_path, dtype, max_tokens=256, block_size=8)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(3)).tolist()
    want = {"r": plain.forward(cfg, weights, toks)}
    for cuts in ([90], [40, 2, 17] + [1] * 31):
        steps, index = steps_of(toks, cuts)
        compare(run_steps(runner, steps), index, want, *tolerance(dtype))


def test_residual_after_every_layer(tmp_path):
    """The fp32 residual stream after each layer (the result that is still pending normed and added) against the plain
    one."""
    from gllm_b200 import ops

    cfg = PIFELIX["A"]
    weights, _, runner = make(cfg, tmp_path, "float32")
    toks = torch.randint(0, cfg["vocab"], (43,), generator=torch.Generator().manual_seed(8)).tolist()
    layers, seen = [], []
    plain.forward(cfg, weights, toks, layers_out=layers)
    for layer in runner.model.layers:
        def wrapped(branch, resid, ctx, cache, inner=layer.forward):
            out, resid = inner(branch, resid, ctx, cache)
            seen.append(resid.double() + plain.rms(ops.as_tensor(out.value).double(), out.post_weight.double(), out.post_eps))
            return out, resid
        layer.forward = wrapped
    run_steps(runner, steps_of(toks, [43])[0])
    assert len(seen) == len(cfg["layers"])
    for i, got in enumerate(seen):
        assert torch.allclose(got.cpu(), layers[i], atol=2e-4, rtol=2e-4), i


# ------------------------------------------------------------------ whole models: cuts, batches, pages used again
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(PIFELIX))
def test_all_cuts_and_mixed_batches(name, dtype, tmp_path):
    from gllm_b200.engine.replay import build_runner

    cfg = PIFELIX[name]
    weights, folder, runner = make(cfg, tmp_path, dtype, max_tokens=rounded(max(LENGTHS.values())),
                                   block_size=PAGE[name])
    seqs = sequences(cfg["vocab"], seed=5)
    want = {k: plain.forward(cfg, weights, v) for k, v in seqs.items()}
    steps, index = single_request_steps(seqs)
    compare(run_steps(runner, steps), index, want, *tolerance(dtype))
    runner.cache.check_invariants()
    # four live requests at most over 448 tokens of pages: pages and slots are used again
    _, small = build_runner(folder, dtype, 448, block_size=PAGE[name])
    steps, index = mixed_steps(seqs, max_tokens=448, seed=9)
    compare(run_steps(small, steps), index, want, *tolerance(dtype))
    small.cache.check_invariants()
    assert all(g.allocator.total_reused > 0 for g in small.cache.groups)


def test_replay_through_the_command(tmp_path):
    cfg = PIFELIX["A"]
    weights = decisive_routing(cfg, draw_weights(cfg, seed=7, sharp=1.5))
    folder = write_model(cfg, weights, str(tmp_path / "model"))
    seqs = sequences(cfg["vocab"], seed=6)
    want = {k: plain.forward(cfg, weights, v) for k, v in seqs.items()}
    steps, index = mixed_steps(seqs, max_tokens=448, seed=3)
    results = replay(folder, "float32", steps, str(tmp_path / "out"), max_tokens=448, vocab=cfg["vocab"])
    compare(results, index, want, FP32_TOL)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_at_every_edge(dtype, tmp_path):
    """Portions that end one token before, at and after every page border and chunk border (pages of 16; chunks of 40,
    64, 96 and 150), down to two tokens, through layers that own their keys and one that reads them."""
    cfg = PIFELIX["C"]
    weights, _, runner = make(cfg, tmp_path, dtype, max_tokens=256, block_size=16)
    toks = torch.randint(0, cfg["vocab"], (200,), generator=torch.Generator().manual_seed(10)).tolist()
    want = {"r": plain.forward(cfg, weights, toks)}
    for cuts in ([39, 2, 22, 2, 14, 2, 14, 2, 22, 2, 27, 3, 49], [40, 24, 16, 16, 24, 8, 22, 2, 48],
                 [41, 24, 2, 12, 3, 14, 1, 30, 21, 1, 2, 49], [2] * 100):
        steps, index = steps_of(toks, cuts)
        compare(run_steps(runner, steps), index, want, *tolerance(dtype))


def _marking_model(chunk, readers=()):
    """Attention that looks for one token: the queries of ``ASK`` and the keys of ``MARK`` lie along one column that is
    not rotated, the query norm makes their score tower above all others; convolutions of one tap keep a key its token's."""
    dim, col = 16, 12
    m = _att(2, 1, dim, 16, 0.25, chunk, 1, 8)
    cfg = one_layer(m, width=32, vocab=60, scale=1.0, mult=1.0)
    for c in readers:
        cfg["layers"].append({"type": "attention", "mixer": dict(m, kv_from=0, mask={"size": c}), "mlp": None})
    weights = draw_weights(cfg, seed=15)
    MARK, ASK = 7, 11
    weights["embed"][:, :2] = 0                                     # the two columns that carry the marks
    weights["embed"][MARK], weights["embed"][ASK] = 0, 0
    weights["embed"][MARK, 0], weights["embed"][ASK, 1] = 8.0, 8.0
    for i in range(len(cfg["layers"])):
        if i + 1 < len(cfg["layers"]):
            weights[f"l{i}.norm1"][:] = 0                           # only the last layer's attention reaches the logits
        for name, column in ((f"l{i}.mix.k", 0), (f"l{i}.mix.q", 1)):
            if name not in weights:
                continue
            weights[name + ".b"][:] = 0
            weights[name + ".conv"][:] = 1
            weights[name][:, column] = 0
            weights[name][col::dim, column] = 6.0
            weights[name + ".norm"][:] = 1.0
        weights[f"l{i}.mix.q.norm"][:] = 4.0
    return cfg, weights, MARK, ASK


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk,readers", [(64, ()), (100, ()), (230, ()), (24, (200,)), (150, (60,))])
def test_decisive_keys_just_inside_and_just_outside_a_chunk(dtype, chunk, readers, tmp_path):
    """A query that looks for one marked token: at the first position of its chunk (seen up to the chunk's last
    position), right before the chunk (never seen), at page borders; read in a prompt, in portions and decoded alone.
    With ``readers`` the asking layer reads an earlier layer's pages over chunks of its own, larger or smaller than
    those of the layer that stored them."""
    cfg, weights, MARK, ASK = _marking_model(chunk, readers)
    c = readers[-1] if readers else chunk
    n = 2 * c + 40
    g = torch.Generator().manual_seed(16)
    base = [int(t) for t in torch.randint(12, 60, (n,), generator=g)]
    _, _, runner = make(cfg, tmp_path, dtype, max_tokens=512, block_size=16, weights=weights)
    for mark, asks in ((c, (c + 1, 2 * c - 1, 2 * c)), (c - 1, (c - 1 + (c == 1), c, c + 5)), (0, (c - 1, c)),
                       (c // 16 * 16 + 16, (2 * c - 1, 2 * c + 3))):
        toks = list(base)
        toks[mark] = MARK
        for p in asks:
            toks[p] = ASK if p != mark else toks[p]
        want = {"r": plain.forward(cfg, weights, toks)}
        without = list(toks)
        without[mark] = 13
        other = plain.forward(cfg, weights, without)
        scale = float(want["r"].abs().max())
        for p in asks:
            seen = mark <= p and mark // c == p // c
            moved = float((other[p] - want["r"][p]).abs().max()) / scale
            assert p == mark or (moved > 0.1 if seen else moved < 1e-6), (mark, p, moved)
        last = max(asks)
        for cuts in ([n], [last - 3, 2] + [1] * (n - last + 1), [c - 1, 1, 1, c - 2, 1, 1, n - 2 * c - 1], [7, 33] * (n // 40) + [n % 40] * (n % 40 > 0)):
            steps, index = steps_of(toks, cuts)
            compare(run_steps(runner, steps), index, want, *tolerance(dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(dtype, tmp_path):
    """Prompts of one, two and three tokens, then hundreds of tokens decoded one by one (replays of the decode
    graph): state that is lost, doubled or started wrong shows at once or adds up."""
    cfg = PIFELIX["A"]
    weights, _, runner = make(cfg, tmp_path, dtype, max_tokens=512)
    g = torch.Generator().manual_seed(12)
    for first in (1, 2, 3):
        n = first + (330 if first == 2 else 20)
        toks = torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
        want = {"r": plain.forward(cfg, weights, toks)}
        steps, index = steps_of(toks, [first] + [1] * (n - first))
        compare(run_steps(runner, steps), index, want, *tolerance(dtype))
    assert runner.graph_replays > 300


def test_long_decoding_with_tensor_core_sizes(tmp_path):
    cfg = PIFELIX["C"]
    weights, _, runner = make(cfg, tmp_path, "bfloat16", max_tokens=512)
    toks = torch.randint(0, cfg["vocab"], (330,), generator=torch.Generator().manual_seed(14)).tolist()
    want = {"r": plain.forward(cfg, weights, toks)}
    steps, index = steps_of(toks, [30] + [1] * 300)
    compare(run_steps(runner, steps), index, want, *tolerance("bfloat16"))


def test_a_slot_and_its_pages_used_again_start_clean(tmp_path):
    """One state slot and a pool of few pages: the second request gets the first one's slot and pages."""
    cfg = PIFELIX["B"]
    weights, _, runner = make(cfg, tmp_path, "float32", max_tokens=64, max_live=1)
    g = torch.Generator().manual_seed(13)
    a = torch.randint(0, cfg["vocab"], (60,), generator=g).tolist()
    b = torch.randint(0, cfg["vocab"], (50,), generator=g).tolist()
    for rid, toks, cuts in (("a", a, [33, 20, 7]), ("b", b, [3, 40] + [1] * 7), ("c", a, [60])):
        steps, index = steps_of(toks, cuts, rid=rid)
        compare(run_steps(runner, steps), index, {rid: plain.forward(cfg, weights, toks)}, FP32_TOL)
    assert runner.cache.groups[0].allocator.total_reused > 0


def test_a_batch_of_unequal_requests_against_each_alone(tmp_path):
    """bf16: portions of 70, 2 and 33 tokens beside three decoded tokens in one step give what each gives alone."""
    cfg = PIFELIX["C"]
    _, _, runner = make(cfg, tmp_path, "bfloat16", max_tokens=1024, max_live=6)
    g = torch.Generator().manual_seed(17)
    heads = {"a": 50, "b": 7, "c": 39, "d": 63, "e": 95, "f": 20}
    tails = {"a": 70, "b": 2, "c": 33, "d": 1, "e": 1, "f": 1}
    toks = {r: torch.randint(0, cfg["vocab"], (heads[r] + tails[r],), generator=g).tolist() for r in heads}
    entry = lambda r, lo, hi: {"id": r, "tokens": toks[r][lo:hi], "want": list(range(hi - lo))}
    steps = [{"step": i, "entries": [entry(r, 0, heads[r])], "end": []} for i, r in enumerate(heads)]
    steps.append({"step": 6, "entries": [entry(r, heads[r], heads[r] + tails[r]) for r in heads], "end": list(heads)})
    together = run_steps(runner, steps)[6]
    at = 0
    for r in heads:
        alone = run_steps(runner, steps_of(toks[r], [heads[r], tails[r]], rid=r)[0])[1]
        assert np.abs(alone - together[at:at + tails[r]]).max() <= 0.02 * max(1.0, np.abs(alone).max()), r
        at += tails[r]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(name, dtype, tmp_path):
    from gllm_b200 import GenerationRequest, GeneratorParams, LLMEngine

    cfg = PIFELIX[name]
    weights = decisive_routing(cfg, draw_weights(cfg, seed=21))
    folder = write_model(cfg, weights, str(tmp_path / "m"))
    g = torch.Generator().manual_seed(4)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (1, 7, 16, 23, 40)]
    # few pages, small portions: chunked prefill, continuous batching and preemption happen
    params = GeneratorParams(block_size=8, max_batch_size=3, max_seq_len=64, num_blocks=10, model_dtype=dtype,
                             max_num_batched_tokens=24, prefill_chunk=8)
    engine = LLMEngine(folder, params, device="cuda:0")
    reqs = [GenerationRequest(prompt_token_ids=p, max_new_tokens=12, temperature=0.0, ignore_eos=True) for p in prompts]
    results = engine.generate(reqs)
    slack = 1e-5 if dtype == "float32" else 0.05
    for p, r in zip(prompts, results):
        assert len(r.token_ids) == 12 and r.finish_reason == "length"
        tokens = list(p)
        for t in r.token_ids:
            logits = plain.forward(cfg, weights, tokens)[-1]
            best = int(logits.argmax())
            if t != best:
                assert float(logits[best] - logits[t]) <= slack * float(logits.abs().max()), (len(tokens), t, best)
            tokens.append(t)
    engine.cache.check_invariants()
    assert not engine.scheduler.has_work
    if dtype == "float32":
        for req, r in zip(reqs, results):
            assert engine.generate([req])[0].token_ids == r.token_ids


def test_random_weights_mode_writes_a_model_that_runs(tmp_path):
    from gllm_b200.config import load_config
    from gllm_b200.engine.replay import build_runner
    from gllm_b200.weights import write_random_model

    folder = write_random_model(str(tmp_path / "m"), load_config(copy.deepcopy(PIFELIX["C"])), seed=3, std=0.05)
    _, runner = build_runner(folder, "bfloat16", 256)
    toks = list(range(1, 70))
    whole = run_steps(runner, steps_of(toks, [69], rid="a")[0])[0]
    cut = run_steps(runner, steps_of(toks, [30, 38, 1], rid="b")[0])
    assert np.isfinite(whole).all()
    assert np.abs(whole[-1] - cut[2][0]).max() <= 0.05 * max(1.0, np.abs(whole).max())
