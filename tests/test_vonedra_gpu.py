"""Vonedra on the GPU against the plain implementation: each kernel of its mechanisms alone, each mechanism alone in a
model of one layer, whole prompts against token by token decoding and portions of every size, mixed batches over a
pool so small that pages and state slots are used again, keys just inside and just outside of every window and of the
kept first tokens, the first tokens, long decoding through the decode graphs, sizes of every kind, and greedy
generation through the engine."""

import copy

import numpy as np
import pytest
import torch

import plain_vonedra as plain
from replay_helpers import (BF16_TOL_MAX, BF16_TOL_MEAN, FP32_TOL, LENGTHS, compare, mixed_steps, replay, rounded,
                            run_steps, sequences, single_request_steps)
from tiny_vonedra import VONEDRA, _att, _delta, _latent, draw_weights, one_layer, write_model

pytestmark = pytest.mark.gpu

PAGE = {"A": 4, "B": 8, "C": 16, "D": 32}
# seeds of the weights: models whose logits rounding alone does not move by several per cent (a result that is nearly
# zero before its norm does that)
SEED = {"A": 7, "B": 7, "C": 8, "D": 7}
F = plain.F


def tolerance(dtype):
    return (FP32_TOL, None) if dtype == "float32" else (BF16_TOL_MAX, BF16_TOL_MEAN)


def make(cfg, tmp_path, dtype, seed=7, max_tokens=512, block_size=16, max_live=4, sharp=None, weights=None):
    from gllm_b200.engine.replay import build_runner

    sharp = (3.0 if dtype == "float32" else 1.5) if sharp is None else sharp
    if weights is None:
        weights = draw_weights(cfg, seed=seed, sharp=sharp)
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


class Step:
    """The flat batch of requests bringing ``lengths`` tokens from positions ``starts``, as the kernels read it."""

    def __init__(self, lengths, starts, slots):
        from gllm_b200.engine.step import Workspace

        dev = "cuda"
        self.cu_q = torch.tensor([0] + list(np.cumsum(lengths)), dtype=torch.int32, device=dev)
        self.context_lens = torch.tensor(starts, dtype=torch.int32, device=dev)
        self.state_slots = torch.tensor(slots, dtype=torch.int32, device=dev)
        self.positions = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lengths)]).to(torch.int32).to(dev)
        self.token_row = torch.cat([torch.full((n,), s) for s, n in zip(slots, lengths)]).to(torch.int32).to(dev)
        self.num_requests, self.max_q_len = len(lengths), max(lengths)
        self.num_prefill_requests = sum(n > 1 for n in lengths)
        assert all(a >= b or b > 1 for a, b in zip(lengths, lengths[1:]))          # portions before single tokens
        self.max_seq_len = max(s + n for s, n in zip(starts, lengths))
        self.workspace = Workspace(dev)


class Requests:
    """Requests fed through a kernel in portions: the state slots and shuffled pages they own, and what is done."""

    def __init__(self, total, slot_of, page=None, seed=0):
        self.total, self.slot_of, self.page = total, slot_of, page
        self.done = {r: 0 for r in total}
        self.got = {r: [] for r in total}
        if page:
            g = torch.Generator().manual_seed(seed)
            per = {r: -(-n // page) for r, n in total.items()}
            self.n_pages = sum(per.values()) + 3
            order = torch.randperm(self.n_pages, generator=g).tolist()
            self.table = torch.full((max(slot_of.values()) + 2, max(per.values())), -1, dtype=torch.int32)
            for r in total:
                for i in range(per[r]):
                    self.table[slot_of[r], i] = order.pop()

    def step(self, plan):
        return Step([n for _, n in plan], [self.done[r] for r, _ in plan], [self.slot_of[r] for r, _ in plan])

    def rows(self, data, plan):
        return torch.cat([data[r][self.done[r]:self.done[r] + n] for r, n in plan]).cuda()

    def slot_map(self, plan):
        return torch.tensor([int(self.table[self.slot_of[r], t // self.page]) * self.page + t % self.page
                             for r, n in plan for t in range(self.done[r], self.done[r] + n)], dtype=torch.int32).cuda()

    def take(self, out, plan):
        at = 0
        for r, n in plan:
            self.got[r].append(out[at:at + n].double().cpu())
            at += n
            self.done[r] += n

    def results(self):
        assert self.done == self.total
        return {r: torch.cat(v) for r, v in self.got.items()}


# ------------------------------------------------------------------ the kernels of each mechanism alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,taps,streams,source", [(64, 3, 3, "tensor"), (50, 4, 0, "splits"), (7, 1, 1, "tensor"),
                                                      (1024, 2, 5, "splits"), (96, 6, 2, "bias"), (36, 9, 0, "bias"),
                                                      (2048, 4, 7, "bias"), (20, 16, 1, "none")])
def test_result_norm_depth_average_and_convolution(dtype, width, taps, streams, source):
    """A sublayer's result (a tensor, unsummed splits, with a bias, none) normed and added, the average over ``streams``
    earlier streams, the convolution over time, for three requests in portions down to one token, on slots that are
    not the requests' numbers; then the norm of chosen rows."""
    from gllm_b200 import ops
    from gllm_b200.ops import depth

    g = torch.Generator().manual_seed(width + taps)
    eps, n_parts = 1e-5, 3
    req = Requests({0: 47, 1: 21, 2: 5}, {0: 3, 1: 1, 2: 4})
    rnd = lambda n, s=1.0: torch.randn(n, width, generator=g) * s
    resid = {r: rnd(n, 2.0) for r, n in req.total.items()}
    parts = {r: torch.randn(n, n_parts, width, generator=g) for r, n in req.total.items()}
    hist = {r: torch.randn(n, max(streams, 1), width, generator=g) for r, n in req.total.items()}
    post_w, bias = 1 + torch.randn(width, generator=g) * 0.2, torch.randn(width, generator=g)
    conv_w, depth_w = torch.randn(width, taps, generator=g) * 0.5, torch.randn(streams + 1, generator=g)
    value = {r: (p[:, 0] + p[:, 1] + p[:, 2]).to(dtype) for r, p in parts.items()}

    def plain_x(r):
        X = resid[r].to(F)
        if source != "none":
            v = value[r].to(F) + (bias.to(F) if source == "bias" else 0)
            X = X + plain.rms(v, eps) * post_w.to(F)
        if not streams:
            return X, X
        return X, sum(depth_w[k].to(F) * hist[r][:, k].to(F) for k in range(streams)) + depth_w[-1].to(F) * X

    state = torch.full((6, taps - 1, width), 7.0, device="cuda")
    for s in req.slot_of.values():
        state[s] = 0
    for plan in ([(0, 2), (2, 1)], [(1, 9), (0, 30), (2, 2)], [(2, 1), (0, 1), (1, 1)], [(0, 3), (1, 11), (2, 1)], [(0, 11)]):
        st = req.step(plan)
        n = st.positions.numel()
        v = None
        if source == "splits":
            v = ops.SplitSum(req.rows(parts, plan).transpose(0, 1).contiguous(), dtype)
        elif source != "none":
            v = req.rows(value, plan)
        kept = None
        if streams:
            kept = torch.cat([req.rows(hist, plan).transpose(0, 1), torch.zeros(1, n, width, device="cuda")]).contiguous()
        pending = ops.DepthPending(v, bias.cuda() if source == "bias" else None, None if v is None else post_w.cuda(), eps,
                                   kept, streams, depth_w.cuda() if streams else None)
        r_in = req.rows(resid, plan)
        before = r_in.clone()
        h, x = depth.depth_conv(pending, r_in, conv_w.t().contiguous().cuda(), state, st.cu_q, st.state_slots,
                                st.num_requests, st.max_q_len, dtype)
        assert torch.equal(r_in, before)
        norm_w = torch.linspace(0.5, 1.5, width)
        pick = torch.tensor([n - 1, 0], dtype=torch.int32)
        if source == "splits":
            pending.value = ops.SplitSum(req.rows(parts, plan).transpose(0, 1).contiguous(), dtype)
        normed = ops.add_rmsnorm(pending, r_in, norm_w.cuda(), eps, dtype, rows=pick.cuda())
        want = plain.rms(x.double().cpu()[pick.long()], eps) * norm_w.to(F)
        tol = 1e-5 if dtype == torch.float32 else 1.5e-2
        assert torch.allclose(normed.double().cpu(), want, atol=tol * 4, rtol=tol)
        both = torch.cat([h.double(), x.double(), kept[streams].double() if streams else x.double()], 1)
        req.take(both, plan)
    got = req.results()
    for r, rows in got.items():
        X, x = plain_x(r)
        y, _ = plain.causal_conv(x, conv_w.to(F), torch.zeros(taps - 1, width, dtype=F))
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        assert torch.allclose(rows[:, width:2 * width], x, atol=1e-4, rtol=1e-4), r
        assert torch.allclose(rows[:, 2 * width:], X, atol=1e-4, rtol=1e-4), r
        assert torch.allclose(rows[:, :width], x + y, atol=tol * 6, rtol=tol), (r, float((rows[:, :width] - x - y).abs().max()))
        if taps > 1:
            kept = torch.cat([torch.zeros(taps - 1, width, dtype=F), x])[-(taps - 1):]
            assert torch.allclose(state[req.slot_of[r]].double().cpu(), kept, atol=1e-4, rtol=1e-4)
    assert taps == 1 or (float(state[0].min()) == 7.0 and float(state[5].max()) == 7.0)       # others' slots


PLANS = [[(0, 37), (1, 9)], [(0, 2), (1, 1)], [(0, 1), (1, 1)], [(0, 64), (1, 30)], [(0, 46)]]


@pytest.mark.parametrize("cores", ["cuda", "tensor"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,size,keep,far,rows,page", [
    (4, 2, 16, 24, 40, 5, 60, 12, 4), (3, 1, 8, 40, 17, 33, 25, 7, 8), (6, 2, 64, 64, 64, 0, 300, 16, 16),
    (8, 1, 128, 128, 100, 20, 90, 32, 16), (2, 2, 32, 8, None, 0, 40.5, 6, 32), (5, 5, 72, 120, 1, 70, 12, 8, 16),
    (16, 1, 56, 40, 63, 64, 500, 10, 16), (12, 1, 24, 16, 65, 1, 33, 5, 8)])
def test_attention_with_a_bias_by_distance(cores, heads, kv_heads, dim, vdim, size, keep, far, rows, page):
    """Biases, norms, the mix of values, the store into shuffled pages and the attention of two requests fed in portions
    and single tokens, against the plain functions.  One early key stands out for every query (inside the kept tokens
    where there are any), the learned biases spread over several units, one head's sink is far above its scores."""
    from gllm_b200.ops import distance

    dtype = torch.bfloat16 if cores == "tensor" else torch.float32
    g = torch.Generator().manual_seed(heads * 100 + dim)
    eps, scale, lam = 1e-5, 4.0 / dim, 0.4
    req = Requests({0: 150, 1: 41}, {0: 2, 1: 0}, page, seed=1)
    qc, kc, vc = heads * dim, kv_heads * dim, kv_heads * vdim
    proj = {r: (torch.randn(n, qc + kc + vc, generator=g)).to(dtype) for r, n in req.total.items()}
    first = {r: torch.randn(n, vc, generator=g).to(dtype) for r, n in req.total.items()}
    bias = torch.randn(qc + kc + vc, generator=g) * 0.3
    star = min(max(0, keep - 1), 40)                       # every query leans towards this key
    for r in proj:
        proj[r][star, qc:qc + kc] = 3.0
        proj[r][:, :qc] += 1.0
    rel, sink = torch.randn(rows, heads, generator=g) * 2, torch.randn(heads, generator=g)
    sink[heads - 1] = 9.0
    stored = (lambda t: t.to(dtype).to(F))                 # what the kernel reads back has the activation type

    def plain_rows(r, size=size, keep=keep, mixed=True):
        x = proj[r].to(F) + bias.to(F)
        T = x.shape[0]
        q = stored(plain.rms(x[:, :qc].view(T, heads, dim), eps))
        k = stored(plain.rms(x[:, qc:qc + kc].view(T, kv_heads, dim), eps))
        v = x[:, qc + kc:].view(T, kv_heads, vdim)
        v = stored((1 - lam) * v + lam * first[r].to(F).view(v.shape)) if mixed else stored(v)
        b = torch.tensor([plain.distance_bucket(n, rows, far) for n in range(T)])
        p = torch.arange(T)
        return plain.attend(q, k, v, p, p, scale, size, keep, bias=lambda d, h: rel.to(F)[b[d.clamp(min=0)], h],
                            sink=sink.to(F))

    table = distance.DistanceBias.build(rel.cuda(), far, sink.cuda())
    cache = torch.zeros(req.n_pages, page * kv_heads * (dim + vdim), device="cuda", dtype=dtype)
    for plan in PLANS:
        st = req.step(plan)
        q = distance.distance_prep(req.rows(proj, plan).contiguous(), bias.cuda(), eps, req.slot_map(plan), cache, heads,
                                   kv_heads, dim, vdim, page, mix=distance.MIXED, first=req.rows(first, plan), lam=lam)
        out = distance.distance_attention(q, cache, req.table.cuda(), st.positions, st.token_row, table, heads, kv_heads,
                                          dim, vdim, page, scale, window=size, keep_first=keep, batch=st)
        req.take(out, plan)
    got = req.results()
    for r in got:
        want = plain_rows(r)
        err = (got[r] - want).abs()
        worst, mean = (3e-5, 3e-6) if dtype == torch.float32 else (3e-2, 4e-3)
        assert float(err.max()) < worst * max(1.0, float(want.abs().max())), (r, float(err.max()))
        assert float(err.mean()) < mean, (r, float(err.mean()))
    # the comparison is sharp: another window, other kept tokens or unmixed values come out differently
    want = plain_rows(0)
    if size is not None:
        assert float((plain_rows(0, size=size + 1) - want).abs().max()) > 0.05
        assert float((plain_rows(0, keep=keep + 1) - want).abs().max()) > 0.05
        if keep:
            assert float((plain_rows(0, keep=keep - 1) - want).abs().max()) > 0.05
    assert float((plain_rows(0, mixed=False) - want).abs().max()) > 0.05


def test_single_tokens_over_ranges_of_keys():
    """Single tokens over contexts long enough that a request's keys are cut into ranges, with and without a window, for
    requests of unequal lengths (some ranges of the short one are empty)."""
    from gllm_b200.ops import distance

    heads, kv_heads, dim, vdim, page = 4, 2, 64, 64, 16
    g = torch.Generator().manual_seed(5)
    bias_rows, far, scale = 16, 200, 0.1
    rel, sink = torch.randn(bias_rows, heads, generator=g), torch.randn(heads, generator=g)
    table = distance.DistanceBias.build(rel.cuda(), far, sink.cuda())
    proj = {r: torch.randn(n, (heads + kv_heads) * dim + kv_heads * vdim, generator=g).to(torch.bfloat16)
            for r, n in ((0, 1205), (1, 70), (2, 400))}
    qc, kc = heads * dim, kv_heads * dim
    for size, keep in ((None, 0), (300, 10), (450, 100)):
        req = Requests({0: 1205, 1: 70, 2: 400}, {0: 1, 1: 2, 2: 0}, page, seed=size or 0)
        cache = torch.zeros(req.n_pages, page * kv_heads * (dim + vdim), device="cuda", dtype=torch.bfloat16)
        split = 0
        for plan in ([(0, 1200), (1, 65), (2, 395)], *[[(0, 1), (1, 1), (2, 1)]] * 5):
            st = req.step(plan)
            q = distance.distance_prep(req.rows(proj, plan).contiguous(), None, 1e-5, req.slot_map(plan), cache, heads,
                                       kv_heads, dim, vdim, page)
            if st.max_q_len == 1:
                most = distance._visited(st.max_seq_len, distance.SINGLE_KEY_TILE, 1, size or 0, keep)
                split += distance._ranges(most, kv_heads * 3, distance.SINGLE_SPLIT_TILES, 2, q.device)[0] > 1
            req.take(distance.distance_attention(q, cache, req.table.cuda(), st.positions, st.token_row, table, heads,
                                                 kv_heads, dim, vdim, page, scale, window=size, keep_first=keep,
                                                 batch=st), plan)
        assert split == 5
        for r, rows in req.results().items():
            x, T = proj[r].to(F), proj[r].shape[0]
            bf = lambda t: t.to(torch.bfloat16).to(F)
            q, k = bf(plain.rms(x[:, :qc].view(T, heads, dim), 1e-5)), bf(plain.rms(x[:, qc:qc + kc].view(T, kv_heads, dim), 1e-5))
            b = torch.tensor([plain.distance_bucket(n, bias_rows, far) for n in range(T)])
            tail = torch.arange(T - 5, T)
            want = plain.attend(q[-5:], k, x[:, qc + kc:].view(T, kv_heads, vdim), tail, torch.arange(T), scale, size, keep,
                                bias=lambda d, h: rel.to(F)[b[d.clamp(min=0)], h], sink=sink.to(F))
            err = (rows[-5:] - want).abs()
            assert float(err.max()) < 6e-3, (size, r, float(err.max()))


def test_values_of_the_first_layer_are_kept():
    """The prep kernel's first-layer mode leaves the values it stores; queries come from unsummed splits as well."""
    from gllm_b200 import ops
    from gllm_b200.ops import distance

    g = torch.Generator().manual_seed(9)
    parts = torch.randn(4, 11, 2 * 16 + 2 * 16 + 2 * 24, generator=g)
    bias = torch.randn(parts.shape[2], generator=g)
    whole = (parts[0] + parts[1] + parts[2] + parts[3]).to(torch.bfloat16)
    results = []
    for proj in (ops.SplitSum(parts.cuda(), torch.bfloat16), whole.cuda()):
        cache = torch.zeros(3, 8 * 2 * 40, device="cuda", dtype=torch.bfloat16)
        first = torch.empty(11, 48, device="cuda", dtype=torch.bfloat16)
        slots = torch.arange(8, 19, dtype=torch.int32, device="cuda")
        q = distance.distance_prep(proj, bias.cuda(), 1e-5, slots, cache, 2, 2, 16, 24, 8, mix=distance.FIRST, first=first)
        results.append((q, cache, first))
        v = cache[:, 8 * 2 * 16:].view(3, 2, 8, 24).permute(0, 2, 1, 3).reshape(24, 48)[8:19]
        assert torch.equal(first, v)
        want = whole.double()[:, 64:] + bias.double()[64:]
        assert torch.allclose(first.double().cpu(), want, atol=0.03, rtol=5e-3)
    for a, b in zip(*results):                                   # (one sums a head's squares in another order)
        assert torch.allclose(a.float(), b.float(), atol=1e-3, rtol=1e-2)


@pytest.mark.parametrize("cores", ["cuda", "tensor"])
@pytest.mark.parametrize("heads,dim,rot,rank,size,page", [(4, 16, 8, 40, 33, 4), (3, 8, 16, 88, 64, 16), (16, 32, 32, 128, 31, 8),
                                                         (8, 64, 64, 512, 100, 16), (1, 24, 24, 72, 1, 16), (20, 8, 8, 200, 65, 8),
                                                         (2, 16, 16, 64, None, 16)])
def test_latent_attention_in_a_window(cores, heads, dim, rot, rank, size, page):
    """The norms of both latents, the rotation of the queries made from theirs, the store into shuffled pages and the
    attention of two requests over the keys a window holds (widths that fill a tensor-core tile and ones that do not),
    in portions and single tokens; what lies before every later token's window is overwritten on the way."""
    from gllm_b200.ops import latent

    dtype = torch.bfloat16 if cores == "tensor" else torch.float32
    assert latent.tensor_core_kernel_takes(dtype, rank, rot) == (cores == "tensor")
    g = torch.Generator().manual_seed(rank + heads)
    q_rank, eps, scale, base = 24, 1e-5, 1.5 / rank ** 0.5, 300.0
    req = Requests({0: 150, 1: 41}, {0: 2, 1: 0}, page, seed=2)
    down = q_rank + rank + rot
    rows = {r: torch.randn(n, down, generator=g).to(dtype) for r, n in req.total.items()}
    w_uq = (torch.randn(heads * (dim + rot), q_rank, generator=g) / q_rank ** 0.5).to(dtype)
    qa = {r: torch.randn(n, heads * rank, generator=g).to(dtype) for r, n in req.total.items()}
    qn, cn = 1 + torch.randn(q_rank, generator=g) * 0.2, 1 + torch.randn(rank, generator=g) * 0.2
    inv_freq = torch.tensor([base ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
    stored = lambda t: t.to(dtype).to(F)

    def plain_rows(r, size=size):
        x, T = rows[r].to(F), rows[r].shape[0]
        p = torch.arange(T)
        cq = stored(plain.rms(x[:, :q_rank], eps) * qn.to(F))
        q = stored(cq @ w_uq.to(F).T).view(T, heads, dim + rot)
        qr = stored(plain.rotate_pairs(q[..., dim:], p, base, rot))
        c = stored(plain.rms(x[:, q_rank:q_rank + rank], eps) * cn.to(F))
        kr = stored(plain.rotate_pairs(x[:, None, q_rank + rank:], p, base, rot)[:, 0])
        keys = torch.cat([c, kr], 1)[:, None]
        qq = torch.cat([qa[r].to(F).view(T, heads, rank), qr], -1)
        return cq, plain.attend(qq, keys, c[:, None], p, p, scale, size)

    cache = torch.zeros(req.n_pages, page * (rank + rot), device="cuda", dtype=dtype)
    for plan in PLANS:
        st = req.step(plan)
        x = req.rows(rows, plan).contiguous()
        cq = latent.latent_prep(x, cn.cuda(), eps, st.positions, inv_freq.cuda(), req.slot_map(plan), cache, 0, dim, rot, rank,
                                q_rank, page, q_latent_norm=qn.cuda())
        q = (cq.float() @ w_uq.cuda().float().T).to(dtype).contiguous()
        q = latent.latent_rotate_q(q, st.positions, inv_freq.cuda(), heads, dim, rot)
        out = latent.attention_latent(req.rows(qa, plan).contiguous(), q, dim + rot, dim, None, cache, req.table.cuda(),
                                      st.positions, st.token_row, heads, rank, rot, page, scale, window=size, batch=st)
        req.take(torch.cat([cq, out], 1), plan)
        if size is not None:                              # a later token sees nothing at or before done - size
            for r in req.total:
                for t in range(max(0, req.done[r] - size + 1)):
                    slot = int(req.table[req.slot_of[r], t // page])
                    cache[slot].view(page, rank + rot)[t % page] = 300.0
    worst, mean = (5e-5, 1e-5) if dtype == torch.float32 else (6e-2, 6e-3)
    for r, got in req.results().items():
        cq, want = plain_rows(r)
        assert torch.allclose(got[:, :q_rank], cq, atol=1e-4 if dtype == torch.float32 else 3e-2)
        err = (got[:, q_rank:] - want).abs()
        assert float(err.max()) < worst * max(1.0, float(want.abs().max())) and float(err.mean()) < mean, (
            r, float(err.max()), float(err.mean()))
    if size is not None:
        assert float((plain_rows(0, size=size + 1)[1] - plain_rows(0)[1]).abs().max()) > 0.05


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(4, 2, 16, 24, 4), (3, 1, 10, 6, 1), (2, 2, 32, 32, 2), (1, 1, 7, 9, 3),
                                                         (4, 4, 64, 64, 4), (2, 1, 128, 40, 3), (2, 2, 256, 16, 2), (6, 3, 4, 8, 4),
                                                         (2, 1, 300, 12, 2), (1, 1, 1, 5, 2), (64, 8, 64, 128, 2)])
def test_delta_rule_with_one_decay_per_head(heads, kv_heads, dim, vdim, taps):
    """Convolutions, unit norms, one decay per head, the recurrence and the norm with its SiLU gate for two requests in
    steps of portions and single tokens, on slots that are not the requests' numbers."""
    from gllm_b200.ops import stateful

    big = heads * dim * vdim > 100000
    g = torch.Generator().manual_seed(heads * 10 + dim)
    req = Requests({0: 12 if big else 45, 1: 5 if big else 20}, {0: 3, 1: 1})
    qk, hv = kv_heads * dim, heads * vdim
    x = {r: torch.randn(n, 2 * qk + hv, generator=g) for r, n in req.total.items()}
    ba = {r: torch.randn(n, 2 * heads, generator=g) for r, n in req.total.items()}
    gate = {r: torch.randn(n, hv, generator=g) for r, n in req.total.items()}
    conv_w = torch.randn(2 * qk + hv, taps, generator=g) * 0.6
    dt_bias, A_log = torch.randn(heads, generator=g), torch.randn(heads, generator=g) * 0.5
    norm_w, eps = 1 + torch.randn(vdim, generator=g) * 0.2, 1e-5

    def plain_request(r):
        T = req.total[r]
        y, _ = plain.causal_conv(x[r].to(F), conv_w.to(F), torch.zeros(taps - 1, 2 * qk + hv, dtype=F))
        y = plain.silu(y)
        q = plain.unit(y[:, :qk].view(T, kv_heads, dim)) * dim ** -0.5
        k = plain.unit(y[:, qk:2 * qk].view(T, kv_heads, dim))
        rep = heads // kv_heads
        beta = torch.sigmoid(ba[r].to(F)[:, :heads])
        decay = torch.exp(-torch.exp(A_log.to(F)) * plain.softplus(ba[r].to(F)[:, heads:] + dt_bias.to(F)))
        o = plain.delta_rule(q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1), y[:, 2 * qk:].view(T, heads, vdim), decay,
                             beta, torch.zeros(heads, dim, vdim, dtype=F))
        o = plain.rms(o, eps) * norm_w.to(F) * plain.silu(gate[r].to(F)).view(T, heads, vdim)
        return o.reshape(T, hv)

    state = torch.full((5, heads, vdim, dim), 7.0, device="cuda")
    conv_state = torch.full((5, taps - 1, 2 * qk + hv), 7.0, device="cuda")
    for s in req.slot_of.values():
        state[s] = 0
        conv_state[s] = 0
    plans = [[(0, 7), (1, 2)], [(0, 2), (1, 1)], [(0, 1), (1, 1)], [(0, 2), (1, 1)]] if big else \
        [[(0, 23), (1, 8)], [(0, 2), (1, 1)], [(0, 1), (1, 1)], [(0, 19), (1, 10)]]
    for plan in plans:
        st = req.step(plan)
        raw = req.rows(ba, plan)
        ops_ = stateful.delta_prep(req.rows(x, plan).contiguous(), conv_w.cuda(), conv_state, st.positions, st.token_row,
                                   st.cu_q, st.state_slots, st.num_requests, raw[:, heads:], dt_bias.cuda(), A_log.cuda(),
                                   raw[:, :heads], heads, kv_heads, dim, vdim, 1e-6, dim ** -0.5, max_q_len=st.max_q_len)
        assert ops_[2].shape[1] == heads
        o = stateful.delta_rule(*ops_, state, st.cu_q, st.state_slots, st.num_requests, heads, kv_heads, dim, vdim,
                                max_q_len=st.max_q_len)
        req.take(stateful.head_norm(o, heads, vdim, norm_w.cuda(), eps, torch.float32, gate=req.rows(gate, plan).contiguous(),
                                    gate_kind="silu"), plan)
    for r, got in req.results().items():
        want = plain_request(r)
        # a head's read-out near zero is divided by its size: compare where the norm does not blow rounding up
        assert torch.allclose(got, want, atol=2e-3, rtol=2e-3), (r, float((got - want).abs().max()))
        assert float((got - want).abs().mean()) < 2e-5
    assert float(state[0].min()) == 7.0 and float(state[4].max()) == 7.0


# ------------------------------------------------------------------ each mechanism alone in a model of one layer
ALONE = {
    "attention": one_layer(_att(4, 2, 16, 24, 0.4, 40, size=20, keep=5)),
    "attention_one_head": one_layer(_att(1, 1, 40, 8, 0.2, 25, size=30, keep=0, v_mix=False), width=40, taps=1),
    "attention_no_window": one_layer(_att(6, 2, 24, 24, 0.3, 60), taps=2),
    "latent": one_layer(_latent(4, 16, 8, 24, 40, 32, 0.3, size=25)),
    "latent_no_window": one_layer(_latent(3, 12, 10, 20, 30, 50, 0.3, dims=6), width=50),
    "delta": one_layer(_delta(4, 2, 16, 24, 4)),
    "delta_odd_sizes": one_layer(_delta(3, 3, 9, 5, 2), width=56),
    "dense": one_layer(_delta(2, 2, 8, 8, 1), 72),
    "long_convolution": one_layer(_delta(2, 2, 8, 8, 2), 40, taps=11),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", sorted(ALONE))
def test_each_mechanism_alone(kind, dtype, tmp_path):
    cfg = ALONE[kind]
    weights, _, runner = make(cfg, tmp_path, dtype, max_tokens=256, block_size=8)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(3)).tolist()
    want = {"r": plain.forward(cfg, weights, toks)}
    for rid, cuts in (("r", [90]), ("r", [40, 2, 17] + [1] * 31)):
        steps, index = steps_of(toks, cuts, rid=rid)
        compare(run_steps(runner, steps), index, want, *tolerance(dtype))


@pytest.mark.parametrize("name", ["A", "C"])
def test_residual_after_every_layer(name, tmp_path):
    """The residual after each layer's average (what is still pending computed here) against the plain one."""
    from gllm_b200 import ops

    cfg = VONEDRA[name]
    weights, _, runner = make(cfg, tmp_path, "float32")
    toks = torch.randint(0, cfg["vocab"], (23,), generator=torch.Generator().manual_seed(8)).tolist()
    layers = []
    plain.forward(cfg, weights, toks, layers_out=layers)
    seen = []
    for layer in runner.model.layers:
        def wrapped(branch, resid, ctx, cache, inner=layer.forward):
            b, x = inner(branch, resid, ctx, cache)
            v = ops.as_tensor(b.value).double() + (0 if b.value_bias is None else b.value_bias.double())
            X = x.double() + plain.rms(v, b.post_eps) * b.post_weight
            w = b.depth_weight.double()
            seen.append(sum(w[k] * b.streams[k] for k in range(b.count)) + w[b.count] * X)
            return b, x
        layer.forward = wrapped
    run_steps(runner, steps_of(toks, [23])[0])
    assert len(seen) == len(cfg["layers"])
    for i, got in enumerate(seen):
        scale = float(layers[i].abs().max())
        assert float((got.cpu() - layers[i]).abs().max()) < 5e-5 * scale, i


# ------------------------------------------------------------------ whole models: cuts, batches, pages used again
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(VONEDRA))
def test_all_cuts_and_mixed_batches(name, dtype, tmp_path):
    from gllm_b200.engine.replay import build_runner

    cfg = VONEDRA[name]
    weights, folder, runner = make(cfg, tmp_path, dtype, max_tokens=rounded(max(LENGTHS.values())),
                                   block_size=PAGE[name], seed=SEED[name])
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
    cfg = VONEDRA["A"]
    weights = draw_weights(cfg, seed=7, sharp=3.0)
    folder = write_model(cfg, weights, str(tmp_path / "model"))
    seqs = sequences(cfg["vocab"], seed=6)
    want = {k: plain.forward(cfg, weights, v) for k, v in seqs.items()}
    steps, index = mixed_steps(seqs, max_tokens=448, seed=3)
    results = replay(folder, "float32", steps, str(tmp_path / "out"), max_tokens=448, vocab=cfg["vocab"])
    compare(results, index, want, FP32_TOL)


def marked_model(kind, size, keep=0):
    """One layer whose queries look for one token: the keys of token MARK and the queries of token ASK lie along one
    direction (score 12 or more above the others), so that an ASK gives nearly all of its weight to a MARK it sees."""
    MARK, ASK = 7, 11
    if kind == "attention":
        cfg = one_layer(_att(2, 1, 16, 16, 1.0, 60, size=size, keep=keep), width=32, vocab=60)
    else:
        cfg = one_layer(_latent(2, 16, 4, 16, 16, 24, 0.3, size=size), width=32, vocab=60)
    w = draw_weights(cfg, seed=15)
    w["embed"][:, :2] = 0                                        # two columns carry the marks
    w["embed"][MARK], w["embed"][ASK] = 0, 0
    w["embed"][MARK, 0], w["embed"][ASK, 1] = 4.0, 4.0
    w["l0.canon1"][:2] = 0                                       # and are not smeared over time
    w["l0.canon1"] *= 0.2
    if kind == "attention":
        w["l0.mix.rel"] *= 0.3
        w["l0.mix.sink"] *= 0
        w["l0.mix.q.b"] *= 0
        w["l0.mix.k.b"] *= 0
        for name, column in (("q", 1), ("k", 0)):
            t = w[f"l0.mix.{name}"]
            t[:, column] = 0
            t[5::16, column] = 8.0                               # column 5 of every head
    else:
        for name, column in (("dq", 1), ("dkv", 0)):
            t = w[f"l0.mix.{name}"]
            t[:, column] = 0
            t[3, column] = 8.0                                   # the latent's third number
            w[f"l0.mix.{name}.norm"][3] = 1.0
        w["l0.mix.dkv"][24:, 0] = 0                              # nothing in the rotated part
        for name, per_head in (("uq", 20), ("uk", 16)):
            t = w[f"l0.mix.{name}"]
            t[:, 3] = 0
            t[5::per_head, 3] = 2.0
    return cfg, {k: v.to(torch.bfloat16).to(torch.float32) for k, v in w.items()}, MARK, ASK


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,size,keep", [("attention", 48, 6), ("attention", 64, 0), ("attention", 33, 17),
                                            ("latent", 48, 0), ("latent", 64, 0)])
def test_keys_just_inside_and_just_outside(kind, size, keep, dtype, tmp_path):
    """A decisive key at the last position a window holds, at the first it does not, at the last kept position, at the
    first that is not kept, far behind the window, and at page borders; read in a prompt, in portions and decoded alone.
    Were the window or the kept tokens off by one, some asked position would move by far more than the tolerance."""
    cfg, weights, MARK, ASK = marked_model(kind, size, keep)
    cases = []                                                   # (where the marks lie, where the asks lie)
    base = 80
    for mark in (base, base + 15, base + 16):
        cases.append(([mark], [mark + size - 1, mark + size, mark + size + 5]))
    if keep:
        cases.append(([keep - 1], [size + keep + 40, 230]))
        cases.append(([keep], [size + keep - 1, size + keep, 230]))
    cases.append(([0], [size - 1, size, 200]))
    _, _, runner = make(cfg, tmp_path, dtype, max_tokens=256, block_size=16, weights=weights)
    g = torch.Generator().manual_seed(16)
    sharp = {"size": 0.0, "keep": 0.0}
    for marks, asks in cases:
        toks = [int(t) for t in torch.randint(12, 60, (240,), generator=g)]
        for p in marks:
            toks[p] = MARK
        for p in asks:
            toks[p] = ASK
        want = {"r": plain.forward(cfg, weights, toks)}
        for what in ("size", "keep"):
            other = copy.deepcopy(cfg)
            mask = other["layers"][0]["mixer"]["mask"]
            if what == "size":
                mask["size"] += 1
            elif kind == "attention":
                mask["keep_first"] = keep + 1
            moved = (plain.forward(other, weights, toks) - want["r"])[asks].abs().max()
            sharp[what] = max(sharp[what], float(moved) / float(want["r"].abs().max()))
        first = asks[0]
        for cuts in ([240], [first, 1, 1] + [238 - first], [50] * 4 + [2, 2] + [1] * 36):
            steps, index = steps_of(toks, cuts)
            compare(run_steps(runner, steps), index, want, *tolerance(dtype))
    assert sharp["size"] > 0.15 and (not keep or sharp["keep"] > 0.15), sharp


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_at_every_edge(dtype, tmp_path):
    """Portions that end one token before, at and after every page border, window edge and the end of the kept tokens,
    down to two tokens."""
    cfg = VONEDRA["C"]
    weights, _, runner = make(cfg, tmp_path, dtype, max_tokens=256, block_size=16, seed=SEED["C"])
    toks = torch.randint(0, cfg["vocab"], (130,), generator=torch.Generator().manual_seed(10)).tolist()
    want = {"r": plain.forward(cfg, weights, toks)}
    for cuts in ([15, 2, 15, 1, 31, 2, 34, 30], [16, 16, 1, 31, 33, 33], [36, 2, 12, 2, 17, 2, 59], [49, 2, 2, 45, 2, 2, 28],
                 [2] * 65, [7, 9, 8, 8, 1, 97]):
        steps, index = steps_of(toks, cuts)
        compare(run_steps(runner, steps), index, want, *tolerance(dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(dtype, tmp_path):
    """Prompts of one, two and three tokens, then hundreds of tokens decoded one by one (replays of the decode graph):
    state that is lost, doubled or started wrong shows at once or adds up; every window passes over decoded tokens."""
    cfg = VONEDRA["A"]
    weights, _, runner = make(cfg, tmp_path, dtype, max_tokens=512)
    g = torch.Generator().manual_seed(12)
    for first in (1, 2, 3):
        n = first + (330 if first == 2 else 20)
        toks = torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
        want = {"r": plain.forward(cfg, weights, toks)}
        steps, index = steps_of(toks, [first] + [1] * (n - first))
        compare(run_steps(runner, steps), index, want, *tolerance(dtype))
    assert runner.graph_replays > 300


def test_a_slot_and_its_pages_used_again_start_clean(tmp_path):
    """One state slot and a pool of four pages: the second request gets the first one's slot and pages."""
    cfg = VONEDRA["D"]
    weights, _, runner = make(cfg, tmp_path, "float32", max_tokens=64, max_live=1)
    g = torch.Generator().manual_seed(13)
    a = torch.randint(0, cfg["vocab"], (60,), generator=g).tolist()
    b = torch.randint(0, cfg["vocab"], (50,), generator=g).tolist()
    for rid, toks, cuts in (("a", a, [33, 20, 7]), ("b", b, [3, 40] + [1] * 7), ("c", a, [60]), ("d", b, [1] * 50)):
        steps, index = steps_of(toks, cuts, rid=rid)
        compare(run_steps(runner, steps), index, {rid: plain.forward(cfg, weights, toks)}, FP32_TOL)
    assert runner.cache.groups[0].allocator.total_reused > 0


def test_a_batch_equals_each_request_alone(tmp_path):
    """Unequal requests in one step against each alone: equal up to the order of fp32 sums."""
    cfg = VONEDRA["A"]
    _, _, runner = make(cfg, tmp_path, "float32", max_tokens=512, block_size=8)
    g = torch.Generator().manual_seed(14)
    toks = {k: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for k, n in (("a", 1), ("b", 77), ("c", 2), ("d", 130))}
    together = run_steps(runner, [{"step": 0, "entries": [{"id": k, "tokens": t, "want": [len(t) - 1]} for k, t in toks.items()],
                                   "end": list(toks)}])[0]
    for i, (k, t) in enumerate(toks.items()):
        alone = run_steps(runner, [{"step": 0, "entries": [{"id": k, "tokens": t, "want": [len(t) - 1]}], "end": [k]}])[0][0]
        assert np.abs(alone - together[i]).max() < 2e-5 * np.abs(alone).max(), k


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(name, dtype, tmp_path):
    from gllm_b200 import GenerationRequest, GeneratorParams, LLMEngine

    cfg = VONEDRA[name]
    weights = draw_weights(cfg, seed=21)
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
        tokens = list(p) + list(r.token_ids)
        logits = plain.forward(cfg, weights, tokens)
        for i, t in enumerate(r.token_ids):
            row = logits[len(p) + i - 1]
            best = int(row.argmax())
            assert t == best or float(row[best] - row[t]) <= slack * float(row.abs().max()), (len(p), i, t, best)
    engine.cache.check_invariants()
    assert not engine.scheduler.has_work
    if dtype == "float32":
        for req, r in zip(reqs, results):
            assert engine.generate([req])[0].token_ids == r.token_ids


def test_captured_portions_over_longer_contexts(tmp_path):
    """A prompt portion captured as a graph early in a prompt is replayed further on, beyond every window."""
    from gllm_b200.cache.manager import CacheManager
    from gllm_b200.engine.step import StepEntry, StepRunner
    from gllm_b200.models.loading import load_model

    cfg = VONEDRA["A"]
    weights = draw_weights(cfg, seed=31, sharp=3.0)
    _, model = load_model(write_model(cfg, weights, str(tmp_path / "m")), "float32", "cuda:0")
    cache = CacheManager(model.cache_requirements(), block_size=16, num_blocks=20, max_batch_size=2, max_seq_len=320,
                         dtype=torch.float32, device="cuda:0")
    runner = StepRunner(model, cache, max_tokens_per_step=320, prefill_graph_tokens=(64,))
    toks = torch.randint(0, cfg["vocab"], (300,), generator=torch.Generator().manual_seed(6)).tolist()
    want = plain.forward(cfg, weights, toks)
    p = 0
    for n in (64, 64, 30, 64, 50, 28):
        got = runner.run([StepEntry("r", toks[p:p + n], [n - 1])]).cpu().double()
        p += n
        assert float((got[0] - want[p - 1]).abs().max()) < FP32_TOL * float(want.abs().max()), p
    assert runner.graph_replays >= 2


def test_random_weights_mode_writes_a_model_that_runs(tmp_path):
    from gllm_b200.config import load_config
    from gllm_b200.engine.replay import build_runner
    from gllm_b200.weights import write_random_model

    folder = write_random_model(str(tmp_path / "m"), load_config(copy.deepcopy(VONEDRA["A"])), seed=3, std=0.05)
    _, runner = build_runner(folder, "bfloat16", 256)
    toks = list(range(1, 70))
    whole = run_steps(runner, steps_of(toks, [69], rid="a")[0])[0]
    cut = run_steps(runner, steps_of(toks, [30, 38, 1], rid="b")[0])
    assert np.isfinite(whole).all()
    assert np.abs(whole[-1] - cut[2][0]).max() <= 0.05 * max(1.0, np.abs(whole).max())
