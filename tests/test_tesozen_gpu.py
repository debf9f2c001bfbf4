"""Tesozen on the device against the plain implementation: the kernels of every mechanism alone (the square of relu in a
product's epilogue, layer norms with a bias alone and riding on a sublayer's closing kernel, heads of two maps into the cache,
differential attention in chunks, its fold, gated per-head products, the choice among the best groups, the matrix memory),
one-layer models, and whole models cut in four ways (whole prompts; a prompt and then token by token; portions down to one and
two tokens; up to three live requests, portions of some beside single tokens of others, on so few pages and slots that they are
used again), in float32 and bfloat16; weights made so that a chunk's edge, a far key, a lost state, a second map shows; greedy
generation through the entry point and the scheduler; the command line; the trace runner."""

from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import helpers as H
import tesozen_models as M
from plain import tesozen_plain as plain

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
F32, BF16 = torch.float32, torch.bfloat16


def make_runner(folder, dtype, page, steps=None, max_live=3, num_pages=None, **kw):
    from lockstep_b200.engine import ModelRunner

    if num_pages is None:
        num_pages = H.max_live_tokens(steps, round_to=page) // page
    return ModelRunner(folder, dtype=dtype, num_pages=num_pages, page_size=page, max_live=max_live,
                       max_seq_len=1024, **kw)


PLANS = {
    "whole": H.plan_whole,
    "then_single": lambda r: H.plan_bulk_then_single(r, tail=70),
    "portions": lambda r: H.plan_portions(r, sizes=(7, 2, 17, 3, 33, 2, 5, 64, 1, 2, 150)),
    "mixed": lambda r: H.plan_mixed(r, max_live=3),
}


def _tol(dtype):
    return 2e-5 if dtype == F32 else 2e-2


def d64(t):
    return t.double().cpu()


# ---------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("tokens", [1, 9, 30, 50, 100, 300])
@pytest.mark.parametrize("n, k", [(56, 72), (512, 256), (1280, 1024), (30, 52)])
def test_squared_relu_in_the_products_epilogue(dtype, tokens, n, k):
    from lockstep_b200 import kernels as K

    torch.manual_seed(tokens + n)
    x = (torch.randn(tokens, k, device=DEV) * 2).to(dtype)
    w = (torch.randn(n, k, device=DEV) * k ** -0.5).to(dtype)
    out = torch.empty(tokens, n, dtype=dtype, device=DEV)
    err = K.new_error_word(DEV)
    K.gemm_nt(x, w, out, K.EPILOGUE_RELU2, err=err)
    want = plain.relu_squared(d64(x) @ d64(w).T)
    assert float((d64(out) - want).abs().max()) <= _tol(dtype) * (1 + float(want.abs().max()))
    assert 0.3 < float((out == 0).float().mean()) < 0.7
    # the norm made inside the product gives the bits of the norm in front of it
    if dtype == BF16 and k % 8 == 0:
        h = torch.randn(tokens, k, device=DEV)
        gain = torch.rand(k, device=DEV) + 0.5
        a, b = torch.empty_like(out), torch.empty_like(out)
        normed = torch.empty(tokens, k, dtype=BF16, device=DEV)
        K.rmsnorm(h, gain, normed, 1e-5, err)
        K.gemm_nt(normed, w, a, K.EPILOGUE_RELU2, err=err)
        if K.gemm_nt_tc_rmsnorm(h, gain, 1e-5, w, b, K.EPILOGUE_RELU2, err):
            assert torch.equal(a, b)
    K.raise_on_fault(err)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [30, 320, 1000, 1024, 2048, 2600])
def test_layer_norms_with_a_bias(dtype, width):
    """A norm alone (all rows, gathered rows), and the norm after a sublayer with the next sublayer's in one kernel: the stream
    and the rows have the bits of the kernels in turn."""
    from lockstep_b200 import kernels as K
    from lockstep_b200.config import PartSpec
    from lockstep_b200.parts import Runtime, build_part

    torch.manual_seed(width)
    err = K.new_error_word(DEV)
    rt = Runtime(device=torch.device(DEV), dtype=dtype, page_size=8, max_positions=8, err=err)
    norms = []
    for _ in range(2):
        part = build_part("norm", PartSpec("layernorm", {"width": width, "eps": 1e-5, "tensor": "", "bias": "b"}), rt)
        part.bind({"": torch.randn(width, device=DEV), "b": torch.randn(width, device=DEV)})
        norms.append(part)
    post, following = norms
    h = torch.randn(37, width, device=DEV) * 3 + 2
    x = torch.randn(37, width, device=DEV) * torch.logspace(-3, 2, 37, device=DEV)[:, None] + 1
    ln = lambda part, z: plain.layer_norm(z, d64(part.gain), d64(part.bias), 1e-5)
    for rows in (None, torch.tensor([36, 0, 5, 5], dtype=torch.int32, device=DEV)):
        got = d64(post.forward(h, rows))
        want = ln(post, d64(h if rows is None else h[rows.long()]))
        assert float((got - want).abs().max()) <= _tol(dtype) * (1 + float(want.abs().max()))
    one, two = h.clone(), h.clone()
    assert post.accumulate(one, x) is None
    want = d64(h) + ln(post, d64(x))
    assert float((d64(one) - want).abs().max()) <= 2e-5 * (1 + float(want.abs().max()))
    rows = post.accumulate(two, x, following)
    assert torch.equal(one, two) and torch.equal(rows, following.forward(one)) and rows.dtype == dtype
    # the kernel that closes mixers side by side takes the norm along too
    gains = torch.rand(2, width, device=DEV) + 0.5
    branches = torch.randn(2, 37, width, device=DEV)
    one, two, out = h.clone(), h.clone(), torch.empty(37, width, dtype=dtype, device=DEV)
    K.norm_merge_add(one, branches, gains, 0.5, post.gain, 1e-5, 1e-5, post_bias=post.bias)
    K.norm_merge_add(two, branches, gains, 0.5, post.gain, 1e-5, 1e-5, post_bias=post.bias,
                     follow=(following.gain, following.bias, 1e-5, out))
    merged = 0.5 * (plain.rms_unit(d64(branches), 1e-5) * d64(gains)[:, None]).sum(0)
    want = d64(h) + ln(post, merged)
    assert float((d64(one) - want).abs().max()) <= 2e-5 * (1 + float(want.abs().max()))
    assert torch.equal(one, two) and torch.equal(out, following.forward(one))
    K.raise_on_fault(err)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads, kv, d, dv", [(4, 2, 12, 40), (3, 1, 5, 6), (2, 2, 32, 64), (6, 3, 24, 16), (1, 1, 64, 128)])
def test_heads_of_two_maps_into_the_cache(dtype, heads, kv, d, dv):
    """Queries between zeros where their map's key lies; a key head's two sub-heads side by side; the values; from columns of a
    wider tensor into scattered pages."""
    from lockstep_b200 import kernels as K

    torch.manual_seed(heads * d)
    pad, page, tokens = -(-max(2 * d, dv) // 16) * 16, 8, 21
    cols = 2 * heads * d + kv * (2 * d + dv)
    wide = torch.randn(tokens, cols + 11, device=DEV).to(dtype)
    table = torch.tensor([[3, 0, 5, -1]], dtype=torch.int32, device=DEV)
    pages = torch.full((7, 2, kv, page, pad), 7.0, dtype=dtype, device=DEV)
    q = torch.full((tokens, 2 * heads * pad), 7.0, dtype=dtype, device=DEV)
    gq, gk = torch.rand(d, device=DEV) + 0.5, torch.rand(d, device=DEV) + 0.5
    err = K.new_error_word(DEV)
    K.qkv_finish(wide[:, :cols], q, pages, gq, gk, None, None, torch.arange(tokens, dtype=torch.int32, device=DEV),
                 torch.zeros(tokens, dtype=torch.int32, device=DEV), table, 2 * heads, kv, d, dv, pad, 0, 1e-5, False, True, True,
                 err, maps=2)
    K.raise_on_fault(err)
    x = d64(wide)
    want_q = plain.rms_unit(x[:, :2 * heads * d].reshape(tokens, heads, 2, d), 1e-5) * d64(gq)
    want_k = plain.rms_unit(x[:, 2 * heads * d:2 * (heads + kv) * d].reshape(tokens, kv, 2, d), 1e-5) * d64(gk)
    want_v = x[:, 2 * (heads + kv) * d:cols].reshape(tokens, kv, dv)
    got_q = d64(q).view(tokens, heads, 2, pad)
    full = torch.zeros(tokens, heads, 2, pad, dtype=torch.float64)
    for i in (0, 1):
        full[:, :, i, i * d:(i + 1) * d] = want_q[:, :, i]
    assert float((got_q - full).abs().max()) <= _tol(dtype) * 4 and float(got_q[full == 0].abs().sum()) == 0.0
    for t in range(tokens):
        cell = d64(pages[[3, 0, 5][t // page], :, :, t % page])
        assert float((cell[0, :, :2 * d] - want_k[t].reshape(kv, 2 * d)).abs().max()) <= _tol(dtype) * 4
        assert float((cell[1, :, :dv] - want_v[t]).abs().max()) <= _tol(dtype) * 4
        assert float(cell[0, :, 2 * d:].abs().sum() + cell[1, :, dv:].abs().sum()) == 0.0
    assert float(pages[1].float().mean()) == 7.0                                       # a page of nobody's


def _fake_step(starts_and_lengths, page, nkv, d, dtype, chunk, gen):
    """A step over requests whose keys lie in scattered pages, the pages of finished chunks poisoned and taken out of the
    block table: (context, cache view, keys and values per request)."""
    from lockstep_b200 import kernels as K
    from lockstep_b200.engine.batch import StepContext, StepEntry

    class View:
        pass

    total = [s + n for s, n in starts_and_lengths]
    per = [-(-t // page) for t in total]
    order = torch.randperm(sum(per), generator=gen).tolist()
    pages = torch.full((sum(per) + 1, 2, nkv, page, d), 1e30, dtype=dtype, device=DEV)
    table = torch.full((len(per), max(per)), -1, dtype=torch.int32)
    keys = []
    for r, (start, _) in enumerate(starts_and_lengths):
        kv = torch.randn(2, nkv, total[r], d, generator=gen).to(dtype)
        keys.append(kv)
        first = start // chunk * chunk // page if chunk else 0
        for lp in range(per[r]):
            phys = order.pop()
            if lp >= first:
                table[r, lp] = phys
                part = kv[:, :, lp * page:(lp + 1) * page]
                pages[phys, :, :, :part.shape[2]] = part.to(DEV)
    view = View()
    view.pages, view.block_table = pages, table.to(DEV)
    entries = [StepEntry(f"u{r}", [0] * n, s, [0]) for r, (s, n) in enumerate(starts_and_lengths)]
    err = K.new_error_word(DEV)
    return StepContext(entries, list(range(len(per))), torch.device(DEV), err, K.attention_split_size()), view, keys, err


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("page", [8, 16, 64])
@pytest.mark.parametrize("heads, kv, d, dv", [(6, 2, 32, 64), (2, 2, 64, 128), (3, 1, 20, 30)])
@pytest.mark.parametrize("chunk", [1, 7, 64, 100, 300, 0])
def test_differential_attention_in_chunks(dtype, page, heads, kv, d, dv, chunk):
    """Portions and single tokens at a chunk's first and last positions, across its edge and far on, against the plain maps
    and their difference; what lies in finished chunks is poison.  A step of single tokens alone folds, subtracts and gates in
    one kernel, with the bits of the kernels in turn."""
    from lockstep_b200 import kernels as K
    from lockstep_b200.parts.attention import MapDifference, ScoreExtras, attend
    from lockstep_b200.parts.base import Runtime

    gen = torch.Generator().manual_seed(chunk * 7 + d)
    D = -(-max(2 * d, dv) // 16) * 16
    c = chunk or 90
    portions = [(0, 40), (c - 1, 9), (5 * c // 2, 2), (700, 130)]
    singles = [(0, 1), (c - 1, 1), (c, 1), (3 * c - 1, 1), (3 * c, 1), (999, 1), (255, 1), (256, 1)]
    err0 = K.new_error_word(DEV)
    rt = Runtime(device=torch.device(DEV), dtype=dtype, page_size=page, max_positions=2048, err=err0)
    lam, diff = 0.7, 0.35
    for work in (portions + singles, singles):
        ctx, view, keys, err = _fake_step(work, page, kv, D, dtype, chunk, gen)
        tokens = ctx.num_tokens
        q = torch.zeros(tokens, heads, 2, D)
        raw = torch.randn(tokens, heads, 2, d, generator=gen).to(dtype)
        for i in (0, 1):
            q[:, :, i, i * d:(i + 1) * d] = raw[:, :, i].float()
        q = q.to(dtype).view(tokens, -1).to(DEV)
        gate = torch.randn(tokens, heads + 3, generator=gen).to(dtype).to(DEV)[:, 3:]
        close = MapDifference(heads, dv, lam, 1.0 - diff, 1e-5, gate)
        before = K.kernel_counts()
        out = attend(rt, q, ctx, view, 2 * heads, kv, D, -chunk, 0.3, dtype == F32, ScoreExtras(), close)
        K.raise_on_fault(err)
        after = K.kernel_counts()
        ran = {k for k in after if after[k] > before.get(k, 0)}
        assert ("map_difference_fold" in ran) == (work is singles) and ("map_difference" in ran) == (work is not singles)
        if dtype == BF16 and D in (64, 128):
            assert "attention_decode_mma" in ran and ("attention_prefill_tc" in ran) == (work is not singles)
        at = 0
        for (start, n), both in zip(work, keys):
            total = start + n
            k, v = d64(both[0]).transpose(0, 1), d64(both[1]).transpose(0, 1)[..., :dv]     # [keys, kv, D]
            seen = plain.visible(total, chunk or None)
            maps = []
            for i in (0, 1):
                qq = torch.zeros(total, heads, d, dtype=torch.float64)
                qq[start:] = d64(raw[at:at + n, :, i])
                maps.append(plain.softmax_attention(qq, k[..., i * d:(i + 1) * d], v, 0.3, seen)[start:])
            want = plain.combine_maps(*maps, lam, diff, d64(gate[at:at + n]), 1e-5)
            got = d64(out[at:at + n]).view(n, heads, dv)
            assert float((got - want).abs().max()) <= (3e-5 if dtype == F32 else 4e-2), (start, n)
            at += n
        if work is singles:
            rows = attend(rt, q, ctx, view, 2 * heads, kv, D, -chunk, 0.3, dtype == F32, ScoreExtras())
            assert torch.equal(out, close.rows(rt, rows))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("tokens, heads, D, dv", [(1, 1, 16, 6), (7, 3, 48, 40), (300, 4, 64, 64), (65, 2, 256, 250)])
def test_difference_of_two_maps(dtype, tokens, heads, D, dv):
    """With and without a gate; rows whose maps nearly cancel, where eps decides."""
    from lockstep_b200 import kernels as K

    torch.manual_seed(tokens + D)
    attn = torch.randn(tokens, heads, 2, D, device=DEV).to(dtype)
    attn[0] = 0.0
    gate = torch.randn(tokens, heads, device=DEV).to(dtype)
    for g in (gate, None):
        out = torch.empty(tokens, heads * dv, dtype=dtype, device=DEV)
        K.map_difference(attn.view(tokens, -1), g, out, heads, dv, -0.4, 1.3, 1e-4)
        a = d64(attn)
        want = plain.combine_maps(a[:, :, 0, :dv], a[:, :, 1, :dv], -0.4, -0.3, d64(g) if g is not None else torch.full((tokens, heads), 50.0), 1e-4)
        assert float((d64(out).view(tokens, heads, dv) - want).abs().max()) <= _tol(dtype) * (1 + float(want.abs().max()))
        assert float(out[0].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("tokens, heads, n, k", [(1, 3, 24, 40), (70, 5, 66, 64), (9, 2, 10, 10), (130, 8, 128, 128)])
def test_per_head_products_with_a_gate(dtype, tokens, heads, n, k):
    from lockstep_b200 import kernels as K

    torch.manual_seed(tokens * n)
    a = torch.randn(tokens, heads * (k + 6), device=DEV).to(dtype)
    w = (torch.randn(heads, n, k, device=DEV) * k ** -0.5).to(dtype)
    gate = (torch.randn(tokens, heads * n + 8, device=DEV) * 2).to(dtype)[:, 8:]
    out, bare = (torch.empty(tokens, heads * n, dtype=dtype, device=DEV) for _ in range(2))
    K.heads_product(a, k + 6, w, out, n, gate=gate)
    K.heads_product(a, k + 6, w, bare, n)
    sums = torch.einsum("thk,hnk->thn", d64(a).view(tokens, heads, k + 6)[..., :k], d64(w)).reshape(tokens, -1)
    assert float((d64(bare) - sums).abs().max()) <= _tol(dtype) * 4
    assert float((d64(out) - sums * torch.sigmoid(d64(gate))).abs().max()) <= _tol(dtype) * 4


@pytest.mark.parametrize("experts, top, groups, scale", [
    (12, 3, (4, 3), 1.4), (6, 2, (3, 1), 1.0), (1, 1, (1, 1), 2.0), (5, 5, None, 0.7), (32, 4, (8, 4), 2.5), (40, 6, (10, 5), 1.0),
    (64, 8, (64, 9), 1.0), (96, 4, (2, 1), 3.0), (300, 7, (60, 13), 1.0), (512, 16, (8, 4), 2.5)])
def test_choice_among_the_best_groups(experts, top, groups, scale):
    """Both kernels of the choice (one that also plans, for few tokens), with negative choice scores and corrections that change
    it; a tie goes to the lower group and the lower expert."""
    from lockstep_b200 import kernels as K

    gen = torch.Generator().manual_seed(experts + top)
    correction = (torch.randn(experts, generator=gen) * 0.2 - 1.5).float()
    router = {"top": top, "scale": scale, "groups": dict(zip(("count", "keep"), groups)) if groups else None}
    pick = {"factor": scale, **({"groups": groups[0], "keep": groups[1]} if groups else {})}
    err = K.new_error_word(DEV)
    for tokens in (5, 200):
        z = torch.randn(tokens, experts + 3, generator=gen)
        z[0] = 0.25                                          # all scores equal: the corrections decide
        logits = z.to(DEV)
        w = {"m.router": torch.eye(experts + 3, dtype=torch.float64)[:experts], "m.correction": correction.double()}
        plain.ROUTING_GAPS = []
        want_ids, want_w = plain.route(z.double(), w, "m", router)
        plain.ROUTING_GAPS = None
        ids = torch.empty(tokens, top, dtype=torch.int32, device=DEV)
        weights = torch.empty(tokens, top, device=DEV)
        if tokens <= K.FEW_TOKENS:
            pairs = tokens * top
            bound = pairs + experts
            plan = torch.empty(1 + 3 * bound, dtype=torch.int32, device=DEV)
            row_token, pair_row = (torch.empty(pairs, dtype=torch.int32, device=DEV) for _ in range(2))
            row_weight = torch.empty(pairs, device=DEV)
            K.experts_route_plan(logits[:, :experts], top, ids, weights, experts, 0, correction.to(DEV), experts, 64, plan, bound,
                                 row_token, row_weight, pair_row, err, **pick)
            assert torch.equal(row_token[pair_row.long()].cpu(), torch.arange(tokens, dtype=torch.int32).repeat_interleave(top))
            assert torch.equal(row_weight[pair_row.long()], weights.view(-1))
        else:
            K.experts_route(logits[:, :experts], top, ids, weights, experts=experts, softmax=0, correction=correction.to(DEV), **pick)
        K.raise_on_fault(err)
        # (a row where float32 might order two scores otherwise is left out: hardly any)
        same = (ids.cpu().long() == want_ids).all(-1)
        assert float(same.float().mean()) > 0.985
        assert float((weights.cpu().double() - want_w)[same].abs().max()) <= 2e-6 * scale
    # ties: no correction, equal scores
    ids, weights = torch.empty(2, top, dtype=torch.int32, device=DEV), torch.empty(2, top, device=DEV)
    K.experts_route(torch.zeros(2, experts, device=DEV), top, ids, weights, experts=experts, softmax=0, **pick)
    assert ids.tolist() == [list(range(top))] * 2 and torch.allclose(weights, torch.full_like(weights, scale / top))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads, dk, dv, cap", [(3, 8, 20, 9.0), (1, 10, 6, 1.5), (4, 64, 96, 15.0)])
def test_matrix_memory_across_calls(dtype, heads, dk, dv, cap):
    """The mixer as a part, three requests in portions across calls, against the plain mixer on the whole sequences; biases so
    large that the running maximum moves."""
    from lockstep_b200 import kernels as K
    from lockstep_b200.config import PartSpec
    from lockstep_b200.parts import Runtime, build_part

    torch.manual_seed(heads * dk + dv)
    width = 40
    err = K.new_error_word(DEV)
    rt = Runtime(device=torch.device(DEV), dtype=dtype, page_size=8, max_positions=8, err=err)
    part = build_part("mixer", PartSpec("mlstm", {"hidden_size": width, "num_heads": heads, "key_dim": dk, "value_dim": dv,
                                                  "gate_cap": cap, "norm_eps": 1e-5}), rt, position=None)
    w = {n: (torch.randn(s.shape) * (width ** -0.5 if s.role == "matrix" else 0.3)).to(dtype) for n, s in part.weight_specs().items()}
    w["i.b"], w["f.b"] = (torch.randn(heads) * 4).to(dtype), (torch.randn(heads) + 3).to(dtype)
    w["norm"] = (torch.rand(heads * dv) + 0.5).to(dtype)
    part.bind({n: t.to(DEV) for n, t in w.items()})
    lengths = {1: 41, 3: 6, 0: 11}
    x = {s: torch.randn(n, width).to(dtype) for s, n in lengths.items()}
    m = {"heads": heads, "dim": dk, "vdim": dv, "gate_cap": cap}
    want = {s: plain.mlstm_mixer(d64(x[s]), {f"m.{n}": d64(t) for n, t in w.items()}, "m", m, 1e-5) for s in lengths}

    class Context:
        pass

    cache = Context()
    cache.state = torch.zeros(5, *part.cache_need().state_shape, device=DEV)
    got = {s: [] for s in lengths}
    for cut in ({1: (0, 17), 3: (0, 1), 0: (0, 2)}, {1: (17, 18), 0: (2, 11)}, {1: (18, 41), 3: (1, 6)}):
        ctx = Context()
        ctx.token_slot = torch.tensor([s for s, (a, b) in cut.items() for _ in range(b - a)], dtype=torch.int32, device=DEV)
        rows = torch.cat([x[s][a:b] for s, (a, b) in cut.items()]).to(DEV).contiguous()
        out = torch.zeros(rows.shape[0], width, device=DEV)
        part.forward(rows, ctx, cache, out)
        at = 0
        for s, (a, b) in cut.items():
            got[s].append(d64(out[at:at + b - a]))
            at += b - a
    K.raise_on_fault(err)
    for s in lengths:
        assert float((torch.cat(got[s]) - want[s]).abs().max()) <= (1e-3 if dtype == F32 else 6e-2) * (1 + float(want[s].abs().max())), s
    assert float(cache.state[2].abs().max()) == 0.0 and float(cache.state[4].abs().max()) == 0.0     # slots nobody used


# ---------------------------------------------------------------------------
# one-layer models: every mechanism in the engine, in every cutting
# ---------------------------------------------------------------------------

SMALL = {
    "attention": [M.bare(M.attention(4, 2, 24, 16, chunk=20))],
    "attention_maps_of_ten": [M.bare(M.attention(2, 2, 10, 12, chunk=9, diff=0.8))],
    "attention_chunk_of_a_page": [M.bare(M.attention(2, 1, 16, 32, chunk=8, diff=0.0))],
    "attention_chunk_of_one": [M.bare(M.attention(2, 1, 16, 24, chunk=1))],
    "attention_no_chunks": [M.bare(M.attention(3, 1, 16, 32, diff=-0.5))],
    "mlstm": [M.bare(M.mlstm(3, 8, 24, cap=6.0))],
    "latent": [M.bare(M.latent(3, 12, 20, 36))],
    "latent_wide": [M.bare(M.latent(1, 40, 8, 176))],
    "dense": [M.dense(M.mlstm(1, 16, 16), 40)],
    "experts": [M.moe(M.latent(1, 16, 16, 16), 6, 2, 24, groups=(3, 2), scale=2.0, shared=16)],
    "experts_of_groups_of_one": [M.moe(M.latent(1, 16, 16, 16), 5, 2, 16, groups=(5, 3), scale=0.5)],
    "experts_all": [M.moe(M.mlstm(1, 16, 16), 4, 4, 8, groups=(2, 2), shared=40)],
}


@pytest.fixture(scope="module")
def zoo(tmp_path_factory):
    cache = {}

    def get(config, dtype, lengths, seed=7, edit=None, key=None):
        key = (key or json.dumps(config, sort_keys=True), dtype, tuple(lengths))
        if key not in cache:
            folder = M.make_folder(tmp_path_factory.mktemp("tesozen"), config, seed=seed, dtype=dtype, edit=edit)
            requests, want = {}, {}
            for i, n in enumerate(lengths):
                # no request rests on a router's close call: another draw of tokens where float32 would decide one
                for draw in range(20):
                    tokens = H.random_tokens(n, config["vocab"], seed=50 + i + 1000 * draw)
                    logits, gap = M.plain_logits_and_gap(folder, tokens)
                    if gap > 5e-5:
                        break
                requests[f"r{i}"], want[f"r{i}"] = tokens, logits.float()
            cache[key] = (folder, requests, want)
        return cache[key]

    return get


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SMALL))
def test_small_models_in_every_cutting(zoo, name, dtype):
    folder, requests, want = zoo(M.layers_model(SMALL[name]), dtype, [45, 130, 9, 77])
    rows = {}
    for plan_name, plan in PLANS.items():
        steps = plan(requests)
        runner = make_runner(folder, dtype, 8, steps)
        rows[plan_name] = H.run_plan(runner, steps)
        M.assert_close(rows[plan_name], want, dtype, f"{name}, {plan_name}",
                       None if name.startswith("experts") else 0.0 if dtype == "float32" else 0.02)
        runner.cache.audit()
    if dtype == "float32":
        # a row's arithmetic does not depend on how its request was cut or on the batch
        for plan_name in PLANS:
            for key, row in rows["whole"].items():
                assert torch.equal(row, rows[plan_name][key]), (name, plan_name, key)


LENGTHS = {"S": [70, 300, 37, 150, 129], "T": [45, 310, 90, 33, 260], "U": [40, 190, 75, 131]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("plan_name", sorted(PLANS))
@pytest.mark.parametrize("model", sorted(M.MODELS))
def test_whole_models_in_every_cutting(zoo, model, plan_name, dtype):
    config, page = M.MODELS[model]
    folder, requests, want = zoo(config, dtype, LENGTHS[model])
    steps = PLANS[plan_name](requests)
    runner = make_runner(folder, dtype, page, steps, poison_freed_pages=True)
    rows = H.run_plan(runner, steps)
    M.assert_close(rows, want, dtype, f"model {model}, {plan_name}")
    runner.cache.audit()
    if plan_name == "mixed":
        assert runner.cache.reused_pages() > 0           # more requests than slots, and few pages
    if plan_name == "then_single" and runner.graphs is not None:
        assert runner.graphs.replays > 100               # decoded tokens ran as recorded steps
    assert sum(g.poisoned for g in runner.cache.paged) > 0


@pytest.mark.parametrize("seed", [1, 4, 9])
def test_configurations_drawn_from_a_seed(zoo, seed):
    """Larger models of sizes nobody chose (see ``tesozen_models.random_config``) in float32: four requests of up to 330
    tokens whole, and on three slots with portions of some beside single tokens of others, with the same bits."""
    config = M.random_config(seed)
    folder, requests, want = zoo(config, "float32", [90, 330, 41, 200], seed=seed, key=f"drawn-{seed}")
    rows = {}
    for plan_name in ("whole", "mixed"):
        steps = PLANS[plan_name](requests)
        runner = make_runner(folder, "float32", 16, steps)
        rows[plan_name] = H.run_plan(runner, steps)
        M.assert_close(rows[plan_name], want, "float32", f"drawn configuration {seed}, {plan_name}")
        runner.cache.audit()
    for key, row in rows["whole"].items():
        assert torch.equal(row, rows["mixed"][key]), key


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_stream_after_every_layer(zoo, dtype):
    from safetensors.torch import load_file

    from lockstep_b200.engine.batch import StepContext, StepEntry

    name = "S" if dtype == "float32" else "U"          # (no router of U has a choice: nothing to call closely)
    config, page = M.MODELS[name]
    folder, requests, _ = zoo(config, dtype, LENGTHS[name])
    tokens = requests["r0"]
    _, want = plain.forward(tokens, load_file(str(folder / "model.safetensors")), json.loads((folder / "config.json").read_text()),
                            streams=True)
    runner = make_runner(folder, dtype, page, num_pages=16, use_graphs=False)
    runner.open("a")
    runner.cache.reserve("a", len(tokens))
    runner.cache.sync()
    ctx = StepContext([StepEntry("a", tokens, 0, [0])], [runner.cache.slots["a"]], runner.device, runner.err, runner.split_size)
    ends, at = [], 1
    for run in runner.spec.schedule:
        at += len(runner.model.blocks[run.layer].steps())
        ends.append(at)
    h, k = None, 0
    for i, (_, fn) in enumerate(runner.program[:-1]):
        h = fn(h, ctx)
        if i + 1 in ends:
            err = float((h.double().cpu() - want[k]).abs().max()) / float(want[k].abs().max())
            assert err <= (2e-5 if dtype == "float32" else 5e-2), (k, err)
            k += 1
    assert k == len(runner.spec.schedule) >= 5


# ---------------------------------------------------------------------------
# weights that make a fault show
# ---------------------------------------------------------------------------

def _map_weights(folder, tokens):
    """[2, heads, n, n]: the softmax weights of both maps of layer 0."""
    from safetensors.torch import load_file

    w = {k: v.double() for k, v in load_file(str(folder / "model.safetensors")).items()}
    cfg = json.loads((folder / "config.json").read_text())
    m, n = cfg["layers"][0]["mixer"], len(tokens)
    x = plain.norm(w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"], w, "l0.norm1", cfg["norm"]["eps"])
    q = plain.rms_unit((x @ w["l0.mix.q"].T).view(n, m["heads"], 2, -1), 1e-5) * w["l0.mix.q.norm"]
    k = plain.rms_unit((x @ w["l0.mix.k"].T).view(n, m["kv_heads"], 2, -1), 1e-5) * w["l0.mix.k.norm"]
    k = k.repeat_interleave(m["heads"] // m["kv_heads"], dim=1)
    s = torch.einsum("ihmd,jhmd->mhij", q, k) * m["scale"]
    return torch.softmax(s.masked_fill(~plain.visible(n, m["mask"]["size"]), float("-inf")), dim=-1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk, dim, vdim", [(37, 16, 16), (64, 32, 64), (200, 64, 128), (30, 24, 96)])
def test_sharp_softmax_at_the_edges_of_chunks(zoo, chunk, dim, vdim, dtype):
    """Scores so large that every row's softmax is a choice of one key: rows of either map whose key is their
    chunk's first; chunks of one position more or less, none at all, or another weight of the second map give other logits.  Freed pages are poisoned."""
    from lockstep_b200 import kernels as K

    # (q and k have length sqrt(dim): the scale makes the scores)
    config = M.layers_model([M.bare(M.attention(2, 1, dim, vdim, chunk=chunk, scale=50.0 / dim, diff=0.5))], width=64)
    folder, requests, want = zoo(config, dtype, [520, 75], key=f"sharp-{chunk}-{dim}")
    pr = _map_weights(folder, requests["r0"])
    rows = torch.arange(520)[None, None]
    sure, best = pr.max(-1).values > 0.4, pr.argmax(-1)
    inside = sure & (best == rows // chunk * chunk) & (rows % chunk > 0) & (rows >= chunk)
    assert int(inside[0].sum()) >= 1 and int(inside[1].sum()) >= 1
    changes = [lambda m: m["mask"].update(size=chunk - 1), lambda m: m["mask"].update(size=chunk + 1), lambda m: m.pop("mask"),
               lambda m: m.update(diff=0.0)]
    for change in changes:
        other = M.plain_logits(folder, requests["r0"], edit=lambda c: change(c["layers"][0]["mixer"]))
        assert float((other.float() - want["r0"]).abs().max()) > 0.3
    before = K.kernel_counts()
    for plan_name, plan in PLANS.items():
        steps = plan(requests)
        runner = make_runner(folder, dtype, 8, steps, poison_freed_pages=True)
        M.assert_close(H.run_plan(runner, steps), want, dtype, f"sharp chunks of {chunk}, {plan_name}", 0.0 if dtype == "float32" else 0.02,
                       slack=1.0 if dtype == "float32" else 2.0)
        assert sum(g.poisoned for g in runner.cache.paged) > 0
    after = K.kernel_counts()
    for kernel in ("attention_prefill_tc", "attention_decode_mma"):
        ran = after.get(kernel, 0) - before.get(kernel, 0)
        assert (ran > 0) == (dtype == "bfloat16" and dim in (32, 64)), kernel


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank", [48, 64, 128])
def test_sharp_latent_attention_reaches_far_keys(zoo, rank, dtype):
    """Scores so large that a row's softmax is a choice of one key, often one hundreds of tokens back; another token there gives
    the row other logits."""
    from safetensors.torch import load_file

    config = M.layers_model([M.bare(M.latent(2, 32, 40, rank, scale=5.0 * rank ** -0.5))], width=64, vocab=1009)
    folder, requests, want = zoo(config, dtype, [500, 61], key=f"far-{rank}")
    tokens = requests["r0"]
    w = {k: v.double() for k, v in load_file(str(folder / "model.safetensors")).items()}
    x = plain.norm(w["embed"][torch.tensor(tokens)] * config["embedding"]["scale"], w, "l0.norm1", 1e-5)
    c = plain.rms_unit(x @ w["l0.mix.dkv"].T, 1e-5) * w["l0.mix.dkv.norm"]
    s = torch.einsum("ihd,jhd->hij", (x @ w["l0.mix.q"].T).view(500, 2, 32), (c @ w["l0.mix.uk"].T).view(500, 2, 32))
    pr = torch.softmax((s * config["layers"][0]["mixer"]["scale"]).masked_fill(~plain.visible(500)[None], float("-inf")), dim=-1)
    rows = torch.arange(500)[None]
    far = (rows - pr.argmax(-1) > 200) & (pr.max(-1).values > 0.5)
    assert int(far.sum()) >= 10
    head, row = far.nonzero()[-1].tolist()
    at = int(pr[head, row].argmax())
    other = tokens[:at] + [(tokens[at] + 5) % 1009] + tokens[at + 1:]
    assert float((M.plain_logits(folder, other)[row].float() - want["r0"][row]).abs().max()) > 0.3
    for plan_name, plan in PLANS.items():
        steps = plan(requests)
        runner = make_runner(folder, dtype, 16, steps)
        M.assert_close(H.run_plan(runner, steps), want, dtype, f"far keys, {plan_name}", 0.0 if dtype == "float32" else 0.02,
                       slack=1.0 if dtype == "float32" else 2.0)


def _remember(tensors):
    for name in tensors:
        if name.endswith(".f.b"):
            tensors[name] = torch.full_like(tensors[name], 8.0)
        if name.endswith(".i"):
            tensors[name] = tensors[name] * 0.2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_open_forget_gates_carry_the_first_tokens_through_long_decoding(zoo, dtype):
    """Forget gates near one: the first token still moves the last logits after 260 tokens, 200 of them decoded
    one by one."""
    config = M.layers_model([M.bare(M.mlstm(2, 16, 16, cap=10.0)), M.bare(M.mlstm(1, 32, 8, cap=12.0))])
    folder, requests, want = zoo(config, dtype, [260], edit=_remember, key="remember")
    tokens = requests["r0"]
    moved = M.plain_logits(folder, [(tokens[0] + 1) % 97] + tokens[1:])[-1]
    assert float((moved.float() - want["r0"][-1]).abs().max()) > 1e-3      # the plain model itself remembers
    plans = dict(PLANS, long_decoding=lambda r: H.plan_bulk_then_single(r, tail=200))
    for plan_name, plan in plans.items():
        steps = plan(requests)
        runner = make_runner(folder, dtype, 16, steps)
        M.assert_close(H.run_plan(runner, steps), want, dtype, f"slow decays, {plan_name}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_steps_of_a_repeating_shape_are_recorded_and_replayed(zoo, dtype):
    """Portions of 300 tokens with two wanted rows: from its third occurrence the step is a recorded one, with the bits of
    an unrecorded step."""
    config, page = M.MODELS["U"]
    folder, requests, want = zoo(config, dtype, [900, 900, 601], key="recorded")
    steps = []
    for uid, toks in requests.items():
        for i in range(0, len(toks) - 1, 300):
            n = min(300, len(toks) - i)
            steps.append({"entries": [(uid, toks[i:i + n], [n - 1, 0])], "end": [uid] if i + n == len(toks) else []})
    steps.append({"entries": [("r2", requests["r2"][600:601], [0])], "end": ["r2"]})
    runner = make_runner(folder, dtype, page, steps, max_live=2)
    rows = H.run_plan(runner, steps)
    assert runner.graphs is not None and runner.graphs.mixed_replays >= 4
    M.assert_close(rows, want, dtype, "recorded steps of 300 tokens")
    fresh = make_runner(folder, dtype, page, steps, max_live=2, use_graphs=False)
    plain_rows = H.run_plan(fresh, steps)
    for key, row in rows.items():
        assert torch.equal(row, plain_rows[key]), key


# ---------------------------------------------------------------------------
# the entry point, the scheduler, the command line, the trace runner
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(tmp_path, dtype):
    from lockstep_b200 import Engine, Request

    config, page = M.MODELS["S"]
    folder = M.make_folder(tmp_path, config, seed=21, dtype=dtype)
    engine = Engine(folder, dtype=dtype, num_pages=64, page_size=page, max_running=12, max_step_tokens=96,
                    max_seq_len=512)
    prompts = {f"g{i}": H.random_tokens(n, config["vocab"], seed=300 + i)
               for i, n in enumerate([33, 7, 120, 1, 64, 18, 45, 2, 90, 11])}
    got = engine.generate([Request(uid=u, prompt=p, max_new_tokens=8) for u, p in prompts.items()])
    wrong = []
    for uid, prompt in prompts.items():
        assert len(got[uid]) == 8
        rows = M.plain_logits(folder, list(prompt) + got[uid])     # causal: one pass gives every step's logits
        for i, tok in enumerate(got[uid]):
            row = rows[len(prompt) + i - 1]
            margin = 2 * M.TOLERANCE[dtype] * (1 + float(row.abs().max()))
            if not float(row[tok]) >= float(row.max()) - margin:
                wrong.append((uid, i, tok))
    assert len(wrong) <= int(M.CLOSE_CALLS[dtype] * 80), (dtype, wrong)
    assert engine.runner.graphs is not None and engine.runner.graphs.replays > 0
    engine.cache.audit()
    assert engine.cache.live == 0


def test_generation_reuses_a_prefix_beside_chunks(tmp_path):
    """Attention layers alone: the next turn of a conversation adopts the pages of the first that its chunk and the latent layer
    still read, and generates what a request without reuse does."""
    from lockstep_b200 import Engine, Request

    config = M.layers_model([M.dense(M.attention(2, 1, 16, 32, chunk=24), 40), M.bare(M.latent(2, 16, 32, 32)),
                             M.bare(M.attention(2, 1, 8, 32, chunk=24, diff=0.6))], width=64)
    folder = M.make_folder(tmp_path, config, seed=5, dtype="float32")
    first = H.random_tokens(90, config["vocab"], 1)
    made = {}
    for reuse in (False, True):
        engine = Engine(folder, dtype="float32", num_pages=64, page_size=8, max_running=2, max_step_tokens=64, max_seq_len=512,
                        enable_prefix_cache=reuse)
        turn = engine.generate([Request(uid="a", prompt=first, max_new_tokens=6)])["a"]
        again = engine.generate([Request(uid="b", prompt=first + turn + [3, 4], max_new_tokens=6)])["b"]
        made[reuse] = (turn, again)
        engine.cache.audit()
    assert made[True] == made[False]


def test_the_command_line_writes_a_random_model_and_runs_a_workload(tmp_path):
    config, page = M.MODELS["U"]
    (tmp_path / "config.json").write_text(json.dumps(config))
    folder = tmp_path / "model"
    lockstep = [sys.executable, str(ROOT / "bin" / "lockstep")]
    proc = subprocess.run(lockstep + ["random-model", "--config", str(tmp_path / "config.json"), "--out", str(folder),
                                      "--seed", "5", "--init-std", "0.15", "--gain-std", "0.1"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    prompts = {f"c{i}": H.random_tokens(n, config["vocab"], 95 + i) for i, n in enumerate([4, 23, 50])}
    workload = tmp_path / "workload.json"
    requests = [{"uid": u, "prompt": p, "max_new_tokens": 10} for u, p in prompts.items()]
    requests += [{"uid": "s0", "prompt": prompts["c1"], "max_new_tokens": 12, "temperature": 0.8, "top_p": 0.9, "seed": 3}]
    workload.write_text(json.dumps(requests))
    proc = subprocess.run(lockstep + ["run", "--model", str(folder), "--dtype", "float32", "--workload", str(workload),
                                      "--policy", "fixed-chunk:16", "--num-blocks", "40", "--block-size", str(page),
                                      "--max-running", "3"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = {l["uid"]: l for l in (json.loads(x) for x in proc.stdout.splitlines() if x.startswith("{"))}
    assert set(lines) == set(prompts) | {"s0"}
    for uid, prompt in prompts.items():
        got = lines[uid]["generated"]
        assert len(got) == 10
        rows = M.plain_logits(folder, list(prompt) + got)
        for i, tok in enumerate(got):
            row = rows[len(prompt) + i - 1]
            assert float(row[tok]) >= float(row.max()) - 2 * M.TOLERANCE["float32"] * (1 + float(row.abs().max()))
    assert len(lines["s0"]["generated"]) == 12 and all(0 <= t < config["vocab"] for t in lines["s0"]["generated"])


def test_trace_runner_replays_a_trace(tmp_path):
    config, page = M.MODELS["T"]
    folder = M.make_folder(tmp_path, config, seed=9, dtype="bfloat16")
    requests = {f"t{i}": H.random_tokens(n, config["vocab"], seed=70 + i) for i, n in enumerate([40, 130, 25, 61, 90])}
    steps = H.plan_mixed(requests, max_live=4)
    out = tmp_path / "out"
    for dtype in ("bfloat16", "float32"):
        proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype,
                               "--out", str(out / dtype), "--max-tokens", str(H.max_live_tokens(steps, 64))],
                              input=H.plan_to_jsonl(steps), capture_output=True, text=True, timeout=900)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
        want = {u: M.plain_logits(folder, t).float() for u, t in requests.items()}
        at = {u: 0 for u in requests}
        rows = {}
        for i, step in enumerate(steps):
            got = np.fromfile(out / dtype / f"{i}.f32", dtype="<f4").reshape(-1, config["vocab"])
            r = 0
            for uid, toks, wanted in step["entries"]:
                for wpos in wanted:
                    rows[(uid, at[uid] + wpos)] = torch.from_numpy(got[r].copy())
                    r += 1
                at[uid] += len(toks)
            assert r == got.shape[0]
        M.assert_close(rows, want, dtype, f"trace runner, {dtype}")
