"""Kusolorn on the device against the plain implementation: the kernels of every mechanism alone (gelu in a product's
epilogue, finishing of heads with rotated pairs, a norm without a gain and mixed values, attention with kept first positions
and capped scores, the matrix memory and the delta rule with a decay per head across calls, the token input), one-layer
models, and whole models cut in four ways (whole prompts; a prompt and then token by token; portions down to one and two
tokens; up to three live requests, portions of some beside single tokens of others, on so few pages and slots that they are
used again), in float32 and bfloat16; weights made so that a window's edge, a kept position, a far key, a lost state shows;
greedy generation through the entry point and the scheduler; the command line; the trace runner."""

from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import helpers as H
import kusolorn_models as M
from plain import kusolorn_plain as plain

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
def test_gelu_in_the_products_epilogue(dtype, tokens, n, k):
    from lockstep_b200 import kernels as K

    torch.manual_seed(tokens + n)
    x = (torch.randn(tokens, k, device=DEV) * 2).to(dtype)
    w = (torch.randn(n, k, device=DEV) * k ** -0.5).to(dtype)
    out = torch.empty(tokens, n, dtype=dtype, device=DEV)
    err = K.new_error_word(DEV)
    K.gemm_nt(x, w, out, K.EPILOGUE_GELU, err=err)
    want = plain.gelu_tanh(d64(x) @ d64(w).T)
    assert float((d64(out) - want).abs().max()) <= _tol(dtype) * (1 + float(want.abs().max()))
    # the norm made inside the product gives the bits of the norm in front of it
    if dtype == BF16 and k % 8 == 0:
        h = torch.randn(tokens, k, device=DEV)
        gain = torch.rand(k, device=DEV) + 0.5
        a, b = torch.empty_like(out), torch.empty_like(out)
        normed = torch.empty(tokens, k, dtype=BF16, device=DEV)
        K.rmsnorm(h, gain, normed, 1e-5, err)
        K.gemm_nt(normed, w, a, K.EPILOGUE_GELU, err=err)
        if K.gemm_nt_tc_rmsnorm(h, gain, 1e-5, w, b, K.EPILOGUE_GELU, err):
            assert torch.equal(a, b)
    K.raise_on_fault(err)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("nq, nkv, d, dv, rot, normed, mixed", [
    (4, 2, 24, 40, 16, True, True), (3, 1, 10, 6, 6, True, False), (2, 2, 64, 64, 64, True, True), (6, 3, 32, 16, 0, False, True),
    (1, 1, 128, 128, 32, True, True)])
def test_heads_with_rotated_pairs_and_mixed_values(dtype, nq, nkv, d, dv, rot, normed, mixed):
    """Queries into their padded heads; keys and values into the right places of scattered pages."""
    from lockstep_b200 import kernels as K

    torch.manual_seed(nq * d)
    pad, page, tokens = -(-max(d, dv) // 16) * 16, 8, 21
    cols = nq * d + nkv * (d + dv)
    qkv = torch.randn(tokens, cols, device=DEV).to(dtype)
    other = torch.randn(tokens, nkv * dv + 9, device=DEV).to(dtype)[:, 9:]            # columns of a wider tensor
    lam = torch.tensor([0.3], device=DEV)
    freq = plain.rotation_frequencies(rot, 300.0) if rot else torch.zeros(0, dtype=torch.float64)
    ang = torch.arange(64, dtype=torch.float64)[:, None] * freq[None]
    cos, sin = ang.cos().float().to(DEV).contiguous(), ang.sin().float().to(DEV).contiguous()
    table = torch.tensor([[3, 0, 5, -1]], dtype=torch.int32, device=DEV)
    pages = torch.full((7, 2, nkv, page, pad), 7.0, dtype=dtype, device=DEV)
    q = torch.empty(tokens, nq * pad, dtype=dtype, device=DEV)
    ones = torch.ones(d, device=DEV)
    err = K.new_error_word(DEV)
    K.qkv_finish(qkv, q, pages, ones if normed else None, ones if normed else None, cos, sin,
                 torch.arange(tokens, dtype=torch.int32, device=DEV), torch.zeros(tokens, dtype=torch.int32, device=DEV), table,
                 nq, nkv, d, dv, pad, rot, 1e-5, False, True, True, err, interleaved=True,
                 v_other=other if mixed else None, v_mix=lam if mixed else None)
    K.raise_on_fault(err)
    x = d64(qkv)
    turn = lambda z: plain.rotate_pairs(z, freq) if rot else z
    unit = lambda z: plain.rms_unit(z, 1e-5) if normed else z
    want_q = unit(turn(x[:, :nq * d].reshape(tokens, nq, d)))
    want_k = unit(turn(x[:, nq * d:(nq + nkv) * d].reshape(tokens, nkv, d)))
    want_v = x[:, (nq + nkv) * d:]
    if mixed:
        want_v = 0.7 * want_v + 0.3 * d64(other)
    want_v = want_v.reshape(tokens, nkv, dv)
    got_q = d64(q).view(tokens, nq, pad)
    assert float((got_q[..., :d] - want_q).abs().max()) <= _tol(dtype) * 4 and float(got_q[..., d:].abs().sum()) == 0.0
    for t in range(tokens):
        cell = d64(pages[[3, 0, 5][t // page], :, :, t % page])
        assert float((cell[0, :, :d] - want_k[t]).abs().max()) <= _tol(dtype) * 4
        assert float((cell[1, :, :dv] - want_v[t]).abs().max()) <= _tol(dtype) * 4
        assert float(cell[0, :, d:].abs().sum() + cell[1, :, dv:].abs().sum()) == 0.0
    assert float(pages[1].float().mean()) == 7.0                                       # a page of nobody's


def _fake_step(starts_and_lengths, page, nkv, d, dtype, window, keep, gen):
    """A step over requests whose keys lie in scattered pages, the pages behind the window poisoned and taken out of the
    block table: (context, cache view, keys and values per request)."""
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
        first = max(0, start - window + 1) // page if window else 0
        for lp in range(per[r]):
            phys = order.pop()
            if lp >= first or lp * page < keep:
                table[r, lp] = phys
                part = kv[:, :, lp * page:(lp + 1) * page]
                pages[phys, :, :, :part.shape[2]] = part.to(DEV)
    view = View()
    view.pages, view.block_table = pages, table.to(DEV)
    entries = [StepEntry(f"u{r}", [0] * n, s, [0]) for r, (s, n) in enumerate(starts_and_lengths)]
    from lockstep_b200 import kernels as K

    err = K.new_error_word(DEV)
    ctx = StepContext(entries, list(range(len(per))), torch.device(DEV), err, K.attention_split_size())
    return ctx, view, keys, err


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("page", [8, 16, 64])
@pytest.mark.parametrize("nq, nkv, d", [(4, 2, 64), (2, 2, 128), (3, 1, 48)])
@pytest.mark.parametrize("window, keep, cap", [(20, 5, 4.0), (100, 1, 0.0), (130, 300, 9.0), (300, 33, 2.0), (7, 64, 0.0), (64, 0, 3.0)])
def test_attention_with_kept_first_positions(dtype, page, nq, nkv, d, window, keep, cap):
    """Portions and single tokens at the start, just past a window and far past it, against the plain softmax; what lies
    between the kept positions and the window is poison."""
    from lockstep_b200 import kernels as K
    from lockstep_b200.parts.attention import ScoreExtras, attend
    from lockstep_b200.parts.base import Runtime

    gen = torch.Generator().manual_seed(window * 7 + keep + d)
    work = [(0, 40), (window - 3, 9), (700, 130), (431, 2), (0, 1), (window, 1), (999, 1), (keep + window - 1, 1), (255, 1), (640, 1)]
    ctx, view, keys, err = _fake_step(work, page, nkv, d, dtype, window, keep, gen)
    tokens = ctx.num_tokens
    q = torch.randn(tokens, nq * d, generator=gen).to(dtype).to(DEV)
    rt = Runtime(device=torch.device(DEV), dtype=dtype, page_size=page, max_positions=2048, err=err)
    before = K.kernel_counts()
    out = attend(rt, q, ctx, view, nq, nkv, d, (window, keep) if keep else window, 0.3, dtype == F32, ScoreExtras(softcap=cap))
    K.raise_on_fault(err)
    after = K.kernel_counts()
    ran = {k for k in after if after[k] > before.get(k, 0) and k.startswith("attention")}
    on_tensor_cores = dtype == BF16 and d in (64, 128)
    assert ({"attention_prefill_tc", "attention_decode_mma"} <= ran) == on_tensor_cores, ran
    at = 0
    for (start, n), kv in zip(work, keys):
        k, v = d64(kv[0]).transpose(0, 1), d64(kv[1]).transpose(0, 1)                  # [keys, nkv, d]
        total = start + n
        qq = torch.zeros(total, nq, d, dtype=torch.float64)
        qq[start:] = d64(q[at:at + n]).view(n, nq, d)
        want = plain.softmax_attention(qq, k, v, 0.3, plain.visible(total, window, keep), cap or None)[start:]
        got = d64(out[at:at + n]).view(n, nq, d)
        assert float((got - want).abs().max()) <= (2e-5 if dtype == F32 else 3e-2), (start, n)
        at += n


def test_recorded_steps_plan_kept_positions_as_unrecorded_ones_do():
    """The work list a recorded decode step fills in equals the one made from scratch."""
    from lockstep_b200 import kernels as K
    from lockstep_b200.engine.batch import StepEntry, plan_attention
    from lockstep_b200.engine.graphs import StaticStepContext, split_items

    masks = [0, 40, (40, 5), (300, 600), (20, 257)]
    starts = [0, 39, 40, 255, 256, 300, 900, 1300, 555, 1023]
    entries = [StepEntry(f"u{i}", [1], s, [0]) for i, s in enumerate(starts)]
    capacity = split_items(entries, masks, 256)
    ctx = StaticStepContext(16, capacity, masks, torch.device(DEV), K.new_error_word(DEV), 256, pad_slot=12)
    ctx.fill(entries, list(range(10)))
    torch.cuda.synchronize()
    for mask in masks:
        _, split, combine, n = plan_attention([(i, i, s, 1) for i, s in enumerate(starts)], mask, 256)
        plan = ctx.attention_plan(mask)
        assert torch.equal(plan.split_work[:n].cpu(), torch.from_numpy(split)) and int(plan.split_work[n:].abs().sum()) == 0
        assert torch.equal(plan.combine_items[:10].cpu(), torch.from_numpy(combine)) and int(plan.combine_items[10:, 3].sum()) == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads, dk, dv, cap", [(3, 8, 20, 9.0), (2, 24, 16, 3.0), (1, 10, 6, 1.5), (4, 64, 96, 15.0), (2, 40, 33, 30.0),
                                                (1, 256, 64, 12.0), (1, 300, 40, 12.0), (5, 16, 1, 5.0)])
def test_matrix_memory_across_calls(dtype, heads, dk, dv, cap):
    """The rule and its read-out for three requests in portions across calls, against the plain functions on the whole
    sequences; gates so large that the running maximum moves, rows whose denominator is |n . q| and rows where it is e^(-m)."""
    from lockstep_b200 import kernels as K

    torch.manual_seed(heads * dk + dv)
    Kd, Vd = heads * dk, heads * dv
    up = lambda n: -(-n // 8) * 8
    at = {"q": 0, "k": up(Kd), "v": 2 * up(Kd), "g": 2 * up(Kd) + up(Vd)}
    lengths = {1: 41, 3: 6, 0: 11}
    proj = {s: torch.randn(n, at["g"] + up(Vd), device=DEV).to(dtype) for s, n in lengths.items()}
    z = {s: torch.randn(n, 2 * heads, device=DEV) * torch.tensor([4.0, 2.0], device=DEV).repeat_interleave(heads) for s, n in lengths.items()}
    bias = torch.cat([torch.randn(heads), torch.randn(heads) + 2.0]).to(DEV)
    gain = torch.rand(Vd, device=DEV) + 0.5
    want_o, want_y, floors = {}, {}, 0
    for s, n in lengths.items():
        p, zz = d64(proj[s]), d64(z[s]) + d64(bias)
        i, f = cap * torch.tanh(zz[:, :heads] / cap), plain.log_sigmoid(cap * torch.tanh(zz[:, heads:] / cap))
        q, k = (p[:, at[c]:at[c] + Kd].reshape(n, heads, dk) for c in "qk")
        v = p[:, at["v"]:at["v"] + Vd].reshape(n, heads, dv)
        o, (S, nrm, m) = plain.mlstm_rule(q * dk ** -0.5, k, v, i, f)
        want_o[s] = (o, S, nrm, m)
        want_y[s] = plain.rms_unit(o, 1e-5).reshape(n, Vd) * d64(gain) * torch.sigmoid(p[:, at["g"]:at["g"] + Vd])
    state = torch.zeros(5, heads * (dk + 1) * (dv + 1), device=DEV)
    err = K.new_error_word(DEV)
    got_o, got_y = {s: [] for s in lengths}, {s: [] for s in lengths}
    cuts = ({1: (0, 17), 3: (0, 1), 0: (0, 2)}, {1: (17, 18), 0: (2, 11)}, {1: (18, 41), 3: (1, 6)})
    for cut in cuts:
        rows = torch.cat([proj[s][a:b] for s, (a, b) in cut.items()]).contiguous()
        gates = torch.cat([z[s][a:b] for s, (a, b) in cut.items()]).contiguous()
        slots = torch.tensor([s for s, (a, b) in cut.items() for _ in range(b - a)], dtype=torch.int32, device=DEV)
        n = rows.shape[0]
        portions = torch.empty(1 + 3 * 4, dtype=torch.int32, device=DEV)
        K.find_portions(slots, portions, 4, err)
        o = torch.empty(n, heads * (dv + 2), device=DEV)
        K.state_rule(K.RULE_MLSTM, dtype, portions, 4, state, *(rows[:, at[c]:at[c] + (Vd if c == "v" else Kd)] for c in "qkv"),
                     gates, None, None, o, None, 0, 0, heads, heads, dk, dv, out_scale=dk ** -0.5, gate_bias=bias, gate_cap=cap)
        y = torch.empty(n, Vd, dtype=dtype, device=DEV)
        K.head_rms_gate(o, gain, None, rows[:, at["g"]:at["g"] + Vd], y, heads, dv, False, 1e-5, gate_logit=True, normalized=True)
        first = 0
        for s, (a, b) in cut.items():
            got_o[s].append(d64(o[first:first + b - a]).view(-1, heads, dv + 2))
            got_y[s].append(d64(y[first:first + b - a]))
            first += b - a
    K.raise_on_fault(err)
    for s in lengths:
        o, S, nrm, m = want_o[s]
        g = torch.cat(got_o[s])
        floors += int((g[..., dv].abs() < g[..., dv + 1]).sum())
        den = torch.maximum(g[..., dv].abs(), g[..., dv + 1]) + 1e-6
        # (relative to a read-out's own size: where n . q cancels the quotient is large)
        size = 1 + (g[..., :dv].abs().amax(-1) / den)
        assert float(((g[..., :dv] / den[..., None] - o).abs().amax(-1) / size / (1 + 1 / den)).max()) <= 3e-5, s
        assert float((torch.cat(got_y[s]) - want_y[s]).abs().max()) <= (1e-3 if dtype == F32 else 3e-2) * (1 + float(want_y[s].abs().max())), s
        kept = d64(state[s]).view(heads, dk + 1, dv + 1)
        assert float((kept[:, :dk, :dv] - S).abs().max()) <= 3e-5 * (1 + float(S.abs().max()))
        assert float((kept[:, :dk, dv] - nrm).abs().max()) <= 3e-5 * (1 + float(nrm.abs().max()))
        assert float((kept[:, dk, :] - m[:, None]).abs().max()) <= 1e-5 * (1 + float(m.abs().max()))
    total = sum(lengths.values()) * heads
    assert 0 < floors < total                                        # both kinds of denominator
    assert float(state[2].abs().max()) == 0.0 and float(state[4].abs().max()) == 0.0     # slots nobody used


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads, groups, dk, dv, taps", [(4, 2, 16, 24, 3), (3, 3, 12, 10, 1), (2, 1, 6, 14, 9), (6, 2, 64, 32, 4),
                                                         (2, 2, 128, 128, 2), (1, 1, 256, 40, 16)])
def test_delta_rule_with_one_decay_per_head_across_calls(dtype, heads, groups, dk, dv, taps):
    from lockstep_b200 import kernels as K

    torch.manual_seed(heads * dk + taps)
    Kd, Vd = groups * dk, heads * dv
    C = 2 * Kd + Vd
    lengths = {2: 37, 0: 12, 1: 5}
    proj = {s: torch.randn(n, C + 5, device=DEV).to(dtype) for s, n in lengths.items()}
    z = {s: torch.randn(n, 2 * heads, device=DEV) for s, n in lengths.items()}
    conv = (torch.randn(C, taps, device=DEV) * 0.5).contiguous()
    dt, a_log = torch.randn(heads, device=DEV) - 1, torch.randn(heads, device=DEV) * 0.5 - 2
    want = {}
    for s, n in lengths.items():
        c = plain.silu(plain.causal_conv(d64(proj[s])[:, :C], d64(conv)))
        unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
        q = unit(c[:, :Kd].reshape(n, groups, dk)) * dk ** -0.5
        k = unit(c[:, Kd:2 * Kd].reshape(n, groups, dk))
        g = torch.exp(-torch.exp(d64(a_log)) * plain.softplus(d64(z[s])[:, heads:] + d64(dt)))
        want[s] = plain.delta_rule(q, k, c[:, 2 * Kd:].reshape(n, heads, dv), g, torch.sigmoid(d64(z[s])[:, :heads]))
    state = torch.zeros(4, heads * dk * dv + (taps - 1) * C, device=DEV)
    err = K.new_error_word(DEV)
    got = {s: [] for s in lengths}
    for cut in ({2: (0, 9), 0: (0, 1), 1: (0, 2)}, {2: (9, 10), 0: (1, 3)}, {2: (10, 37), 0: (3, 12), 1: (2, 5)}):
        rows = torch.cat([proj[s][a:b] for s, (a, b) in cut.items()]).contiguous()
        gates = torch.cat([z[s][a:b] for s, (a, b) in cut.items()]).contiguous()
        slots = torch.tensor([s for s, (a, b) in cut.items() for _ in range(b - a)], dtype=torch.int32, device=DEV)
        n = rows.shape[0]
        portions = torch.empty(1 + 3 * 4, dtype=torch.int32, device=DEV)
        K.find_portions(slots, portions, 4, err)
        qkv, decay, beta = (torch.empty(n, c, device=DEV) for c in (C, heads, heads))
        K.delta_prep(rows, conv, dt, a_log, state, slots, qkv, decay, beta, heads, groups, dk, dv, taps, 1e-6, gates=gates)
        o = torch.empty(n, Vd, device=DEV)
        K.state_rule(K.RULE_DELTA_HEAD, dtype, portions, 4, state, qkv, None, None, decay, beta, None, o, rows, C, taps - 1,
                     heads, groups, dk, dv)
        at = 0
        for s, (a, b) in cut.items():
            got[s].append(d64(o[at:at + b - a]).view(-1, heads, dv))
            at += b - a
    K.raise_on_fault(err)
    for s in lengths:
        o, S = want[s]
        assert float((torch.cat(got[s]) - o).abs().max()) <= 2e-5 * (1 + float(o.abs().max())), s
        kept = d64(state[s, :heads * dk * dv]).view(heads, dk, dv)
        assert float((kept - S).abs().max()) <= 2e-5 * (1 + float(S.abs().max())), s
    assert float(state[3].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("tokens, width, dim", [(7, 72, 12), (40, 128, 40), (300, 256, 32), (3, 52, 5), (8, 1024, 128), (33, 1024, 256)])
def test_token_input(dtype, tokens, width, dim):
    """The part alone: the second of three layers' columns of a shared table."""
    from lockstep_b200 import kernels as K
    from lockstep_b200.config import PartSpec
    from lockstep_b200.parts import Runtime, build_part

    torch.manual_seed(tokens + width)
    err = K.new_error_word(DEV)
    rt = Runtime(device=torch.device(DEV), dtype=dtype, page_size=8, max_positions=8, err=err)
    table = build_part("table", PartSpec("token_table", {"vocab_size": 50, "columns": 3 * dim, "tensor": "t"}), rt)
    rt.shared["rows"] = table
    part = build_part("side", PartSpec("token_input", {"hidden_size": width, "dim": dim, "at": dim, "table": "rows",
                                                       "norm_eps": 1e-5}), rt)
    w = {"side.embed": torch.randn(50, 3 * dim), "l1.side.gate": torch.randn(dim, width) * width ** -0.5,
         "l1.side.proj": torch.randn(width, dim) * dim ** -0.5, "l1.side.norm": torch.rand(width) + 0.5}
    w = {k: v.to(dtype) for k, v in w.items()}
    table.bind({"t": w["side.embed"].to(DEV)})
    part.bind({k.split(".")[-1]: v.to(DEV) for k, v in w.items() if k.startswith("l1")})

    class Ctx:
        pass

    ctx = Ctx()
    ids = H.random_tokens(tokens, 50, 3)
    ctx.token_ids = torch.tensor(ids, dtype=torch.int32, device=DEV)
    h = torch.randn(tokens, width, device=DEV) * 2
    x = d64(h)
    before = K.kernel_counts()
    part.forward(h, ctx)
    K.raise_on_fault(err)
    want = x + plain.token_side(x, ids, {k: d64(v) for k, v in w.items()}, 1, dim, 1e-5)
    assert float((d64(h) - want).abs().max()) <= _tol(dtype) * (1 + float(want.abs().max()))
    few = K.kernel_counts()["side_gate_few"] - before["side_gate_few"]
    assert few == (1 if dtype == BF16 and tokens <= K.FEW_TOKENS and width % 8 == 0 else 0)


# ---------------------------------------------------------------------------
# one-layer models: every mechanism in the engine, in every cutting
# ---------------------------------------------------------------------------

SMALL = {
    "attention": [M.bare(M.attention(4, 2, 24, 16, window=20, keep=3, rot=8, scaling=(4.0, 1.0, 3.0, 64)))],
    "attention_heads_of_20": [M.bare(M.attention(2, 2, 20, 12, window=9, keep=9, rot=20, v_mix=False))],
    "attention_no_window": [M.bare(M.attention(3, 1, 16, 32, softcap=None))],
    "attention_window_of_one_page": [M.bare(M.attention(2, 1, 32, 32, window=8, keep=8, rot=16, v_mix=False))],
    "mixed_values": [M.bare(M.attention(4, 2, 16, 16, window=30, keep=2, rot=16)), M.bare(M.mlstm(1, 8, 8)),
                     M.bare(M.attention(2, 2, 32, 16)), M.bare(M.attention(6, 2, 10, 16, window=11))],
    "mlstm": [M.bare(M.mlstm(3, 8, 24, cap=6.0))],
    "delta": [M.bare(M.delta(4, 2, 8, 24, 4))],
    "dense": [M.dense(M.delta(1, 1, 16, 16, 2), 40)],
    "experts": [M.moe(M.mlstm(1, 16, 16), 6, 2, 24, 0.5)],
    "experts_all": [M.moe(M.delta(1, 1, 16, 16, 3), 3, 3, 8, 2.0)],
}
SMALL_KW = {"mlstm": {"side": None}, "experts": {"side": 5}, "attention_no_window": {"side": 48}}


@pytest.fixture(scope="module")
def zoo(tmp_path_factory):
    cache = {}

    def get(config, dtype, lengths, seed=7, edit=None, key=None):
        key = (key or json.dumps(config, sort_keys=True), dtype, tuple(lengths))
        if key not in cache:
            folder = M.make_folder(tmp_path_factory.mktemp("kusolorn"), config, seed=seed, dtype=dtype, edit=edit)
            requests, want = {}, {}
            for i, n in enumerate(lengths):
                # no request rests on a router's close call: another draw of tokens where float32 would decide one
                for draw in range(20):
                    tokens = H.random_tokens(n, config["vocab"], seed=50 + i + 1000 * draw)
                    logits, gap = M.plain_logits_and_gap(folder, tokens)
                    if gap > 1e-3:
                        break
                requests[f"r{i}"], want[f"r{i}"] = tokens, logits.float()
            cache[key] = (folder, requests, want)
        return cache[key]

    return get


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SMALL))
def test_small_models_in_every_cutting(zoo, name, dtype):
    folder, requests, want = zoo(M.layers_model(SMALL[name], **SMALL_KW.get(name, {})), dtype, [45, 130, 9, 77])
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
    """Larger models of sizes nobody chose (see ``kusolorn_models.random_config``) in float32: four requests of up to 330
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
    assert k == len(runner.spec.schedule) == 5


# ---------------------------------------------------------------------------
# weights that make a fault show
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window, keep, dim, vdim", [(37, 5, 16, 16), (64, 8, 64, 64), (200, 12, 64, 64), (30, 20, 48, 96)])
def test_sharp_softmax_at_the_edges_of_windows_and_kept_positions(zoo, window, keep, dim, vdim, dtype):
    """Scores so large that every row's softmax is a choice of one key: rows whose key is the window's first, rows whose key
    is the last kept position hundreds of tokens back; a model with one position more or less at either edge gives other
    logits.  Freed pages are poisoned."""
    from safetensors.torch import load_file

    from lockstep_b200 import kernels as K

    # (q and k have length sqrt(dim): the scale makes the scores)
    config = M.layers_model([M.bare(M.attention(2, 1, dim, vdim, window=window, keep=keep, rot=dim // 2, softcap=60.0,
                                                scale=60.0 / dim, v_mix=False))], width=64, side=None)
    folder, requests, want = zoo(config, dtype, [520, 75], key=f"sharp-{window}-{keep}-{dim}")
    w = {k: v.double() for k, v in load_file(str(folder / "model.safetensors")).items()}
    m = config["layers"][0]["mixer"]
    x = plain.rms_norm(w["embed"][torch.tensor(requests["r0"])], w["l0.norm1"], 1e-5)
    pr, _ = plain.attention_mixer(x, w, "l0.mix", m, 1e-5, weights=True)
    best, sure = pr.argmax(-1), pr.max(-1).values > 0.4               # [heads, rows]
    rows = torch.arange(520)[None]
    past = rows >= window + keep
    assert int((sure & past & (best == rows - window + 1)).sum()) >= 1        # the window's first key
    assert int((sure & past & (best < keep)).sum()) >= 5                      # a kept position behind the window
    assert int((sure & past & (best == keep - 1)).sum()) >= 1                 # the last of them
    for change in ({"size": window - 1}, {"size": window + 1}, {"keep_first": keep - 1}, {"keep_first": keep + 1}, {"keep_first": 0}):
        other = M.plain_logits(folder, requests["r0"], edit=lambda c: c["layers"][0]["mixer"]["mask"].update(change))
        assert float((other.float() - want["r0"]).abs().max()) > 0.3, change
    before = K.kernel_counts()
    for plan_name, plan in PLANS.items():
        steps = plan(requests)
        runner = make_runner(folder, dtype, 8, steps, poison_freed_pages=True)
        M.assert_close(H.run_plan(runner, steps), want, dtype, f"sharp window of {window} with {keep}, {plan_name}", 0.0,
                       slack=1.0 if dtype == "float32" else 2.0)
    after = K.kernel_counts()
    for kernel in ("attention_prefill_tc", "attention_decode_mma"):
        ran = after.get(kernel, 0) - before.get(kernel, 0)
        assert (ran > 0) == (dtype == "bfloat16" and dim == 64), kernel


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [32, 64])
def test_sharp_attention_without_a_window_reaches_far_keys(zoo, dim, dtype):
    from safetensors.torch import load_file

    config = M.layers_model([M.bare(M.attention(4, 2, dim, 32, rot=dim, base=1e6, scaling=(8.0, 1.0, 4.0, 64), softcap=30.0,
                                                scale=40.0 / dim, v_mix=False))], width=64, side=None)
    folder, requests, want = zoo(config, dtype, [500, 61], key=f"far-{dim}")
    w = {k: v.double() for k, v in load_file(str(folder / "model.safetensors")).items()}
    x = plain.rms_norm(w["embed"][torch.tensor(requests["r0"])], w["l0.norm1"], 1e-5)
    pr, _ = plain.attention_mixer(x, w, "l0.mix", config["layers"][0]["mixer"], 1e-5, weights=True)
    far = (torch.arange(500)[None] - pr.argmax(-1) > 200) & (pr.max(-1).values > 0.3)
    assert int(far.sum()) >= 3
    for change in (lambda m: m.pop("softcap"), lambda m: m["rot"].pop("scaling")):
        other = M.plain_logits(folder, requests["r0"], edit=lambda c: change(c["layers"][0]["mixer"]))
        assert float((other.float() - want["r0"]).abs().max()) > 0.3
    for plan_name, plan in PLANS.items():
        steps = plan(requests)
        runner = make_runner(folder, dtype, 16, steps)
        M.assert_close(H.run_plan(runner, steps), want, dtype, f"far keys, {plan_name}", 0.0,
                       slack=1.0 if dtype == "float32" else 2.0)


def _remember(tensors):
    for name in tensors:
        if name.endswith(".f.b"):
            tensors[name] = torch.full_like(tensors[name], 8.0)
        if name.endswith(".i"):
            tensors[name] = tensors[name] * 0.2
        if name.endswith(".A_log"):
            tensors[name] = torch.full_like(tensors[name], -8.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slow_decays_carry_the_first_tokens_through_long_decoding(zoo, dtype):
    """Forget gates and decays near one: the first token still moves the last logits after 260 tokens, 200 of them decoded
    one by one."""
    config = M.layers_model([M.bare(M.mlstm(2, 16, 16, cap=10.0)), M.bare(M.delta(2, 1, 32, 16, 3))], side=None)
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


def test_generation_reuses_a_prefix_beside_kept_positions(tmp_path):
    """Attention layers alone: the next turn of a conversation adopts the pages of the first, the kept first positions
    among them, and generates what a request without reuse does."""
    from lockstep_b200 import Engine, Request

    config = M.layers_model([M.dense(M.attention(2, 1, 32, 32, window=24, keep=5, rot=16), 40),
                             M.bare(M.attention(2, 1, 16, 32, window=24, keep=5))], width=64)
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
