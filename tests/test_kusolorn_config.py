"""Kusolorn without a device: the configuration and its errors, names and shapes of the tensors, the stretched rotation,
cache needs and the pages of first positions that stay visible, the attention plans around them, the plain
implementation's own properties."""

from __future__ import annotations

import copy

import pytest
import torch

import kusolorn_models as M
from plain import kusolorn_plain as plain

from lockstep_b200.cache import CacheManager, PrefixIndex
from lockstep_b200.config import ConfigError, PartSpec, config_from_dict
from lockstep_b200.engine.batch import kept_splits, mask_parts, plan_attention
from lockstep_b200.engine.model import Model, expected_weights
from lockstep_b200.parts import CacheNeed, Runtime, build_part


def _runtime(positions=64):
    return Runtime(device=torch.device("cpu"), dtype=torch.float32, page_size=16, max_positions=positions,
                   err=torch.zeros(2, dtype=torch.int32))


def _model(config):
    return Model(config_from_dict(config).model_spec(), _runtime())


def test_names_and_shapes():
    w = expected_weights(config_from_dict(M.MODEL_S).model_spec())
    assert w["embed"].shape == (193, 72) and w["head"].shape == (193, 72) and w["side.embed"].shape == (193, 5 * 12)
    assert w["l0.mix.k"].shape == (32, 72) and w["l0.mix.v.conv"].shape == (96, 3) and w["l0.mix.a"].shape == (4, 72)
    assert w["l0.mix.dt_bias"].shape == (4,) and w["l0.mix.norm"].shape == (24,) and w["l0.mix.g"].shape == (96, 72)
    assert w["l0.mlp.up"].shape == (56, 72) and "l0.mlp.gate" not in w
    assert w["l1.mix.v"].shape == (120, 72) and "l1.mix.q.norm" not in w and w["l1.mlp.e4.down"].shape == (72, 24)
    assert "l1.mix.vmix" not in w and w["l3.mix.vmix"].shape == ()              # the first mixing layer has nothing to mix in
    assert w["l2.mix.i.b"].shape == (2,) and w["l2.mix.norm"].shape == (32,) and "l2.norm2" not in w and "l2.mlp.up" not in w
    assert w["l4.side.gate"].shape == (12, 72) and w["l4.side.proj"].shape == (72, 12) and w["l4.side.norm"].shape == (72,)
    assert config_from_dict(M.MODEL_S).model_spec().optional_tensors == ("l1.mix.vmix", "l2.norm2")
    u = expected_weights(config_from_dict(M.MODEL_U).model_spec())
    assert not any("side" in name for name in u)
    t = config_from_dict(M.MODEL_T).model_spec()
    assert [l.mixer.get("value_mix") for l in t.layers] == [None, None, "first", None, "later"]


def test_cache_needs_in_the_manager():
    needs = _model(M.MODEL_S).cache_needs()
    assert needs[0].kind == "state" and needs[0].state_shape == (4 * 16 * 24 + 2 * (64 + 96),)
    assert (needs[1].window, needs[1].keep_first, needs[1].head_dim) == (20, 3, 48)
    assert needs[2].state_shape == (2 * 25 * 17,)                               # S, n as a column and m as a row
    cm = CacheManager(needs, num_pages=8, page_size=16, max_live=2, max_seq_len=64, allocate=False)
    assert len(cm.paged) == 2 and len(cm.states) == 3


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "high"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "mixes in"),
    (lambda c: c["layers"][2]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["token_side"].update(dim=0), "dim"),
    (lambda c: c["norm"].update(eps=0), "eps"),
])
def test_configuration_errors(change, message):
    cfg = copy.deepcopy(M.MODEL_S)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(cfg)


@pytest.mark.parametrize("dims, base, scaling", [(8, 500.0, (4.0, 1.0, 3.0, 64)), (64, 1e6, (8.0, 1.0, 4.0, 1024)),
                                                 (32, 1e4, (2.0, 0.5, 8.0, 256)), (12, 77.0, None)])
def test_stretched_frequencies(dims, base, scaling):
    names = ("factor", "low", "high", "original")
    raw = dict(zip(names, scaling)) if scaling else None
    part = build_part("position", PartSpec("scaled_rotary", {
        "dim": dims, "theta": base, "interleaved": True, "scaling": {"kind": "wavelength", **raw} if raw else None}),
        _runtime(300))
    cos, sin, rot_dim = part.rotary()
    freq = plain.rotation_frequencies(dims, base, raw)
    ang = torch.arange(300, dtype=torch.float64)[:, None] * freq[None]
    assert rot_dim == dims and part.rotary_interleaved
    assert torch.allclose(cos.double(), ang.cos(), atol=1e-6) and torch.allclose(sin.double(), ang.sin(), atol=1e-6)
    if scaling:
        own = plain.rotation_frequencies(dims, base)
        ratio = freq / own                                            # some kept, some divided, some in between
        assert bool((ratio > 1 - 1e-12).any()) and bool((ratio < 1 / scaling[0] + 1e-12).any())


def test_plans_with_kept_first_positions():
    assert mask_parts(7) == (7, 0) and mask_parts((7, 3)) == (7, 3)
    # the window lies in the kept positions' split, or just past it, or far past it
    assert [kept_splits(p, (20, 5), 256) for p in (3, 100, 275, 276, 2000)] == [0, 0, 1, 1, 1]
    assert kept_splits(2000, (20, 300), 256) == 2 and kept_splits(600, (300, 300), 256) == 1 and kept_splits(900, 20, 256) == 0
    _, split, combine, slots = plan_attention([(1, 0, 2000, 1), (2, 1, 100, 1)], (20, 5), 256)
    assert split[:, 4].tolist() == [0, 7, 0] and combine[:, 3].tolist() == [2, 1] and slots == 3
    tile, _, _, _ = plan_attention([(0, 0, 1000, 33)], (20, 300), 256)
    assert sorted(map(tuple, tile[:, [2, 3, 4, 5, 7]].tolist())) == [(1, 1032, 3, 5, 2), (16, 1000, 3, 4, 2), (16, 1016, 3, 5, 2)]


def test_the_cache_keeps_the_first_pages_behind_a_window():
    need = CacheNeed("paged_kv", kv_heads=1, head_dim=16, window=20, keep_first=11)
    cm = CacheManager([need], num_pages=12, page_size=8, max_live=2, max_seq_len=400, allocate=False)
    group = cm.paged[0]
    cm.create("a")
    for n in range(1, 201):
        cm.reserve("a", n)
        cm.advance("a", n)
        pages = group.seqs["a"].pages
        held = [i for i, p in enumerate(pages) if p >= 0]
        first = max(0, n - 20 + 1) // 8
        assert held == sorted(set(range(min(2, len(pages)))) | set(range(first, len(pages)))), n
        assert len(held) <= cm.peak_pages(200, 1)
        cm.audit()
    cm.release("a")
    assert group.allocator.free_pages == 12
    # a reader of another layer's keys asks for more of the first ones, and for a longer window
    wide = CacheNeed("paged_kv", kv_heads=1, head_dim=16, window=30, keep_first=2)
    assert (need.widened(wide).window, need.widened(wide).keep_first) == (30, 11)
    assert need.widened(CacheNeed("paged_kv", kv_heads=1, head_dim=16)).keep_first == 0       # every key: no window


def test_prefix_reuse_needs_the_first_pages_too():
    need = CacheNeed("paged_kv", kv_heads=1, head_dim=16, window=16, keep_first=5)
    cm = CacheManager([need], num_pages=40, page_size=8, max_live=3, max_seq_len=400, allocate=False)
    cm.keep_boundary_windows()
    index = PrefixIndex(page_size=8)
    tokens = list(range(100))
    cm.create("a")
    cm.reserve("a", 100)
    cm.advance("a", 100)
    index.insert(tokens, cm.paged, "a")
    cm.release("a")
    n, pages = index.lookup(tokens + [7], cm.paged)
    assert n == 96 and pages[0][0] >= 0 and pages[0][1] == -1 and pages[0][10] >= 0 and pages[0][11] >= 0
    cm.create("b")
    cm.paged[0].adopt("b", pages[0])
    cm.lengths["b"] = n
    assert cm.paged[0].table_host[cm.slots["b"], 0] == pages[0][0]
    # without its first page the prefix cannot serve: what is read of it is gone
    for e in index.entries.values():
        if e.pages[0] == pages[0][0]:
            e.pages[0] = -1
            break
    assert index.lookup(tokens + [7], cm.paged)[0] == 0


def test_plain_pieces():
    torch.manual_seed(0)
    f64 = torch.float64
    # masks: positions a query sees
    seen = plain.visible(12, 4, 2)
    assert seen[9].nonzero().view(-1).tolist() == [0, 1, 6, 7, 8, 9] and seen[3].nonzero().view(-1).tolist() == [0, 1, 2, 3]
    assert plain.visible(5)[4].all()
    # rotation of pairs keeps lengths, and the product of two rotated vectors depends on their distance alone
    freq = plain.rotation_frequencies(6, 100.0)
    x = torch.randn(1, 2, 10, dtype=f64).expand(9, 2, 10)
    y = plain.rotate_pairs(x, freq)
    assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1)) and torch.equal(y[..., 6:], x[..., 6:])
    assert torch.allclose((y[7] * y[4]).sum(-1), (y[5] * y[2]).sum(-1)) and torch.equal(y[0], x[0])
    # the matrix memory continues from its state, and a gate's running maximum changes nothing but the scale
    q, k, v = (torch.randn(9, 2, 5, dtype=f64) for _ in range(3))
    i, f = torch.randn(9, 2, dtype=f64) * 4, -torch.rand(9, 2, dtype=f64)
    whole, (S, n, m) = plain.mlstm_rule(q, k, v, i, f)
    _, state = plain.mlstm_rule(q[:4], k[:4], v[:4], i[:4], f[:4])
    rest, _ = plain.mlstm_rule(q[4:], k[4:], v[4:], i[4:], f[4:], state)
    assert torch.allclose(whole[4:], rest, atol=1e-14)
    direct = sum(torch.exp(i[s] + f[s + 1:].sum(0))[:, None, None] * k[s][:, :, None] * v[s][:, None, :] for s in range(9))
    assert torch.allclose(S * torch.exp(m)[:, None, None], direct)
    # the delta rule with beta one writes its value exactly: reading with the key gives the value back
    k1 = torch.nn.functional.normalize(torch.randn(6, 1, 4, dtype=f64), dim=-1)
    v1 = torch.randn(6, 2, 3, dtype=f64)
    o, _ = plain.delta_rule(k1, k1, v1, torch.rand(6, 2, dtype=f64), torch.ones(6, 2, dtype=f64))
    assert torch.allclose(o, v1)
    # the chosen experts' weights sum to one
    z = torch.randn(5, 12, dtype=f64)
    ids, weights = plain.route(z, {"m.router": torch.randn(6, 12, dtype=f64)}, "m", 3)
    assert torch.allclose(weights.sum(-1), torch.ones(5, dtype=f64)) and bool((weights[:, 0] >= weights[:, 2]).all())
