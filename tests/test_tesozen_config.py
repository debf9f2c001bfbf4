"""Tesozen without a device: the configuration and its errors, names and shapes of the tensors, cache needs and the pages
of finished chunks, prefix reuse beside chunks, the order in which layers hand their normed rows on, the plain
implementation's own properties."""

from __future__ import annotations

import copy

import pytest
import torch

import tesozen_models as M
from plain import tesozen_plain as plain

from lockstep_b200.cache import CacheManager, PrefixIndex
from lockstep_b200.config import ConfigError, LayerRun, config_from_dict
from lockstep_b200.engine.model import Model, expected_weights
from lockstep_b200.parts import CacheNeed, Runtime


def _model(config):
    rt = Runtime(device=torch.device("cpu"), dtype=torch.float32, page_size=16, max_positions=64,
                 err=torch.zeros(2, dtype=torch.int32))
    return Model(config_from_dict(config).model_spec(), rt)


def test_names_and_shapes():
    w = expected_weights(config_from_dict(M.MODEL_S).model_spec())
    assert w["embed"].shape == (193, 72) and "head" not in w and w["final.norm"].shape == w["final.norm.b"].shape == (72,)
    assert w["l0.mix.q"].shape == (64, 72) and w["l0.mix.dkv"].shape == (40, 72) and w["l0.mix.dkv.norm"].shape == (40,)
    assert w["l0.mix.uk"].shape == (64, 40) and w["l0.mix.uv"].shape == (96, 40) and w["l0.mix.g"].shape == (96, 72)
    assert w["l0.mlp.up"].shape == (56, 72) and "l0.mlp.gate" not in w and w["l0.norm2b.b"].shape == (72,)
    assert w["l1.mix.q"].shape == (3 * 2 * 24, 72) and w["l1.mix.k"].shape == (3 * 2 * 24, 72) and w["l1.mix.v"].shape == (120, 72)
    assert w["l1.mix.q.norm"].shape == w["l1.mix.lq2"].shape == (24,) and w["l1.mix.g"].shape == (3, 72)
    assert w["l1.mix.o"].shape == (72, 120) and w["l3.mix.k"].shape == (3 * 2 * 12, 72)
    assert w["l1.mlp.router"].shape == (6, 72) and w["l1.mlp.correction"].shape == (6,) and w["l1.mlp.e5.gate"].shape == (24, 72)
    assert w["l1.mlp.shared.down"].shape == (72, 40)
    assert w["l2.mix.i.b"].shape == (2,) and w["l2.mix.norm"].shape == (32,) and "l2.norm2" not in w and "l2.mlp.up" not in w
    assert config_from_dict(M.MODEL_S).model_spec().optional_tensors == ("l2.norm2", "l2.norm2.b", "l2.norm2b", "l2.norm2b.b")
    u = expected_weights(config_from_dict(M.MODEL_U).model_spec())
    assert "l2.mlp.shared.up" not in u and u["l0.mlp.shared.up"].shape == (9, 52)


def test_cache_needs_in_the_manager():
    needs = _model(M.MODEL_S).cache_needs()
    assert (needs[0].kv_heads, needs[0].head_dim, needs[0].window) == (1, 48, 0)              # the latent, padded to 16
    assert (needs[1].kv_heads, needs[1].head_dim, needs[1].window) == (3, 48, -20)            # two maps of 24 in one row
    assert needs[2].state_shape == (2 * 25 * 17,)
    assert (needs[3].kv_heads, needs[3].head_dim, needs[3].window) == (3, 48, -50)            # a value of 40 beside maps of 12
    assert _model(M.MODEL_T).cache_needs()[4].head_dim == 128                                 # both at once: nothing padded
    cm = CacheManager(needs, num_pages=8, page_size=16, max_live=2, max_seq_len=64, allocate=False)
    assert len(cm.paged) == 3 and len(cm.states) == 2


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=2), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][2]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][2]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(scale=0), "scale"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "divide"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][3]["mlp"]["router"]["groups"].update(keep=2), "fewer than top"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["norm"].update(eps=0), "eps"),
])
def test_configuration_errors(change, message):
    cfg = copy.deepcopy(M.MODEL_S)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(cfg)


def test_layers_that_follow_one_another_share_a_kernel():
    """A layer closes with the norm of the one that runs next; not the last, and not where a layer runs twice."""
    from dataclasses import replace

    model = _model(M.MODEL_S)
    assert [b.next_norm is not None for b in model.blocks] == [True, True, True, True, False]
    assert model.blocks[1].next_norm is model.blocks[2].mixer_norm
    spec = config_from_dict(M.MODEL_S).model_spec()
    twice = replace(spec, schedule=(*spec.schedule, LayerRun(layer=1, cache=5)))
    assert all(b.next_norm is None for b in Model(twice, model.rt).blocks)


def test_pages_of_finished_chunks_are_given_back():
    need = CacheNeed("paged_kv", kv_heads=1, head_dim=16, window=-20)
    cm = CacheManager([need], num_pages=12, page_size=8, max_live=2, max_seq_len=400, allocate=False)
    group = cm.paged[0]
    cm.create("a")
    for n in range(1, 201):
        cm.reserve("a", n)
        cm.advance("a", n)
        held = [i for i, p in enumerate(group.seqs["a"].pages) if p >= 0]
        # what the next position, and every later one, reads: from the page of the first key of its chunk on
        assert held == list(range(n // 20 * 20 // 8, len(group.seqs["a"].pages))), n
        assert len(held) <= cm.peak_pages(200, 1)
        cm.audit()
    cm.release("a")
    assert group.allocator.free_pages == 12
    # a layer that reads another's keys: chunks of one size stay, anything else keeps every key
    reader = lambda window: CacheNeed("paged_kv", kv_heads=1, head_dim=16, window=window)
    assert need.widened(reader(-20)).window == -20 and need.widened(None).window == -20
    assert [need.widened(reader(w)).window for w in (-40, 30, 0)] == [0, 0, 0] and reader(30).widened(need).window == 0


def test_prefix_reuse_beside_chunks():
    """What a request that goes on from a whole-page boundary reads of the last chunk is kept; finished chunks need not be there."""
    need = CacheNeed("paged_kv", kv_heads=1, head_dim=16, window=-20)
    cm = CacheManager([need], num_pages=40, page_size=8, max_live=3, max_seq_len=400, allocate=False)
    cm.keep_boundary_windows()
    index = PrefixIndex(page_size=8)
    tokens = list(range(117))
    cm.create("a")
    cm.reserve("a", 117)
    cm.advance("a", 117)
    index.insert(tokens, cm.paged, "a")
    cm.release("a")
    n, pages = index.lookup(tokens + [7], cm.paged)
    # 112 positions: the last boundary; its chunk began at 100, in page 12
    assert n == 112 and [p >= 0 for p in pages[0]] == [False] * 12 + [True] * 2


def test_plain_pieces():
    torch.manual_seed(0)
    f64 = torch.float64
    seen = plain.visible(12, 5)
    assert seen[9].nonzero().view(-1).tolist() == [5, 6, 7, 8, 9] and seen[10].nonzero().view(-1).tolist() == [10]
    assert plain.visible(5)[4].all()
    # with the second map's weight at zero, two equal maps are one attention, up to the norm
    a = torch.randn(6, 2, 8, dtype=f64)
    gate = torch.full((6, 2), 40.0, dtype=f64)
    assert torch.allclose(plain.combine_maps(a, a, 0.0, 0.25, gate, 1e-12), 0.75 * plain.rms_unit(a, 1e-12))
    # a row that is alone in its chunk sees one key: both maps give its value, and any weight below one the same direction
    assert torch.allclose(plain.combine_maps(a, a, 0.6, 0.25, gate, 1e-12), plain.combine_maps(a, a, -3.0, 0.25, gate, 1e-12))
    # the layer norm
    x = torch.randn(4, 9, dtype=f64) * 3 + 1
    y = plain.layer_norm(x, torch.ones(9, dtype=f64), torch.full((9,), 0.5, dtype=f64), 0.0)
    assert torch.allclose(y.mean(-1), torch.full((4,), 0.5, dtype=f64)) and torch.allclose(y.var(-1, unbiased=False), torch.ones(4, dtype=f64))
    # the matrix memory is the sum of its decayed writes, whatever the running maximum does
    q, k, v = (torch.randn(9, 2, 5, dtype=f64) for _ in range(3))
    i, f = torch.randn(9, 2, dtype=f64) * 4, -torch.rand(9, 2, dtype=f64)
    o = plain.mlstm_rule(q, k, v, i, f)
    weight = torch.stack([torch.exp(i[s] + f[s + 1:].sum(0)) for s in range(9)])              # [9, heads]
    score = torch.einsum("shk,hk->sh", k, q[8]) * weight
    want = torch.einsum("sh,shv->hv", score, v) / (torch.maximum(score.sum(0).abs(), torch.ones(2, dtype=f64)))[:, None]
    assert torch.allclose(o[8], want, rtol=1e-4)
    # groups: two middling experts beat one good one; choice scores below zero; weights are shares of the uncorrected scores
    choice = torch.tensor([[-0.2, -2.0, -0.7, -0.8]], dtype=f64)
    assert plain.allowed_experts(choice, {"count": 2, "keep": 1}).tolist() == [[False, False, True, True]]
    logits = torch.tensor([[3.0, -3.0, 0.5, 0.4]], dtype=f64)
    w = {"m.router": torch.eye(4, dtype=f64), "m.correction": torch.tensor([-1.2, -1.2, -1.1, -1.1], dtype=f64)}
    ids, weights = plain.route(logits, w, "m", {"top": 2, "scale": 1.5, "groups": {"count": 2, "keep": 1}})
    s = torch.sigmoid(logits[0])
    assert ids.tolist() == [[2, 3]] and torch.allclose(weights, (1.5 * s[2:] / s[2:].sum())[None])
    assert plain.route(logits, w, "m", {"top": 2, "scale": 1.5})[0].tolist() == [[0, 2]]
