"""Small Kusolorn configurations for the tests, and what the tests share.

The configurations differ from each other in every size and option: heads, key heads (one, some, as many as heads), head
sizes (multiples of 16 and not), rotated parts (whole heads, parts of them, none) with and without stretched frequencies,
windows with many, one and no kept first positions and no window at all, capped scores and not, mixed values in some, all
and none of the attention layers, values smaller and larger than keys, matrix memories of one and several heads, delta
mixers with one to nine taps, dense and routed feed-forwards (one expert, all experts chosen), layers without one, models
with and without the tokens' rows, eps, vocabulary, width (also no multiple of 8), page size.
"""

from __future__ import annotations

import json
from pathlib import Path

import torch


def attention(heads, kv_heads, dim, vdim, window=None, keep=None, rot=None, base=10000.0, scaling=None, scale=None,
              softcap=20.0, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale or dim ** -0.5), "v_mix": v_mix}
    if softcap is not None:
        m["softcap"] = float(softcap)
    if window is not None:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if rot is not None:
        m["rot"] = {"dims": rot, "base": float(base)}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m}


def mlstm(heads, dim, vdim, cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": float(cap)}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def moe(layer, experts, top, ff, limit=1.0):
    return {**layer, "mlp": {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": float(limit)}}}


def bare(layer):
    return {**layer, "mlp": None}


def model(width, vocab, eps, layers, side=12):
    cfg = {"architecture": "Kusolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": list(layers)}
    if side is not None:
        cfg["token_side"] = {"dim": side}
    return cfg


# S: every kind of layer and feed-forward; heads of 16 to 40 elements
MODEL_S = model(72, 193, 1e-5, [
    dense(delta(4, 2, 16, 24, 3), 56),
    moe(attention(3, 3, 16, 40, window=20, keep=3, rot=8, base=500.0, scaling=(4.0, 1.0, 3.0, 64)), 5, 2, 24, 0.7),
    bare(mlstm(2, 24, 16, cap=4.0)),
    moe(attention(6, 3, 32, 40, window=50, keep=17, rot=32, base=1e4, scaling=(2.0, 0.5, 8.0, 256), softcap=5.0), 3, 1, 16),
    dense(mlstm(3, 8, 20), 40),
])
PAGE_S = 16

# T: heads the tensor-core attention takes (64 and 128, the second by padding), sizes the tensor-core products take, forty
# experts; mixing starts in the second attention layer; one layer without a window
MODEL_T = model(128, 211, 3e-6, [
    moe(attention(4, 1, 64, 64, window=90, keep=5, rot=64, base=250000.0, softcap=15.0, v_mix=False), 40, 4, 72, 2.0),
    dense(mlstm(4, 32, 64, cap=12.0), 256),
    dense(attention(6, 2, 112, 128, window=200, keep=1, rot=40, base=1e6, scaling=(8.0, 1.0, 4.0, 512)), 128),
    moe(delta(6, 3, 32, 32, 5), 6, 6, 40, 0.5),
    dense(attention(2, 2, 64, 128, rot=16, softcap=None), 72),
], side=40)
PAGE_T = 8

# U: odd sizes everywhere: a width and a vocabulary that are no multiples of 8, heads of 6 to 14 elements, one expert, one
# tap and nine, no rotation, a window without kept positions, no rows of the tokens' own
MODEL_U = model(52, 101, 2e-6, [
    moe(mlstm(1, 10, 6, cap=1.5), 1, 1, 27, 3.0),
    dense(attention(3, 1, 10, 6, window=7, rot=6, base=77.0, softcap=2.0), 30),
    moe(delta(3, 3, 12, 10, 1), 7, 7, 10, 0.4),
    bare(attention(2, 1, 14, 6, window=30, keep=30, softcap=50.0)),
    bare(delta(2, 1, 6, 14, 9)),
], side=None)
PAGE_U = 32

MODELS = {"S": (MODEL_S, PAGE_S), "T": (MODEL_T, PAGE_T), "U": (MODEL_U, PAGE_U)}


def layers_model(layers, width=48, vocab=97, eps=1e-5, **kw):
    return model(width, vocab, eps, list(layers), **kw)


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: widths of 128 to 512, three to seven layers of any kind in any order, heads of 32
    to 128 elements on one to four key heads, windows of 48 to 384 with up to 40 kept positions, two to five taps, any
    feed-forward."""
    import random

    r = random.Random(seed)
    width, vocab = r.choice([128, 160, 256, 320, 384, 512]), r.choice([257, 384, 500, 512, 1000])
    layers, values = [], None
    for _ in range(r.choice([3, 4, 5, 6, 7])):
        kind = r.random()
        if kind < 0.4:
            kv, vdim = values or (r.choice([1, 2, 4]), r.choice([32, 64, 96]))
            values = (kv, vdim)
            dim = r.choice([32, 48, 64, 96, 128])
            layer = attention(kv * r.choice([1, 2, 4]), kv, dim, vdim, window=r.choice([48, 64, 100, 128, 384]),
                              keep=r.choice([1, 2, 8, 40]), rot=r.choice([dim, dim // 2, 16]), base=r.choice([1e4, 1e6, 2e5]),
                              scaling=r.choice([None, (4.0, 1.0, 4.0, 128), (8.0, 1.0, 4.0, 1024)]),
                              scale=r.choice([dim ** -0.5, 0.1, 0.2]), softcap=r.choice([10.0, 40.0]), v_mix=r.random() < 0.8)
        elif kind < 0.7:
            layer = mlstm(r.choice([2, 3, 4, 6]), r.choice([16, 32, 64]), r.choice([32, 64, 80]), cap=r.choice([8.0, 15.0, 30.0]))
        else:
            kv = r.choice([1, 2, 3])
            layer = delta(kv * r.choice([1, 2, 3]), kv, r.choice([16, 32, 64]), r.choice([32, 64]), r.choice([2, 3, 4, 5]))
        kind = r.random()
        if kind < 0.15:
            layers.append(bare(layer))
        elif kind < 0.5:
            layers.append(dense(layer, r.choice([128, 256, 384])))
        else:
            experts = r.choice([4, 8, 12])
            layers.append(moe(layer, experts, r.choice([1, 2, 3]), r.choice([32, 64, 96]), r.choice([0.8, 2.0, 7.0])))
    return model(width, vocab, r.choice([1e-6, 1e-5]), layers, side=r.choice([16, 32, 40]))


INIT_STD = 0.15


def make_folder(tmp_path, config, seed: int, dtype: str, init_std: float = INIT_STD, edit=None) -> Path:
    """A model folder of random weights; ``edit(tensors)`` may change them before they are written (a test that
    needs weights which make a fault show)."""
    from safetensors.torch import save_file

    from lockstep_b200.config import config_from_dict
    from lockstep_b200.engine.model import expected_weights
    from lockstep_b200.weights.random_init import random_tensors

    folder = Path(tmp_path) / f"kusolorn-{seed}-{dtype}"
    folder.mkdir(parents=True, exist_ok=True)
    cfg = config_from_dict(config)
    tensors = random_tensors(expected_weights(cfg.model_spec()), seed, dtype, init_std, 0.1)
    for name in tensors:
        # routers whose logits lie well apart
        if name.endswith(".router"):
            tensors[name] = (tensors[name].float() * 4.0).to(tensors[name].dtype)
    # a number of the first mixing layer's own, which nothing reads
    tensors.update({name: torch.tensor(0.9).to(next(iter(tensors.values())).dtype)
                    for name in cfg.model_spec().optional_tensors if name.endswith(".vmix")})
    if edit is not None:
        edit(tensors)
    (folder / "config.json").write_text(json.dumps(cfg.to_dict(), indent=1))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder


def plain_logits(folder, tokens, edit=None) -> torch.Tensor:
    from plain import kusolorn_plain as plain

    return plain.model_logits(folder, tokens, torch.float64, edit=edit)


def plain_logits_and_gap(folder, tokens):
    """The plain logits, and the smallest gap between a chosen and a rejected router logit anywhere in the run (inf
    where nothing is routed): where it is tiny, float32 rounding decides a choice, and every later row of the request
    carries the other expert through the recurrent states."""
    from plain import kusolorn_plain as plain

    plain.ROUTING_GAPS = []
    try:
        logits = plain.model_logits(folder, tokens, torch.float64)
        return logits, min(plain.ROUTING_GAPS, default=float("inf"))
    finally:
        plain.ROUTING_GAPS = None


# Error bounds relative to 1 + the request's largest plain logit (float32: the rounding of sums and carried states;
# bfloat16: the rounding of every product's output, a few dozen deep).
TOLERANCE = {"float32": 4e-5, "bfloat16": 8e-2}
# In bfloat16 a router's input carries the rounding of everything before it; where two logits lie closer than that
# the engine and the plain run choose differently, and the row differs by an expert's output, rightly.  Its float32
# run, on requests without a close call, is what holds every row.
CLOSE_CALLS = {"float32": 0.0, "bfloat16": 0.10}


def assert_close(rows, plain_by_uid, dtype, what, close_calls=None, slack=1.0):
    worst, bad = 0.0, []
    for (uid, pos), got in sorted(rows.items()):
        want = plain_by_uid[uid][pos].float()
        err = float((got - want).abs().max()) / (1.0 + float(plain_by_uid[uid].abs().max()))
        worst = max(worst, err)
        if not err <= slack * TOLERANCE[dtype]:
            bad.append((uid, pos, err))
    allowed = int((CLOSE_CALLS[dtype] if close_calls is None else close_calls) * len(rows))
    assert len(bad) <= allowed, (
        f"{what}: {len(bad)} of {len(rows)} rows are off ({allowed} allowed); the first is request {bad[0][0]} "
        f"position {bad[0][1]}: relative error {bad[0][2]:.3e} > {slack * TOLERANCE[dtype]:.1e}")
    return worst
