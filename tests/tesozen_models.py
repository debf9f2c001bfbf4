"""Small Tesozen configurations for the tests, and what the tests share.

The configurations differ from each other in every size and option: heads, key heads (one, some, as many as heads), maps of
5 to 64 elements beside values smaller and larger than a map and than both maps together, chunks of 1 to 300 positions and
none, weights of the second map near and far from one, matrix memories of one and several heads, latents of 10 to 176
elements, dense and routed feed-forwards (one expert, all experts chosen, groups of one expert, one group, every group kept,
no groups) with and without a shared expert of other sizes, layers without a feed-forward, eps, embedding factor, vocabulary,
width (also no multiple of 8), page size.
"""

from __future__ import annotations

import json
from pathlib import Path

import torch


def attention(heads, kv_heads, dim, vdim, chunk=None, scale=None, diff=0.35):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale or dim ** -0.5), "diff": float(diff)}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": m}


def mlstm(heads, dim, vdim, cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": float(cap)}}


def latent(heads, dim, vdim, kv_rank, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": float(scale or dim ** -0.5)}}


def dense(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def moe(layer, experts, top, ff, groups=None, scale=1.0, shared=None):
    """``groups``: (count, keep) or None."""
    router = {"experts": experts, "top": top, "scale": float(scale)}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return {**layer, "mlp": mlp}


def bare(layer):
    return {**layer, "mlp": None}


def model(width, vocab, eps, scale, layers):
    return {"architecture": "Tesozen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": float(scale)},
            "layers": list(layers)}


# S: every kind of layer and feed-forward; maps whose two sub-heads are wider than the value, and narrower
MODEL_S = model(72, 193, 1e-5, 6.5, [
    dense(latent(4, 16, 24, 40), 56),
    moe(attention(3, 3, 24, 40, chunk=20), 6, 2, 24, groups=(3, 2), scale=1.7, shared=40),
    bare(mlstm(2, 24, 16, cap=4.0)),
    moe(attention(6, 3, 12, 40, chunk=50, diff=0.8), 4, 3, 16, groups=(4, 3), scale=0.6, shared=16),
    dense(mlstm(3, 8, 20), 40),
])
PAGE_S = 16

# T: heads and latents the tensor-core attention takes (64 and 128), sizes the tensor-core products take, forty experts
MODEL_T = model(128, 211, 3e-6, 11.0, [
    moe(attention(4, 1, 32, 64, chunk=90), 40, 4, 72, groups=(8, 3), scale=2.5, shared=136),
    dense(mlstm(4, 32, 64, cap=12.0), 256),
    dense(attention(6, 2, 64, 112, chunk=200, diff=0.1), 128),
    moe(latent(5, 24, 32, 64), 6, 6, 40, groups=(2, 2), shared=48),
    dense(attention(2, 2, 64, 128, diff=-0.2), 72),
    bare(latent(3, 40, 64, 128)),
])
PAGE_T = 8

# U: odd sizes everywhere: a width and a vocabulary that are no multiples of 8, maps of 5 and 14 elements, a latent of 10,
# one expert, experts without groups or a shared one, chunks of seven positions, an embedding factor of one
MODEL_U = model(52, 101, 2e-6, 1.0, [
    moe(mlstm(1, 10, 6, cap=1.5), 1, 1, 27, groups=(1, 1), scale=3.0, shared=9),
    dense(attention(3, 1, 5, 6, chunk=7, diff=0.9), 30),
    moe(latent(3, 6, 10, 10), 7, 7, 10),
    bare(attention(2, 1, 14, 6, diff=0.0)),
    bare(attention(4, 2, 8, 30, chunk=1)),
])
PAGE_U = 32

MODELS = {"S": (MODEL_S, PAGE_S), "T": (MODEL_T, PAGE_T), "U": (MODEL_U, PAGE_U)}


def layers_model(layers, width=48, vocab=97, eps=1e-5, scale=5.0):
    return model(width, vocab, eps, scale, list(layers))


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: widths of 128 to 512, three to seven layers of any kind in any order, maps of 16 to
    64 elements on one to four key heads, chunks of 48 to 384, latents of 32 to 192, any feed-forward."""
    import random

    r = random.Random(seed)
    width, vocab = r.choice([128, 160, 256, 352, 384, 512]), r.choice([257, 384, 500, 512, 1000])
    layers = []
    for _ in range(r.choice([3, 4, 5, 6, 7])):
        kind = r.random()
        dim = r.choice([16, 24, 32, 48, 64])
        if kind < 0.4:
            kv = r.choice([1, 2, 4])
            layer = attention(kv * r.choice([1, 2, 3]), kv, dim, r.choice([32, 48, 64, 96]), chunk=r.choice([48, 64, 100, 128, 384]),
                              scale=r.choice([dim ** -0.5, 0.1, 0.2]), diff=r.choice([0.1, 0.3, 0.5, 0.75]))
        elif kind < 0.7:
            layer = mlstm(r.choice([2, 3, 4, 6]), r.choice([16, 32, 64]), r.choice([32, 64, 80]), cap=r.choice([8.0, 15.0, 30.0]))
        else:
            layer = latent(r.choice([2, 3, 4, 8]), dim, r.choice([32, 48, 64]), r.choice([32, 64, 96, 128, 192]))
        kind = r.random()
        if kind < 0.15:
            layers.append(bare(layer))
        elif kind < 0.5:
            layers.append(dense(layer, r.choice([128, 256, 384])))
        else:
            count, size = r.choice([2, 3, 4, 6]), r.choice([2, 3, 4])
            keep = r.choice(range(1, count + 1))
            layers.append(moe(layer, count * size, r.randint(1, min(4, keep * size)), r.choice([32, 64, 96]), (count, keep),
                              r.choice([1.0, 1.5, 2.5]), r.choice([None, 32, 64, 128])))
    return model(width, vocab, r.choice([1e-6, 1e-5]), r.choice([1.0, width ** 0.5]), layers)


INIT_STD = 0.15


def make_folder(tmp_path, config, seed: int, dtype: str, init_std: float = INIT_STD, edit=None) -> Path:
    """A model folder of random weights; ``edit(tensors)`` may change them before they are written (a test that
    needs weights which make a fault show)."""
    from safetensors.torch import save_file

    from lockstep_b200.config import config_from_dict
    from lockstep_b200.engine.model import expected_weights
    from lockstep_b200.weights.random_init import random_tensors

    folder = Path(tmp_path) / f"tesozen-{seed}-{dtype}"
    folder.mkdir(parents=True, exist_ok=True)
    cfg = config_from_dict(config)
    tensors = random_tensors(expected_weights(cfg.model_spec()), seed, dtype, init_std, 0.1)

    def change(name, fn):
        tensors[name] = fn(tensors[name].float()).to(tensors[name].dtype)

    for name in tensors:
        if name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            change(name, lambda t: 3.0 * t)          # the layer's lambda well away from ``diff``
        elif name.endswith(".correction"):
            change(name, lambda t: 8.0 * t - 1.5)    # choice scores below zero
        elif name.endswith(".b") and "norm" in name:
            change(name, lambda t: 10.0 * t)         # biases that show
    if edit is not None:
        edit(tensors)
    (folder / "config.json").write_text(json.dumps(cfg.to_dict(), indent=1))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder


def plain_logits(folder, tokens, edit=None) -> torch.Tensor:
    from plain import tesozen_plain as plain

    return plain.model_logits(folder, tokens, torch.float64, edit=edit)


def plain_logits_and_gap(folder, tokens):
    """The plain logits, and the smallest gap between a chosen and a rejected group or expert anywhere in the run (inf
    where nothing is routed): where it is tiny, float32 rounding decides a choice, and every later row of the request
    carries the other expert through the recurrent states."""
    from plain import tesozen_plain as plain

    plain.ROUTING_GAPS = []
    try:
        logits = plain.model_logits(folder, tokens, torch.float64)
        return logits, min(plain.ROUTING_GAPS, default=float("inf"))
    finally:
        plain.ROUTING_GAPS = None


# Error bounds relative to 1 + the request's largest plain logit (float32: the rounding of sums and carried states;
# bfloat16: the rounding of every product's output, a few dozen deep).
TOLERANCE = {"float32": 4e-5, "bfloat16": 8e-2}
# In bfloat16 a router's input carries the rounding of everything before it; where two choice scores lie closer than that
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
