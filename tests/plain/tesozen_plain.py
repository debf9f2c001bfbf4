"""The Tesozen design written out plainly, one function per mechanism, in float64 by default, whole
sequences at a time and without a cache.  It shares no code with the engine: tests compare the engine's
kernels, cache and step function with it.

Notation: ``x`` [n, width] is a sequence of n tokens at positions 0 .. n-1; linear weights are
[out, in] and applied as ``x @ W.T``; a "mixer" maps the normed residual stream to what is added
to it.  ``w`` is the dictionary of the model's tensors by name, ``p`` a tensor-name prefix.
"""

from __future__ import annotations

import torch


# ---------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------

def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, gain, bias, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * gain + bias


def norm(x, w, p, eps):
    return layer_norm(x, w[p], w[p + ".b"], eps)


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.relu(z) ** 2


def log_sigmoid(z):
    return -torch.logaddexp(-z, torch.zeros_like(z))


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------

def visible(n, chunk=None):
    """[n, n] bool: query i sees key j <= i, in its own run of ``chunk`` positions only where there are chunks."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen if chunk is None else seen & (i // chunk == j // chunk)


def softmax_attention(q, k, v, scale, seen):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; query head h reads key head h // (H / G)."""
    rep = q.shape[1] // k.shape[1]
    kk, vv = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    pr = torch.softmax(s.masked_fill(~seen[None], float("-inf")), dim=-1)
    return torch.einsum("hij,jhd->ihd", pr, vv)


def difference_weight(w, p, diff):
    """The layer's lambda: what the second map's output is multiplied by before it is taken off the first's."""
    return (torch.exp((w[p + ".lq1"] * w[p + ".lk1"]).sum()) - torch.exp((w[p + ".lq2"] * w[p + ".lk2"]).sum()) + diff)


def differential_maps(x, w, p, m, eps):
    """The two maps' outputs, [n, H, vdim] each, before they are combined."""
    n = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit((x @ w[p + ".q"].T).view(n, H, 2, d), eps) * w[p + ".q.norm"]
    k = rms_unit((x @ w[p + ".k"].T).view(n, G, 2, d), eps) * w[p + ".k.norm"]
    v = (x @ w[p + ".v"].T).view(n, G, dv)
    seen = visible(n, (m.get("mask") or {}).get("size"))
    return [softmax_attention(q[:, :, i], k[:, :, i], v, m["scale"], seen) for i in (0, 1)]


def combine_maps(first, second, lam, diff, gate, eps):
    """first, second [n, H, dv], gate [n, H] (logits)."""
    return rms_unit(first - lam * second, eps) * (1.0 - diff) * torch.sigmoid(gate)[..., None]


def attention_mixer(x, w, p, m, eps):
    first, second = differential_maps(x, w, p, m, eps)
    o = combine_maps(first, second, difference_weight(w, p, m["diff"]), m["diff"], x @ w[p + ".g"].T, eps)
    return o.reshape(x.shape[0], -1) @ w[p + ".o"].T


def latent_mixer(x, w, p, m, eps):
    n = x.shape[0]
    H, d, dv, rank = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
    q = (x @ w[p + ".q"].T).view(n, H, d)
    c = rms_unit(x @ w[p + ".dkv"].T, eps) * w[p + ".dkv.norm"]
    k, v = (c @ w[p + ".uk"].T).view(n, H, d), (c @ w[p + ".uv"].T).view(n, H, dv)
    o = softmax_attention(q, k, v, m["scale"], visible(n)).reshape(n, H * dv)
    return (o * torch.sigmoid(x @ w[p + ".g"].T)) @ w[p + ".o"].T


# ---------------------------------------------------------------------------
# the matrix memory
# ---------------------------------------------------------------------------

def mlstm_gates(x, w, p, cap):
    """(log input gate, log forget gate), [n, heads] each."""
    i = cap * torch.tanh((x @ w[p + ".i"].T + w[p + ".i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((x @ w[p + ".f"].T + w[p + ".f.b"]) / cap))
    return i, f


def mlstm_rule(q, k, v, i, f):
    """q, k [n, H, dk] (q scaled), v [n, H, dv], i, f [n, H].  From S = 0, n = 0, m = 0: m_t = max(f + m, i),
    S_t = e^(f + m - m_t) S + e^(i - m_t) k v^T, n_t likewise with k; o = S^T q / (max(|n . q|, e^(-m_t)) + 1e-6)."""
    n_tok, H, dk = q.shape
    S, nrm = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype), torch.zeros(H, dk, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(n_tok):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        nrm = keep[:, None] * nrm + put[:, None] * k[t]
        m = m_new
        den = torch.maximum((nrm * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hkv,hk->hv", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm_mixer(x, w, p, m, eps):
    n = x.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (x @ w[p + ".q"].T).view(n, H, dk) * dk ** -0.5
    k = (x @ w[p + ".k"].T).view(n, H, dk)
    v = (x @ w[p + ".v"].T).view(n, H, dv)
    i, f = mlstm_gates(x, w, p, float(m["gate_cap"]))
    o = rms_unit(mlstm_rule(q, k, v, i, f), eps).reshape(n, H * dv)
    return (o * w[p + ".norm"] * torch.sigmoid(x @ w[p + ".g"].T)) @ w[p + ".o"].T


MIXERS = {"attention": attention_mixer, "mlstm": mlstm_mixer, "latent_attention": latent_mixer}


# ---------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------

# a list here collects, per routed layer, the smallest gap between what was chosen and what was turned away (groups and
# experts): where it is tiny, rounding decides a choice
ROUTING_GAPS = None


def _gap(values, kept):
    """values [n, many] sorted downwards: the smallest distance between the last kept and the first other one."""
    if ROUTING_GAPS is not None and values.shape[1] > kept:
        gap = (values[:, kept - 1] - values[:, kept])
        ROUTING_GAPS.append(float(gap[torch.isfinite(gap)].min()) if torch.isfinite(gap).any() else float("inf"))


def allowed_experts(choice, groups):
    """choice [n, E]: True for the experts of the ``keep`` best of ``count`` equal runs of neighbours, a run's score the
    sum of its two largest choice scores (ties to the lower run)."""
    n, experts = choice.shape
    if not groups:
        return torch.ones_like(choice, dtype=torch.bool)
    by_group = choice.view(n, groups["count"], -1)
    score = torch.sort(by_group, dim=-1, descending=True).values[..., :2].sum(-1)
    ranked = torch.sort(score, dim=-1, descending=True, stable=True)
    _gap(ranked.values, groups["keep"])
    kept = torch.zeros_like(score, dtype=torch.bool).scatter(1, ranked.indices[:, :groups["keep"]], True)
    return kept.repeat_interleave(experts // groups["count"], dim=1)


def route(x, w, p, router):
    """Chosen experts [n, top] (largest choice score first, ties to the lower index) and their weights."""
    s = torch.sigmoid(x @ w[p + ".router"].T)
    choice = s + w[p + ".correction"]
    choice = choice.masked_fill(~allowed_experts(choice, router.get("groups")), float("-inf"))
    ranked = torch.sort(choice, dim=-1, descending=True, stable=True)
    _gap(ranked.values, router["top"])
    ids = ranked.indices[:, :router["top"]]
    chosen = s.gather(1, ids)
    return ids, chosen / (chosen.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def expert(x, w, p):
    return (silu(x @ w[p + ".gate"].T) * (x @ w[p + ".up"].T)) @ w[p + ".down"].T


def feed_forward(x, w, p, f):
    if f["kind"] == "dense":
        return relu_squared(x @ w[p + ".up"].T) @ w[p + ".down"].T
    ids, weights = route(x, w, p, f["router"])
    out = torch.zeros_like(x)
    for e in range(f["router"]["experts"]):
        out = out + expert(x, w, f"{p}.e{e}") * (weights * (ids == e)).sum(-1, keepdim=True)
    return out + expert(x, w, p + ".shared") if f.get("shared") else out


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def forward(tokens, w, cfg, dtype=torch.float64, streams=False):
    """Logits [n, vocab] of the whole sequence (and, with ``streams``, the residual stream after every layer)."""
    w = {k: (t.to(dtype) if t.is_floating_point() else t) for k, t in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)] * cfg["embedding"]["scale"]
    kept = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        y = MIXERS[layer["type"]](norm(x, w, p + ".norm1", eps), w, p + ".mix", layer["mixer"], eps)
        x = x + norm(y, w, p + ".norm1b", eps)
        if layer.get("mlp"):
            x = x + norm(feed_forward(norm(x, w, p + ".norm2", eps), w, p + ".mlp", layer["mlp"]), w, p + ".norm2b", eps)
        kept.append(x)
    logits = norm(x, w, "final.norm", eps) @ w["embed"].T
    return (logits, torch.stack(kept)) if streams else logits


def model_logits(folder, tokens, dtype=torch.float64, edit=None):
    """Logits of the model stored in ``folder`` (config.json, model.safetensors) for the whole sequence.
    ``edit(config)`` may change the configuration first (a test that asks what a mechanism is worth)."""
    import json
    from pathlib import Path

    from safetensors.torch import load_file

    cfg = json.loads((Path(folder) / "config.json").read_text())
    if edit is not None:
        edit(cfg)
    return forward(tokens, load_file(str(Path(folder) / "model.safetensors")), cfg, dtype)
