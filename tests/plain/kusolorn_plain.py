"""The Kusolorn design written out plainly, one function per mechanism, in float64 by default, whole
sequences at a time and without a cache.  It shares no code with the engine: tests compare the engine's
kernels, cache and step function with it.

Notation: ``x`` [n, width] is a sequence of n tokens at positions 0 .. n-1; linear weights are
[out, in] and applied as ``x @ W.T``; a "mixer" maps the normed residual stream to what is added
to it.  ``w`` is the dictionary of the model's tensors by name, ``p`` a tensor-name prefix.
"""

from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------

def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, gain, eps):
    return rms_unit(x, eps) * gain


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def log_sigmoid(z):
    return -softplus(-z)


# ---------------------------------------------------------------------------
# rotation
# ---------------------------------------------------------------------------

def rotation_frequencies(dims, base, scaling=None):
    """f_i = base^(-2i/dims); with ``scaling`` a frequency whose wavelength 2 pi / f is below original / high stays,
    one above original / low is divided by the factor, and between the two it moves linearly in original / wavelength."""
    freq = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling:
        factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
        for i, f in enumerate(freq):
            wavelength = 2.0 * math.pi / f
            if wavelength < original / high:
                continue
            if wavelength > original / low:
                freq[i] = f / factor
            else:
                s = (original / wavelength - low) / (high - low)
                freq[i] = (1.0 - s) * f / factor + s * f
    return torch.tensor(freq, dtype=torch.float64)


def rotate_pairs(x, freq):
    """x [n, heads, d]: elements 2i and 2i + 1 of the first 2 len(freq) are the pair (u, v) -> (u cos a - v sin a,
    v cos a + u sin a) with a = position * freq_i; the other elements pass."""
    n, dims = x.shape[0], 2 * len(freq)
    ang = torch.arange(n, dtype=torch.float64)[:, None] * freq[None, :]
    cos, sin = ang.cos().to(x.dtype)[:, None, :], ang.sin().to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------

def visible(n, size=None, keep_first=0):
    """[n, n] bool: query i sees key j <= i where i - j < size (all of them without a size) or j < keep_first."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def softmax_attention(q, k, v, scale, seen, softcap=None, weights=False):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; query head h reads key head h // (H / G)."""
    rep = q.shape[1] // k.shape[1]
    kk, vv = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    pr = torch.softmax(s.masked_fill(~seen[None], float("-inf")), dim=-1)
    return pr if weights else torch.einsum("hij,jhd->ihd", pr, vv)


def attention_mixer(x, w, p, m, eps, v_first=None, weights=False):
    """Returns (result, this layer's own values as projected): ``v_first`` [n, G, dv] are the values of the first layer
    that mixes, None in that layer itself and in layers that do not mix."""
    n = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ w[p + ".q"].T).view(n, H, d)
    k = (x @ w[p + ".k"].T).view(n, G, d)
    v = own = (x @ w[p + ".v"].T).view(n, G, dv)
    if m.get("rot"):
        freq = rotation_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q, k = rotate_pairs(q, freq), rotate_pairs(k, freq)
    q, k = rms_unit(q, eps), rms_unit(k, eps)
    if v_first is not None:
        lam = w[p + ".vmix"]
        v = (1.0 - lam) * v + lam * v_first
    mask = m.get("mask") or {}
    seen = visible(n, mask.get("size"), mask.get("keep_first", 0))
    o = softmax_attention(q, k, v, m["scale"], seen, m.get("softcap"), weights)
    return (o if weights else o.reshape(n, H * dv) @ w[p + ".o"].T), own


# ---------------------------------------------------------------------------
# recurrences
# ---------------------------------------------------------------------------

def mlstm_gates(x, w, p, cap):
    """(log input gate, log forget gate), [n, heads] each."""
    i = cap * torch.tanh((x @ w[p + ".i"].T + w[p + ".i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((x @ w[p + ".f"].T + w[p + ".f.b"]) / cap))
    return i, f


def mlstm_rule(q, k, v, i, f, state=None):
    """q, k [n, H, dk] (q scaled), v [n, H, dv], i, f [n, H].  m_t = max(f + m, i) from m = 0, S_t = e^(f + m - m_t) S +
    e^(i - m_t) k v^T, n_t likewise with k; o = S^T q / (max(|n . q|, e^(-m_t)) + 1e-6).  Returns (o, (S, n, m))."""
    n_tok, H, dk = q.shape
    if state is None:
        state = (torch.zeros(H, dk, v.shape[-1], dtype=q.dtype), torch.zeros(H, dk, dtype=q.dtype),
                 torch.zeros(H, dtype=q.dtype))
    S, nrm, m = state
    out = []
    for t in range(n_tok):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        nrm = keep[:, None] * nrm + put[:, None] * k[t]
        m = m_new
        den = torch.maximum((nrm * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hkv,hk->hv", S, q[t]) / den[:, None])
    return torch.stack(out), (S, nrm, m)


def mlstm_mixer(x, w, p, m, eps):
    n = x.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (x @ w[p + ".q"].T).view(n, H, dk) * dk ** -0.5
    k = (x @ w[p + ".k"].T).view(n, H, dk)
    v = (x @ w[p + ".v"].T).view(n, H, dv)
    i, f = mlstm_gates(x, w, p, float(m["gate_cap"]))
    o, _ = mlstm_rule(q, k, v, i, f)
    o = rms_unit(o, eps).reshape(n, H * dv) * w[p + ".norm"] * torch.sigmoid(x @ w[p + ".g"].T)
    return o @ w[p + ".o"].T


def causal_conv(x, taps_w):
    """x [n, c], taps_w [c, taps] (last column the current token's), zeros before the start."""
    n, c = x.shape
    taps = taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, c, dtype=x.dtype), x], dim=0)
    return sum(padded[j:j + n] * taps_w[:, j] for j in range(taps))


def delta_decay(x, w, p):
    """[n, heads]: exp(-exp(A_log) softplus(W_a x + dt_bias))."""
    return torch.exp(-torch.exp(w[p + ".A_log"]) * softplus(x @ w[p + ".a"].T + w[p + ".dt_bias"]))


def delta_rule(q, k, v, g, beta, state=None):
    """q, k [n, G, dk] (unit, q scaled), v [n, H, dv], g, beta [n, H].  S <- g S; u = beta (v - S^T k); S <- S + k u^T;
    o = S^T q."""
    n, H = v.shape[:2]
    rep = H // q.shape[1]
    S = torch.zeros(H, q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(n):
        qq, kk = q[t].repeat_interleave(rep, dim=0), k[t].repeat_interleave(rep, dim=0)
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, kk))
        S = S + kk[:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, qq))
    return torch.stack(out), S


def delta_inputs(x, w, p, m):
    """q, k [n, G, dk] as unit vectors (q times dk^(-1/2)) and v [n, H, dv], after convolution and silu."""
    n = x.shape[0]
    q, k, v = (silu(causal_conv(x @ w[f"{p}.{s}"].T, w[f"{p}.{s}.conv"])) for s in "qkv")
    unit = lambda z: z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6)
    q = unit(q.view(n, m["kv_heads"], m["dim"])) * m["dim"] ** -0.5
    return q, unit(k.view(n, m["kv_heads"], m["dim"])), v.view(n, m["heads"], m["vdim"])


def delta_mixer(x, w, p, m, eps):
    n = x.shape[0]
    H, dv = m["heads"], m["vdim"]
    q, k, v = delta_inputs(x, w, p, m)
    o, _ = delta_rule(q, k, v, delta_decay(x, w, p), torch.sigmoid(x @ w[p + ".b"].T))
    o = rms_norm(o, w[p + ".norm"], eps) * silu(x @ w[p + ".g"].T).view(n, H, dv)
    return o.reshape(n, H * dv) @ w[p + ".o"].T


# ---------------------------------------------------------------------------
# feed-forward, per-layer token input
# ---------------------------------------------------------------------------

# a list here collects, per routed layer, the smallest gap between the last chosen and the first rejected logit
ROUTING_GAPS = None


def route(x, w, p, top):
    """Chosen experts [n, top] (largest logits first, ties to the lower index) and the softmax over their logits."""
    z = x @ w[p + ".router"].T
    ranked = torch.sort(z, dim=-1, descending=True, stable=True)
    if ROUTING_GAPS is not None and z.shape[1] > top:
        ROUTING_GAPS.append(float((ranked.values[:, top - 1] - ranked.values[:, top]).min()))
    return ranked.indices[:, :top], torch.softmax(ranked.values[:, :top], dim=-1)


def clamped_expert(x, w, p, limit):
    g = (x @ w[p + ".gate"].T).clamp(max=limit)
    u = (x @ w[p + ".up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + ".down"].T


def feed_forward(x, w, p, f):
    if f["kind"] == "dense":
        return gelu_tanh(x @ w[p + ".up"].T) @ w[p + ".down"].T
    ids, weights = route(x, w, p, f["router"]["top"])
    out = torch.zeros_like(x)
    for e in range(f["router"]["experts"]):
        out = out + clamped_expert(x, w, f"{p}.e{e}", float(f["expert"]["limit"])) * (weights * (ids == e)).sum(-1, keepdim=True)
    return out


def token_side(x, tokens, w, layer, dim, eps):
    """What layer ``layer`` adds for the tokens themselves: x is the stream after the feed-forward."""
    e = w["side.embed"][torch.tensor(list(tokens), dtype=torch.long)][:, layer * dim:(layer + 1) * dim]
    p = f"l{layer}.side"
    return rms_norm((gelu_tanh(x @ w[p + ".gate"].T) * e) @ w[p + ".proj"].T, w[p + ".norm"], eps)


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def forward(tokens, w, cfg, dtype=torch.float64, streams=False):
    """Logits [n, vocab] of the whole sequence (and, with ``streams``, the residual stream after every layer)."""
    w = {k: (t.to(dtype) if t.is_floating_point() else t) for k, t in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
    v_first, kept = None, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = rms_norm(x, w[p + ".norm1"], eps)
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention_mixer(h, w, p + ".mix", m, eps, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        else:
            y = {"mlstm": mlstm_mixer, "delta": delta_mixer}[layer["type"]](h, w, p + ".mix", m, eps)
        x = x + y
        if layer.get("mlp"):
            x = x + feed_forward(rms_norm(x, w[p + ".norm2"], eps), w, p + ".mlp", layer["mlp"])
        if cfg.get("token_side"):
            x = x + token_side(x, tokens, w, i, cfg["token_side"]["dim"], eps)
        kept.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
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
