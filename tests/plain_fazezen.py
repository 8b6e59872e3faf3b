"""A plain, slow implementation of the Fazezen decoder: one function per mechanism, whole sequences at once, float64 on
the CPU, no cache and no state carried between calls.  It shares no code with the package; the tests compare the engine
with it.

Notation: T tokens, x [T, width]; weights are a dict of float tensors by checkpoint name, a linear weight is
[out, in] and is applied as x @ W.T; ``p`` is a layer's name prefix (``l3.``) or a mixer's (``l3.mix.``), ``m`` a mixer's
record of the configuration."""
from __future__ import annotations

import math

import torch

F = torch.float64


# ---------------------------------------------------------------- small functions
_ROUNDING = [None]   # a function applied to what every product reads and returns while ``forward(..., reads=f)`` runs


def product(x, w):
    """x @ w.T; while a rounding is set, of the rounded x, and rounded itself."""
    f = _ROUNDING[0]
    return x @ w.T if f is None else f(f(x) @ w.T)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def over_root_mean_square(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm_around_zero(x, w, eps):
    return over_root_mean_square(x, eps) * (1.0 + w)


# ---------------------------------------------------------------- positions
def pair_frequencies(base, dims):
    """base^(-2i/dims) for the dims / 2 pairs."""
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def stretched_frequencies(freqs, scaling):
    """Slow pairs (wavelength above original / low) turn ``factor`` times slower, fast ones (below original / high) as
    they did, those between are blended in original / wavelength."""
    if not scaling:
        return list(freqs)
    factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for f in freqs:
        wave = 2.0 * math.pi / f
        if wave < original / high:
            out.append(f)
        elif wave > original / low:
            out.append(f / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def turn_halves(x, freqs, sign=1.0):
    """x [T, heads, d]: with n = len(freqs), the pair (x[i], x[i + n]) of the token at position p turns by
    sign * p * freqs[i]; columns from 2 n on pass."""
    n = len(freqs)
    if n == 0:
        return x
    T = x.shape[0]
    a = sign * torch.arange(T, dtype=F)[:, None] * torch.tensor(freqs, dtype=F)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


# ---------------------------------------------------------------- attention
def chunk_mask(T, size):
    """[T, T]: i sees j <= i of its own run of ``size`` positions, runs counted from position 0."""
    i = torch.arange(T)
    causal = i[None, :] <= i[:, None]
    if size is None:
        return causal
    return causal & (torch.div(i, size, rounding_mode="floor")[None, :] == torch.div(i, size, rounding_mode="floor")[:, None])


def softmax_with_silent_key(s, mask):
    """exp(s_j) / (1 + sum exp(s_j)) over the visible keys: a further key of score 0 that has no value."""
    s = torch.where(mask, s, torch.full_like(s, -math.inf))
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def chunked_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = product(h, W[p + "q"]).view(T, H, d)
    k = product(h, W[p + "k"]).view(T, G, d)
    v = product(h, W[p + "v"]).view(T, G, dv)
    q = over_root_mean_square(q, eps) * W[p + "q.norm"]
    k = over_root_mean_square(k, eps) * W[p + "k.norm"]
    rot = m.get("rot")
    if rot and rot.get("dims"):
        freqs = stretched_frequencies(pair_frequencies(rot["base"], rot["dims"]), rot.get("scaling"))
        q, k = turn_halves(q, freqs), turn_halves(k, freqs)
    if rot:
        v = turn_halves(v, pair_frequencies(rot["base"], dv))
    rep = H // G
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    P = softmax_with_silent_key(s, chunk_mask(T, (m.get("mask") or {}).get("size")))
    o = torch.einsum("hij,jhd->ihd", P, v)
    if rot:
        o = turn_halves(o, pair_frequencies(rot["base"], dv), sign=-1.0)
    return product(o.reshape(T, H * dv), W[p + "o"])


# ---------------------------------------------------------------- recurrences
def decayed_outer_sum(q, k, v, decay):
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, per head; q, k [T, H, d], v [T, H, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    g = torch.tensor([float(x) for x in decay], dtype=q.dtype)[:, None, None]
    out = []
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def retention(h, W, p, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = product(h, W[p + "q"]).view(T, H, d)
    k = product(h, W[p + "k"]).view(T, H, d)
    v = product(h, W[p + "v"]).view(T, H, dv)
    rot = m.get("rot")
    if rot and rot.get("dims"):
        freqs = pair_frequencies(rot["base"], rot["dims"])
        q, k = turn_halves(q, freqs), turn_halves(k, freqs)
    o = decayed_outer_sum(q, k * d ** -0.5, v, m["decay"])
    o = over_root_mean_square(o, eps).reshape(T, H * dv)
    return product(o * silu(product(h, W[p + "g"])), W[p + "o"])


def lightning_attention(h, W, p, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(product(h, W[p + "q"])).view(T, H, d)
    k = silu(product(h, W[p + "k"])).view(T, H, d)
    v = silu(product(h, W[p + "v"])).view(T, H, dv)
    o = decayed_outer_sum(q, k, v, m["decay"]).reshape(T, H * dv)
    o = over_root_mean_square(o, eps) * W[p + "norm"]
    return product(o * torch.sigmoid(product(h, W[p + "g"])), W[p + "o"])


def side_by_side(h, W, p, m, eps):
    """Two mixers on the same input, each with a factor of its own."""
    left = chunked_attention(h, W, p + "left.", m["left"], eps)
    right = retention(h, W, p + "right.", m["right"], eps)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


def mixer(h, W, p, kind, m, eps):
    return side_by_side(h, W, p, m, eps) if kind == "parallel" else lightning_attention(h, W, p, m, eps)


# ---------------------------------------------------------------- feed-forward
def dense_feed_forward(h, W, p):
    up = product(h, W[p + "up"]) + W[p + "up.b"]
    gate = product(h, W[p + "gate"]) + W[p + "gate.b"]
    return product(gelu_tanh(gate) * up, W[p + "down"]) + W[p + "down.b"]


# ---------------------------------------------------------------- the model
def layer(x, W, config, i):
    L = config["layers"][i]
    p, eps = f"l{i}.", float(config["norm"]["eps"])
    y = mixer(rms_norm_around_zero(x, W[p + "norm1"], eps), W, p + "mix.", L["type"], L["mixer"], eps)
    if L.get("mlp") is not None:
        y = y + dense_feed_forward(rms_norm_around_zero(x, W[p + "norm2"], eps), W, p + "mlp.")
    return x + y


def forward(config, weights, tokens, return_layers=False, reads=None):
    """Logits [T, vocab] of one sequence (float64); with ``return_layers`` also the stream after every layer.  ``reads``:
    a rounding applied to what every product reads and to what it returns (to see how far roundings alone move the
    result)."""
    W = {k: (v.to(F) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    _ROUNDING[0] = reads
    x = rms_norm_around_zero(W["embed"][tokens], W["embed.norm"], eps)
    layers = []
    for i in range(len(config["layers"])):
        x = layer(x, W, config, i)
        layers.append(x)
    last = rms_norm_around_zero(x, W["final.norm"], eps)
    logits = (reads(last) if reads else last) @ W["embed"].T
    _ROUNDING[0] = None
    return (logits, layers) if return_layers else logits
