"""A plain, slow implementation of the Zanezen decoder: one function per mechanism, whole sequences at once, float64 on
the CPU, no cache and no state carried between calls.  It shares no code with the package; the tests compare the engine
with it.

Notation: T tokens, x [T, width]; weights are a dict of float tensors by checkpoint name, a linear weight is
[out, in] and is applied as x @ W.T; ``p`` is a layer's name prefix (``l3.``), a mixer's (``l3.mix.``) or a
feed-forward's (``l3.mlp.``), ``m`` a mixer's record of the configuration."""
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


def silu(z):
    return z * torch.sigmoid(z)


def squared_relu(z):
    return torch.clamp(z, min=0.0) ** 2


def over_root_mean_square(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return over_root_mean_square(x, eps) * w


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


# ---------------------------------------------------------------- positions
def pair_frequencies(base, dims, scaling=None):
    """(frequencies of the dims / 2 pairs, factor on cosine and sine).  With ``scaling`` {factor, original, fast, slow} the
    pairs that turn fewer than ``slow`` times over ``original`` positions are slowed by ``factor``, those that turn more than
    ``fast`` times are left, the ones between (in pair index) are blended."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, original, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))

    def index_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def turn_halves(x, freqs, magnitude=1.0):
    """x [T, ..., d]: with n = len(freqs), the pair (x[i], x[i + n]) of the token at position p turns by p * freqs[i] and is
    multiplied by ``magnitude``; columns from 2 n on pass."""
    n = len(freqs)
    if n == 0:
        return x
    a = torch.arange(x.shape[0], dtype=F)[:, None] * torch.tensor(freqs, dtype=F)[None, :]
    a = a.view(x.shape[0], *([1] * (x.dim() - 2)), n)
    c, s = torch.cos(a) * magnitude, torch.sin(a) * magnitude
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def rotation(m):
    rot = m.get("rot")
    return pair_frequencies(rot["base"], rot["dims"], rot.get("scaling")) if rot and rot.get("dims") else ([], 1.0)


# ---------------------------------------------------------------- attention
def causal_mask(T):
    i = torch.arange(T)
    return i[None, :] <= i[:, None]


def causal_convolution(u, w):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros in front; u [T, channels], w [channels, taps]."""
    if w is None:
        return u
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    y = sum(w[:, j] * padded[j:j + T] for j in range(taps))
    return y if _ROUNDING[0] is None else _ROUNDING[0](y)


def softmax_over_visible(s, mask, sink=None):
    """exp(s_j) / (exp(sink) + sum exp(s_j)) over the visible keys; ``sink`` None: no further term, else one number per head
    (s [heads, T, T])."""
    s = torch.where(mask, s, torch.full_like(s, -math.inf))
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink.view(-1, 1, 1))
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink.view(-1, 1, 1) - top)
    return e / total


def difference_weight(W, p, m):
    return (torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + float(m["diff"]))


def differential_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_convolution(product(h, W[p + n]), W.get(p + n + ".conv")) for n in ("q", "k", "v"))
    q, k, v = q.view(T, H, 2, d), k.view(T, G, 2, d), v.view(T, G, dv)
    freqs, magnitude = rotation(m)
    q, k = turn_halves(q, freqs, magnitude), turn_halves(k, freqs, magnitude)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    mask, a = causal_mask(T), []
    for i in range(2):
        s = soft_cap(torch.einsum("ihd,jhd->hij", q[:, :, i], k[:, :, i]) * float(m["scale"]), m.get("softcap"))
        a.append(torch.einsum("hij,jhd->ihd", softmax_over_visible(s, mask), v))
    o = a[0] - difference_weight(W, p, m) * a[1]
    o = over_root_mean_square(o, eps) * (1.0 - float(m["diff"]))
    return product(o.reshape(T, H * dv), W[p + "o"])


def latent_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = product(h, W[p + "q"]).view(T, H, d + dr)
    down = product(h, W[p + "dkv"])
    c = rms_norm(down[:, :R], W[p + "dkv.norm"], eps)
    if _ROUNDING[0] is not None:
        c = _ROUNDING[0](c)
    freqs, magnitude = rotation(m)
    q_rot = turn_halves(q[..., d:], freqs, magnitude)
    k_rot = turn_halves(down[:, R:], freqs, magnitude)
    k = product(c, W[p + "uk"]).view(T, H, d)
    v = product(c, W[p + "uv"]).view(T, H, dv)
    s = torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    P = softmax_over_visible(s * float(m["scale"]), causal_mask(T), W[p + "sink"])
    o = torch.einsum("hij,jhd->ihd", P, v) * torch.sigmoid(product(h, W[p + "g"]))[:, :, None]
    return product(o.reshape(T, H * dv), W[p + "o"])


# ---------------------------------------------------------------- recurrence
def matrix_memory(q, k, v, log_input, log_forget):
    """Per head: m_t = max(f_t + m_(t-1), i_t);  S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T;  n_t alike with
    k_t alone;  o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6).  q, k [T, H, d], v [T, H, dv], gates [T, H]; the state and
    m start at zero.  Returns (o [T, H, dv], S, n, m)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(H, d, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        new = torch.maximum(log_forget[t] + m, log_input[t])
        keep, take = torch.exp(log_forget[t] + m - new), torch.exp(log_input[t] - new)
        m = new
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        total = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / total[:, None])
    return torch.stack(out), S, n, m


def mlstm(h, W, p, m, eps):
    T, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q = product(h, W[p + "q"]).view(T, H, d) * d ** -0.5
    k = product(h, W[p + "k"]).view(T, H, d)
    v = product(h, W[p + "v"]).view(T, H, dv)
    log_input = soft_cap(product(h, W[p + "i"]) + W[p + "i.b"], cap)
    log_forget = torch.nn.functional.logsigmoid(soft_cap(product(h, W[p + "f"]) + W[p + "f.b"], cap))
    o = over_root_mean_square(matrix_memory(q, k, v, log_input, log_forget)[0], eps).reshape(T, H * dv)
    return product(o * W[p + "norm"] * torch.sigmoid(product(h, W[p + "g"])), W[p + "o"])


MIXERS = {"mlstm": mlstm, "attention": differential_attention, "latent_attention": latent_attention}


# ---------------------------------------------------------------- feed-forward
def dense_feed_forward(h, W, p):
    gate, up = product(h, W[p + "gate"]) + W[p + "gate.b"], product(h, W[p + "up"]) + W[p + "up.b"]
    return product(silu(gate) * up, W[p + "down"]) + W[p + "down.b"]


def route(h, W, p, router):
    """(chosen experts [T, top], their weights [T, top], the distance of the last chosen choice score to the first that was
    left out [T])."""
    s = torch.sigmoid(h @ W[p + "router"].T)
    choice = s + W[p + "correction"]
    order = torch.argsort(choice, dim=-1, descending=True, stable=True)
    top = router["top"]
    chosen = order[:, :top]
    w = torch.gather(s, 1, chosen)
    ranked = torch.gather(choice, 1, order)
    margin = ranked[:, top - 1] - ranked[:, top] if top < s.shape[1] else torch.full((h.shape[0],), math.inf, dtype=h.dtype)
    return chosen, w / (w.sum(dim=-1, keepdim=True) + 1e-20) * float(router["scale"]), margin


def expert(h, W, p):
    return product(squared_relu(product(h, W[p + "up"])), W[p + "down"])


_MARGINS = [None]    # a list that every routed layer appends its margins [T] to while ``forward(..., margins=list)`` runs


def mixture(h, W, p, mlp):
    f = _ROUNDING[0]
    chosen, weights, margin = route(h if f is None else f(h), W, p, mlp["router"])
    if _MARGINS[0] is not None:
        _MARGINS[0].append(margin)
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, place = (chosen == e).nonzero(as_tuple=True)
        if t.numel():
            y[t] += weights[t, place][:, None] * expert(h[t], W, p + f"e{e}.")
    if mlp.get("shared") is not None:
        y = y + expert(h, W, p + "shared.") * torch.sigmoid(product(h, W[p + "shared.sg"]))
    return y


# ---------------------------------------------------------------- the model
def layer(x, W, config, i):
    L = config["layers"][i]
    p, eps = f"l{i}.", float(config["norm"]["eps"])
    h = rms_norm(x, W[p + "norm1"], eps)
    y = MIXERS[L["type"]](h, W, p + "mix.", L["mixer"], eps)
    mlp = L.get("mlp")
    if mlp is not None:
        y = y + (dense_feed_forward(h, W, p + "mlp.") if mlp["kind"] == "dense" else mixture(h, W, p + "mlp.", mlp))
    return x + float(config["residual_mult"]) * y


def forward(config, weights, tokens, return_layers=False, reads=None, margins=None):
    """Logits [T, vocab] of one sequence (float64); with ``return_layers`` also the stream after every layer.  ``reads``:
    a rounding applied to what every product reads and to what it returns (to see how far roundings alone move the
    result).  ``margins``: a list every routed layer appends its margins to (see ``route``)."""
    W = {k: (v.to(F) if v.is_floating_point() else v) for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    _ROUNDING[0], _MARGINS[0] = reads, margins
    x = W["embed"][tokens] * float(config["embedding"]["scale"])
    layers = []
    for i in range(len(config["layers"])):
        x = layer(x, W, config, i)
        layers.append(x)
    last = rms_norm(x, W["final.norm"], float(config["norm"]["eps"]))
    logits = (reads(last) if reads else last) @ W["head"].T
    _ROUNDING[0] = _MARGINS[0] = None
    return (logits, layers) if return_layers else logits
