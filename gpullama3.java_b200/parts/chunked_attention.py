"""Attention within runs of positions, over values that are cached turned by their own positions.

    q = W_q h  [H heads x d],  k = W_k h  [G kv heads x d],  v = W_v h  [G x dv]            query head h reads kv head h / (H / G)
    every row of q and k: divided by its root mean square (eps inside the root), times a weight of d numbers shared by all
        heads (``norm_eps``), then its first ``rotary_dim`` numbers turned by the token's position (halves)
    v_j <- v_j turned by j over all dv numbers (halves, frequencies of their own): so it is cached          (``value_position``)
    p_j = exp(s_j) / (e^sink + sum_j' exp(s_j')),  s_j = scale q_i . k_j,  over j <= i with floor(i / chunk) = floor(j / chunk)
        (``chunk`` None: every j <= i; ``sink`` None: no further term in the denominator)
    o_i = (sum_j p_j v_j) turned by -i ;  out = W_o o                             so a value enters turned by j - i

Turning is linear, so turning the sum back by -i leaves every value turned by its distance alone.  The attention kernels
are those every attention mixer shares (``attend``): ``head_rows`` finishes queries, keys and values in one launch on their
way into the cache (rows widened with zeros to a size the kernels take), ``turn_back_rows`` turns the result back, in 32
bits, and leaves the dv numbers of every head in the rows of the last product.  Norms, angles, scores and softmax are 32-bit
in both precisions."""
from __future__ import annotations

import torch

from ..cache.sequence_cache import KVCacheNeed, KVView
from ..config.base import ConfigError
from ..kernels import ops
from ..weights.loader import ParamSpec
from .attention import attend, kernel_head_dim, plan_decode_attention
from .base import Mixer, OpenEnded, PositionEncoding, StepContext, register_mixer
from .linear import Linear
from .position import PAIRING_CODES


class _KernelShape:
    """The layer as the attention kernels see it."""
    keep_first = 0
    slopes = None
    window = None

    def __init__(self, n_heads: int, n_kv_heads: int, head_dim: int, chunk: int | None):
        self.n_heads, self.n_kv_heads, self.head_dim, self.chunk = n_heads, n_kv_heads, head_dim, chunk
        self.sinks = None

    @property
    def has_terms(self):
        return self.chunk is not None or self.sinks is not None

    def plan_decode(self, ctx: StepContext, cache: KVView):
        return plan_decode_attention(self, ctx, cache)


class ChunkedAttention(Mixer, OpenEnded):
    graph_safe = True
    gives_input = True
    pad_safe = True

    def __init__(self, hidden_size: int, n_heads: int, n_kv_heads: int, head_dim: int, value_dim: int, scale: float,
                 position: PositionEncoding, value_position: PositionEncoding | None = None, norm_eps: float | None = None,
                 chunk: int | None = None, sink: float | None = None):
        """``sink``: the score of a further key without a value that every query sees (0: one is added to the softmax's
        denominator); ``value_position``: how values are turned, over all their numbers."""
        if n_heads < 1 or n_kv_heads < 1 or n_heads % n_kv_heads:
            raise ConfigError(f"n_heads {n_heads} must be a multiple of n_kv_heads {n_kv_heads}")
        if min(head_dim, value_dim) < 1:
            raise ConfigError(f"head sizes must be positive, got {head_dim} and {value_dim}")
        if chunk is not None and chunk < 1:
            raise ConfigError(f"chunk {chunk} must be at least 1 (or None for no runs)")
        if position.rotary_dim % 2 or position.rotary_dim > head_dim:
            raise ConfigError(f"rotary_dim {position.rotary_dim} must be even and at most head_dim {head_dim}")
        if value_position is not None and value_position.rotary_dim and value_position.rotary_dim != value_dim:
            raise ConfigError(f"values are turned over all their {value_dim} numbers, not over {value_position.rotary_dim}")
        for p in (position, value_position):
            if p is not None and p.rotary_dim and p.pairing != PAIRING_CODES["half"]:
                raise ConfigError("this mixer turns pairs over the halves of a row (i, i + n)")
        self.hidden_size, self.heads, self.kv_heads = int(hidden_size), int(n_heads), int(n_kv_heads)
        self.key_dim, self.value_dim, self.scale = int(head_dim), int(value_dim), float(scale)
        self.position, self.value_position = position, value_position
        self.norm_eps, self.sink = norm_eps, (float(sink) if sink is not None else None)
        D = kernel_head_dim(max(self.key_dim, self.value_dim))
        if D > ops.MAX_HEAD_DIM:
            raise ConfigError(f"heads of {max(head_dim, value_dim)} do not fit the attention kernels' {ops.MAX_HEAD_DIM} numbers")
        self.row_dim = D
        self.shape = _KernelShape(self.heads, self.kv_heads, D, int(chunk) if chunk is not None else None)
        self.qkv: Linear | None = None
        self.o: Linear | None = None

    def parameters(self):
        H, G, d, dv, h = self.heads, self.kv_heads, self.key_dim, self.value_dim, self.hidden_size
        p = {"q": ParamSpec((H * d, h)), "k": ParamSpec((G * d, h)), "v": ParamSpec((G * dv, h)), "o": ParamSpec((h, H * dv))}
        if self.norm_eps is not None:
            p["q_norm"], p["k_norm"] = ParamSpec((d,), "norm"), ParamSpec((d,), "norm")
        return p

    def children(self):
        c = {"position": self.position}
        if self.value_position is not None:
            c["value_position"] = self.value_position
        return c

    def cache_need(self):
        return KVCacheNeed(self.kv_heads, self.row_dim, chunk=self.shape.chunk)

    def load(self, tensors, dtype, device):
        H, G, d, dv, D = self.heads, self.kv_heads, self.key_dim, self.value_dim, self.row_dim
        mats = [tensors[n].to(device) for n in ("q", "k", "v")]
        common = torch.float32 if (dtype == torch.float32 or any(m.dtype == torch.float32 for m in mats)) else mats[0].dtype
        rows = sum(m.shape[0] for m in mats)
        if rows % 8:   # the products' rows of 16-bit results start on 16-byte boundaries
            mats.append(torch.zeros((8 - rows % 8, self.hidden_size), dtype=common, device=device))
        self.qkv = Linear(torch.cat([m.to(common) for m in mats], dim=0).contiguous())
        o = tensors["o"].to(device)
        self.o = Linear(o.to(torch.float32 if dtype == torch.float32 else o.dtype).contiguous())
        normed = self.norm_eps is not None
        self.norm_weights = None
        if normed:
            self.norm_weights = torch.cat([tensors[n].to(device=device, dtype=torch.float32) for n in ("q_norm", "k_norm")]).contiguous()
        if self.sink is not None:
            self.shape.sinks = torch.full((H,), self.sink, dtype=torch.float32, device=device)
        # the keys' frequencies, then the values'
        n_k, n_v = self.position.rotary_dim // 2, (self.value_position.rotary_dim // 2 if self.value_position is not None else 0)
        self.value_freq = self.value_position.inverse_frequencies(device)[:n_v].contiguous() if n_v else None
        freqs = [self.position.inverse_frequencies(device)[:n_k]] if n_k else []
        freqs += [self.value_freq] if n_v else []
        self.freqs = torch.cat(freqs).contiguous() if freqs else None
        # the scale is folded into the queries: the attention kernels divide every score by sqrt(their head size)
        mul = self.scale * D ** 0.5
        norm = 1 if normed else 0
        wq, wk = (0, d) if normed else (-1, -1)
        query = ops.head_row_segment(0, H, d, 0, D, norm=norm, weight_off=wq, mul=mul, half_pairs=n_k)
        keys = ops.head_row_segment(H * d, G, d, 0, D, norm=norm, weight_off=wk, half_pairs=n_k, target=ops.TO_CACHE_KEYS)
        values = ops.head_row_segment((H + G) * d, G, dv, 0, D, half_pairs=n_v, freq_off=n_k, target=ops.TO_CACHE_VALUES)
        self.segments = ops.head_row_segments(query, keys, values)
        self.query_segment = ops.head_row_segments(query)

    def open_columns(self):
        return self.heads * self.value_dim

    def take_output(self):
        weight, self.o = self.o.weight, None
        return weight, None

    def take_input(self):
        weight, self.qkv = self.qkv.weight, None
        return weight

    def takes_scaled_rows(self, ctx: StepContext) -> bool:
        return ctx.all_decode and self.qkv is not None and self.qkv.links_with(ctx.n_tokens, ctx.dtype)

    def rows_into(self, x, ctx: StepContext, cache: KVView, rows, writes_cache=True, mul=1.0):
        self.rows_from(self.qkv.store(x, ctx.dtype, ctx.empty), ctx, cache, rows, writes_cache, mul)

    def rows_from(self, raw, ctx: StepContext, cache: KVView, rows, writes_cache=True, mul=1.0):
        H, dv, D, T = self.heads, self.value_dim, self.row_dim, raw.shape[0]
        table = ctx.page_tables[cache.group]
        q = ctx.empty((T, H * D), ctx.dtype)
        ops.head_rows(raw, q, self.segments if writes_cache else self.query_segment, self.norm_eps or 0.0, None, self.norm_weights,
                      cache=(ctx.positions, ctx.seq_ids, table, cache.k, cache.v) if writes_cache else None,
                      rotary=(ctx.positions, self.freqs) if self.freqs is not None else None)
        out = ctx.empty((T, H * D), ctx.dtype)
        attend(self.shape, q, out, ctx, table, cache)
        ops.turn_back_rows(out, ctx.positions, self.value_freq, rows, H, dv, D, mul)

    def forward(self, x, ctx: StepContext, cache: KVView, residual, writes_cache=True, then_norm=None):
        rows = ctx.empty((x.shape[0], self.open_columns()), ctx.dtype)
        self.rows_into(x, ctx, cache, rows, writes_cache)
        return self.o.add_to(rows, residual, then_norm)


register_mixer("chunked_attention", ChunkedAttention)
