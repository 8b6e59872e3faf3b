"""Recurrent mixers whose memory is one matrix per head that decays and gains an outer product per token, without the
delta rule's correction:  S_t = diag(g_t) S_(t-1) + k_t (b_t v_t)^T,  o_t = S_t^T q_t.  Four of them:

``GatedLinearAttention`` (``gla``): a decay per key channel from a low-rank projection,

    q = W_q x * d_k^(-1/2) ;  k = W_k x  [heads, d_k] ;  v = W_v x  [heads, d_v]
    g = sigmoid(W_a2 (W_a1 x) + bias)^(1 / tau)  [heads, d_k] ;  b = 1
    y = W_o ( o / rms(o) * norm_weight * silu(W_g x) )                          rms over d_v, per head

``StateSpaceDuality`` (``ssd``, the Mamba-2 layer): one scalar decay per head and a step size on the value,

    [z | x | B | C | dt] = W_in u ;  x, B, C pass a short causal convolution with bias, then SiLU
    dt = softplus(dt + dt_bias)  [heads] ;  g = exp(-exp(A_log[h]) dt) ;  b = dt
    k = B, q = C  [groups, state] (head h reads group h / (heads / groups)) ;  v = x  [heads, d_v]
    o_t += D_h x_t ;  y = W_o ( norm( o * silu(z) ) )       the gate first, then an RMS norm in ``norm_groups`` equal parts

``FixedDecayAttention`` (``fixed_decay``): a decay per head that the configuration gives, b = 1 (retention, lightning attention),

    q, k = act(W_q x), act(W_k x)  [heads, d_k] ;  v = act(W_v x)  [heads, d_v] ;  act: SiLU or none
    q and k turned by the token's position (halves; optional) ;  q times ``scale`` (it stands for a factor on the keys as well)
    y = W_o ( norm(o) * gate(W_g x) )      norm over each head's numbers or over all heads together, with a weight or none

``MatrixMemory`` (``mlstm``): an exponential input gate and a forget gate per head and token, both soft-capped logarithms,

    q = W_q x * d_k^(-1/2), k = W_k x  [heads, d_k] ;  v = W_v x  [heads, d_v]
    i = cap tanh((W_i x + b_i) / cap),  f = log sigmoid(cap tanh((W_f x + b_f) / cap))  [heads]
    m_t = max(f + m_(t-1), i) from m = 0 ;  g = e^(f + m_(t-1) - m_t), b = e^(i - m_t) ;  n_t = g n_(t-1) + b k_t
    o = S^T q / (max(|n . q|, e^(-m)) + 1e-6) ;  y = W_o ( o / rms(o) per head * norm_weight * gate(W_g x) )

All keep, per sequence, S of every head in 32 bits (and the convolution's last inputs) in one row of their cache slot,
starting from zero.  Decays, step sizes, the recurrence and the output norms are 32-bit in both precisions; projections
and the convolution are computed in the run's precision.  The scan is the kernel of the delta rule, told to leave out
the correction; a decay fixed per head and the matrix memory have kernels of their own, which take runs of tokens at once
(``ops.fixed_decay``, ``ops.matrix_memory``)."""
from __future__ import annotations

import torch

from ..cache.sequence_cache import StateNeed, StateView
from ..config.base import ConfigError
from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import Mixer, OpenEnded, PositionEncoding, StepContext, register_mixer
from .linear import Linear
from .position import PAIRING_CODES


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


def _stacked(groups: list[torch.Tensor], device, silu_groups: int = 0) -> tuple[Linear, list[int]]:
    """One product for several weights: their rows one after the other, each group padded to a multiple of 8 rows.
    ``silu_groups``: so many of the first groups' results are stored activated."""
    common = torch.float32 if any(g.dtype == torch.float32 for g in groups) else groups[0].dtype
    rows, offsets, at = [], [], 0
    for g in groups:
        offsets.append(at)
        rows.append(g.to(common))
        pad = _pad8(g.shape[0]) - g.shape[0]
        if pad:
            rows.append(torch.zeros((pad, g.shape[1]), dtype=common, device=device))
        at += _pad8(g.shape[0])
    offsets.append(at)
    return Linear(torch.cat(rows, dim=0).contiguous(), silu_columns=offsets[silu_groups]), offsets[:-1]


class GatedLinearAttention(Mixer):
    graph_safe = True   # slots and lengths reach the kernels through the step's device tensors
    pad_safe = False    # every token it sees enters the state

    def __init__(self, hidden_size: int, n_heads: int, head_dim: int, value_dim: int, decay_temperature: float,
                 norm_eps: float, decay_rank: int | None = None):
        """``decay_temperature`` tau: the decay is sigmoid(.)^(1 / tau).  ``decay_rank``: inner size of the decay's two
        products; None reads it from the checkpoint's shapes (it is needed to make random weights)."""
        if min(n_heads, head_dim, value_dim) < 1 or head_dim > 512:
            raise ConfigError(f"gated linear attention: key size {head_dim} must be between 1 and 512, heads and value size positive")
        if not decay_temperature > 0:
            raise ConfigError(f"gated linear attention: the decay's temperature must be positive, got {decay_temperature}")
        self.hidden_size, self.n_heads, self.key_dim, self.value_dim = int(hidden_size), int(n_heads), int(head_dim), int(value_dim)
        self.tau, self.norm_eps, self.decay_rank = float(decay_temperature), float(norm_eps), decay_rank
        self.state_floats = self.n_heads * self.key_dim * self.value_dim

    def parameters(self):
        H, dk, dv, h = self.n_heads, self.key_dim, self.value_dim, self.hidden_size
        r = self.decay_rank if self.decay_rank is not None else -1
        return {"q": ParamSpec((H * dk, h)), "k": ParamSpec((H * dk, h)), "v": ParamSpec((H * dv, h)),
                "g": ParamSpec((H * dv, h)), "o": ParamSpec((h, H * dv)), "norm": ParamSpec((dv,), "norm"),
                "a1": ParamSpec((r, h)), "a2": ParamSpec((H * dk, r)), "a2_bias": ParamSpec((H * dk,), "normal", 2.0, 1.0)}

    def cache_need(self):
        return StateNeed((self.state_floats,), torch.float32)

    def load(self, tensors, dtype, device):
        run = lambda t: t.to(device).to(torch.float32 if dtype == torch.float32 else t.dtype)
        f32 = lambda n: tensors[n].to(device=device, dtype=torch.float32).contiguous()
        self.inputs, (self.q_off, self.k_off, self.v_off, self.g_off, self.a1_off) = _stacked(
            [run(tensors[n]) for n in ("q", "k", "v", "g", "a1")], device)
        self.decay_rank = tensors["a1"].shape[0]
        self.a2 = Linear(run(tensors["a2"]).contiguous())
        self.o = Linear(run(tensors["o"]).contiguous())
        self.decay_bias, self.norm_weight = f32("a2_bias"), f32("norm")
        if device.type == "cuda" and not ops.delta_rule_supported(self.key_dim):
            raise ConfigError(f"gated linear attention: no kernel holds a state column of {self.key_dim} rows")

    def forward(self, x, ctx: StepContext, cache: StateView, residual, writes_cache=True, then_norm=None):
        H, dk, dv, T = self.n_heads, self.key_dim, self.value_dim, x.shape[0]
        proj = self.inputs.store(x, ctx.dtype, ctx.empty)
        decay = self.a2.store(proj[:, self.a1_off:self.a1_off + self.decay_rank], ctx.dtype, ctx.empty)    # [T, H dk]
        o = ctx.empty((T, H * dv), torch.float32)
        ops.linear_scan(proj[:, self.q_off:], proj[:, self.k_off:], proj[:, self.v_off:], decay, cache.data, ctx.slots_dev,
                        ctx.cu_seqlens, o, H, H, dk, dv, decay_kind=ops.DECAY_SIGMOID_POWER, decay_bias=self.decay_bias,
                        power=1.0 / self.tau, q_scale=dk ** -0.5, alloc=ctx.empty)
        gated = ctx.empty((T, H * dv), ctx.dtype)
        ops.gated_rmsnorm(o, self.norm_weight, proj[:, self.g_off:], gated, H, dv, self.norm_eps, "silu")
        return self.o.add_to(gated, residual, then_norm)


class StateSpaceDuality(Mixer):
    graph_safe = True
    pad_safe = False

    def __init__(self, hidden_size: int, n_heads: int, value_dim: int, state_dim: int, n_groups: int, conv_taps: int,
                 norm_eps: float, norm_groups: int = 1):
        if min(n_heads, value_dim, state_dim, n_groups, norm_groups) < 1 or state_dim > 512:
            raise ConfigError(f"state-space mixer: state size {state_dim} must be between 1 and 512, the other sizes positive")
        if n_heads % n_groups:
            raise ConfigError(f"state-space mixer: {n_heads} heads do not share {n_groups} groups equally")
        if (n_heads * value_dim) % norm_groups:
            raise ConfigError(f"state-space mixer: {n_heads * value_dim} numbers cannot be normed in {norm_groups} equal parts")
        if not (1 <= conv_taps <= ops.MAX_CONV_TAPS):
            raise ConfigError(f"conv taps {conv_taps}: the convolution kernel takes 1 to {ops.MAX_CONV_TAPS}")
        self.hidden_size, self.n_heads, self.value_dim, self.state_dim = int(hidden_size), int(n_heads), int(value_dim), int(state_dim)
        self.n_groups, self.taps, self.norm_eps, self.norm_groups = int(n_groups), int(conv_taps), float(norm_eps), int(norm_groups)
        self.inner = self.n_heads * self.value_dim
        self.channels = self.inner + 2 * self.n_groups * self.state_dim      # what the convolution runs over: x, B, C
        self.state_floats = self.n_heads * self.state_dim * self.value_dim
        self.conv_floats = (self.taps - 1) * self.channels

    def parameters(self):
        H, h = self.n_heads, self.hidden_size
        return {"in": ParamSpec((2 * self.inner + 2 * self.n_groups * self.state_dim + H, h)),
                "conv": ParamSpec((self.channels, self.taps), "normal", 0.0, 1.0 / self.taps ** 0.5),
                "conv_bias": ParamSpec((self.channels,), "normal", 0.0, 0.1),
                "dt_bias": ParamSpec((H,), "normal", 0.0, 1.0), "A_log": ParamSpec((H,), "normal", -1.0, 0.5),
                "D": ParamSpec((H,), "normal", 1.0, 0.2), "norm": ParamSpec((self.inner,), "norm"),
                "o": ParamSpec((h, self.inner))}

    def cache_need(self):
        return StateNeed((self.state_floats + self.conv_floats,), torch.float32)

    def load(self, tensors, dtype, device):
        run = lambda t: t.to(device).to(torch.float32 if dtype == torch.float32 else t.dtype)
        f32 = lambda n: tensors[n].to(device=device, dtype=torch.float32).contiguous()
        w = run(tensors["in"])
        i, gn = self.inner, self.n_groups * self.state_dim
        # rows as stored: z, then x | B | C (one run of columns for the convolution), then dt; dt's group starts on a multiple of 8
        self.inputs, (self.z_off, self.conv_off, self.dt_off) = _stacked([w[:i], w[i:2 * i + 2 * gn], w[2 * i + 2 * gn:]], device)
        self.o = Linear(run(tensors["o"]).contiguous())
        self.conv_weight, self.conv_bias = f32("conv"), f32("conv_bias")
        self.dt_bias, self.a_log, self.skip, self.norm_weight = f32("dt_bias"), f32("A_log"), f32("D"), f32("norm")
        if device.type == "cuda" and not ops.delta_rule_supported(self.state_dim):
            raise ConfigError(f"state-space mixer: no kernel holds a state column of {self.state_dim} rows")

    def forward(self, x, ctx: StepContext, cache: StateView, residual, writes_cache=True, then_norm=None):
        H, G, N, dv, T, gn = self.n_heads, self.n_groups, self.state_dim, self.value_dim, x.shape[0], self.n_groups * self.state_dim
        state = cache.data                                                    # [slots, S of every head | convolution inputs]
        proj = self.inputs.store(x, ctx.dtype, ctx.empty)
        xbc = ctx.empty((T, self.channels), ctx.dtype)
        ops.causal_conv(proj[:, self.conv_off:], self.conv_weight, state[:, self.state_floats:], ctx.slots_dev, ctx.seq_ids,
                        ctx.cu_seqlens, xbc, self.channels, bias=self.conv_bias, activation="silu", update_state=writes_cache)
        o = ctx.empty((T, self.inner), torch.float32)
        ops.linear_scan(xbc[:, self.inner + gn:], xbc[:, self.inner:], xbc, proj[:, self.dt_off:], state, ctx.slots_dev,
                        ctx.cu_seqlens, o, H, G, N, dv, decay_kind=ops.DECAY_SOFTPLUS_RATE, decay_per_head=True,
                        decay_bias=self.dt_bias, a_log=self.a_log, step_scales_value=True, skip=self.skip, alloc=ctx.empty)
        gated = ctx.empty((T, self.inner), ctx.dtype)
        ops.gated_rmsnorm(o, self.norm_weight, proj[:, self.z_off:], gated, self.norm_groups, self.inner // self.norm_groups,
                          self.norm_eps, "silu", gate_first=True)
        return self.o.add_to(gated, residual, then_norm)


class FixedDecayAttention(Mixer, OpenEnded):
    graph_safe = True
    gives_input = True
    pad_safe = False

    def __init__(self, hidden_size: int, n_heads: int, head_dim: int, value_dim: int, decay, norm_eps: float, *,
                 activation: str | None = None, position: PositionEncoding | None = None, scale: float = 1.0,
                 norm_over: str = "head", norm_weight: bool = False, gate: str = "silu"):
        """``decay``: one number per head.  ``norm_over``: ``head`` (every head by its own root mean square) or ``all`` (all heads
        together).  ``norm_weight``: the norm has a weight per number.  ``gate``: the activation of the output gate."""
        if min(n_heads, head_dim, value_dim) < 1 or head_dim > 512:
            raise ConfigError(f"fixed-decay attention: key size {head_dim} must be between 1 and 512, heads and value size positive")
        if len(decay) != n_heads or not all(0.0 <= float(g) <= 1.0 for g in decay):
            raise ConfigError(f"fixed-decay attention: {n_heads} heads need as many decays between 0 and 1, got {list(decay)}")
        if activation not in (None, "silu") or norm_over not in ("head", "all") or gate not in ops.GATE_ACTIVATIONS:
            raise ConfigError(f"fixed-decay attention: activation {activation!r}, norm over {norm_over!r}, gate {gate!r}")
        if position is not None and position.rotary_dim:
            if position.rotary_dim > head_dim or position.pairing != PAIRING_CODES["half"]:
                raise ConfigError(f"fixed-decay attention turns pairs over halves of at most {head_dim} numbers")
        self.hidden_size, self.n_heads, self.key_dim, self.value_dim = int(hidden_size), int(n_heads), int(head_dim), int(value_dim)
        self.decay, self.norm_eps, self.scale = [float(g) for g in decay], float(norm_eps), float(scale)
        self.silu, self.position, self.norm_over = activation == "silu", position, norm_over
        self.norm_weight, self.gate = bool(norm_weight), gate
        self.state_floats = self.n_heads * self.key_dim * self.value_dim
        self.inputs: Linear | None = None
        self.o: Linear | None = None

    def parameters(self):
        H, dk, dv, h = self.n_heads, self.key_dim, self.value_dim, self.hidden_size
        p = {"q": ParamSpec((H * dk, h)), "k": ParamSpec((H * dk, h)), "v": ParamSpec((H * dv, h)), "g": ParamSpec((H * dv, h)),
             "o": ParamSpec((h, H * dv))}
        if self.norm_weight:
            p["norm"] = ParamSpec((H * dv if self.norm_over == "all" else dv,), "norm")
        return p

    def children(self):
        return {"position": self.position} if self.position is not None else {}

    def cache_need(self):
        return StateNeed((self.state_floats,), torch.float32)

    def load(self, tensors, dtype, device):
        run = lambda t: t.to(device).to(torch.float32 if dtype == torch.float32 else t.dtype)
        self.inputs, (self.q_off, self.k_off, self.v_off, self.g_off) = _stacked([run(tensors[n]) for n in ("q", "k", "v", "g")], device,
                                                                                      silu_groups=3 if self.silu else 0)
        self.o = Linear(run(tensors["o"]).contiguous())
        self.weight = tensors["norm"].to(device=device, dtype=torch.float32).contiguous() if self.norm_weight else None
        self.decays = torch.tensor(self.decay, dtype=torch.float64).to(torch.float32).to(device)
        self.inv_freq = None
        if self.position is not None and self.position.rotary_dim:
            self.inv_freq = self.position.inverse_frequencies(device)[:self.position.rotary_dim // 2].contiguous()
        if device.type == "cuda" and not ops.delta_rule_supported(self.key_dim):
            raise ConfigError(f"fixed-decay attention: no kernel holds a state column of {self.key_dim} rows")

    def open_columns(self):
        return self.n_heads * self.value_dim

    def take_output(self):
        weight, self.o = self.o.weight, None
        return weight, None

    def take_input(self):
        weight, self.inputs = self.inputs.weight, None
        return weight     # (whoever multiplies with it stores the results as they are: ``rows_from`` activates them)

    def takes_scaled_rows(self, ctx: StepContext) -> bool:
        return ctx.all_decode and self.inputs is not None and self.inputs.links_with(ctx.n_tokens, ctx.dtype)

    def rows_into(self, x, ctx: StepContext, cache: StateView, rows, writes_cache=True, mul=1.0):
        self._recur(self.inputs.store(x, ctx.dtype, ctx.empty), ctx, cache, rows, mul, silu=False)   # (activated by the product)

    def rows_from(self, raw, ctx: StepContext, cache: StateView, rows, writes_cache=True, mul=1.0):
        self._recur(raw, ctx, cache, rows, mul, silu=self.silu)

    def _recur(self, raw, ctx: StepContext, cache: StateView, rows, mul: float, silu: bool):
        """``silu``: whether the projections still have to be activated."""
        H, dk, dv, T = self.n_heads, self.key_dim, self.value_dim, raw.shape[0]
        q, k, v, g = (raw[:, at:] for at in (self.q_off, self.k_off, self.v_off, self.g_off))
        if ops.fixed_decay_takes(ctx.dtype, ctx.all_decode, dk, dv):
            # (a head that is normed alone and without a weight is finished where its values are)
            finish = None
            if self.norm_over == "head" and self.weight is None and ops.fixed_decay_finishes(ctx.all_decode, dk, dv):
                finish = (rows, g, self.gate, self.norm_eps, mul)
            o = None if finish is not None else ctx.empty((T, H * dv), torch.float32)
            ops.fixed_decay(q, k, v, self.decays, cache.data, ctx.slots_dev, ctx.cu_seqlens, ctx.positions, H, dk, dv, ctx.max_q_len,
                            q_scale=self.scale, qk_silu=silu, v_silu=silu, inv_freq=self.inv_freq, out=o,
                            finish=finish, alloc=ctx.empty)
            if finish is not None:
                return
        else:
            # (the true 32-bit run's prompts, and keys too long for a run's tiles: token by token)
            o = ctx.empty((T, H * dv), torch.float32)
            ops.linear_scan(q, k, v, None, cache.data, ctx.slots_dev, ctx.cu_seqlens, o, H, H, dk, dv, decay_kind=ops.DECAY_FIXED,
                            decay_per_head=True, a_log=self.decays, q_scale=self.scale, qk_silu=silu, v_silu=silu,
                            rotary=(ctx.positions, self.inv_freq) if self.inv_freq is not None else None, alloc=ctx.empty)
        parts, d = (H, dv) if self.norm_over == "head" else (1, H * dv)
        ops.gated_rmsnorm(o, self.weight, g, rows, parts, d, self.norm_eps, self.gate, mul=mul)

    def forward(self, x, ctx: StepContext, cache: StateView, residual, writes_cache=True, then_norm=None):
        rows = ctx.empty((x.shape[0], self.open_columns()), ctx.dtype)
        self.rows_into(x, ctx, cache, rows, writes_cache)
        return self.o.add_to(rows, residual, then_norm)


class MatrixMemory(Mixer, OpenEnded):
    graph_safe = True
    pad_safe = False
    gives_input = True

    def __init__(self, hidden_size: int, n_heads: int, head_dim: int, value_dim: int, gate_cap: float, norm_eps: float, *,
                 gate: str = "sigmoid"):
        """``gate_cap``: the soft cap on both gates' logits.  ``gate``: the activation of the output gate."""
        if min(n_heads, head_dim, value_dim) < 1 or head_dim > ops.MAX_MEMORY_KEYS:
            raise ConfigError(f"matrix memory: key size {head_dim} must be between 1 and {ops.MAX_MEMORY_KEYS}, heads and value size positive")
        if not gate_cap > 0:
            raise ConfigError(f"matrix memory: the gates' cap must be positive, got {gate_cap}")
        if gate not in ops.GATE_ACTIVATIONS:
            raise ConfigError(f"matrix memory: gate {gate!r}; known: {', '.join(sorted(ops.GATE_ACTIVATIONS))}")
        self.hidden_size, self.n_heads, self.key_dim, self.value_dim = int(hidden_size), int(n_heads), int(head_dim), int(value_dim)
        self.cap, self.norm_eps, self.gate, self.scale = float(gate_cap), float(norm_eps), gate, int(head_dim) ** -0.5
        self.inputs: Linear | None = None
        self.o: Linear | None = None

    def parameters(self):
        H, dk, dv, h = self.n_heads, self.key_dim, self.value_dim, self.hidden_size
        return {"q": ParamSpec((H * dk, h)), "k": ParamSpec((H * dk, h)), "v": ParamSpec((H * dv, h)), "g": ParamSpec((H * dv, h)),
                "o": ParamSpec((h, H * dv)), "norm": ParamSpec((H * dv,), "norm"), "i": ParamSpec((H, h)), "f": ParamSpec((H, h)),
                "i_bias": ParamSpec((H,), "normal", -1.0, 1.0), "f_bias": ParamSpec((H,), "normal", 4.0, 1.0)}

    def cache_need(self):
        return StateNeed((ops.matrix_memory_state(self.n_heads, self.key_dim, self.value_dim),), torch.float32)

    def load(self, tensors, dtype, device):
        run = lambda t: t.to(device).to(torch.float32 if dtype == torch.float32 else t.dtype)
        f32 = lambda n: tensors[n].to(device=device, dtype=torch.float32).contiguous()
        self.inputs, (self.q_off, self.k_off, self.v_off, self.g_off, self.i_off, self.f_off) = _stacked(
            [run(tensors[n]) for n in ("q", "k", "v", "g", "i", "f")], device)
        self.o = Linear(run(tensors["o"]).contiguous())
        self.weight, self.i_bias, self.f_bias = f32("norm"), f32("i_bias"), f32("f_bias")

    def open_columns(self):
        return self.n_heads * self.value_dim

    def take_output(self):
        weight, self.o = self.o.weight, None
        return weight, None

    def take_input(self):
        weight, self.inputs = self.inputs.weight, None
        return weight

    def takes_scaled_rows(self, ctx: StepContext) -> bool:
        return ctx.all_decode and self.inputs is not None and self.inputs.links_with(ctx.n_tokens, ctx.dtype)

    def rows_into(self, x, ctx: StepContext, cache: StateView, rows, writes_cache=True, mul=1.0):
        self.rows_from(self.inputs.store(x, ctx.dtype, ctx.empty), ctx, cache, rows, writes_cache, mul)

    def rows_from(self, raw, ctx: StepContext, cache: StateView, rows, writes_cache=True, mul=1.0):
        assert mul == 1.0
        H, dk, dv, T = self.n_heads, self.key_dim, self.value_dim, raw.shape[0]
        q, k, v, g, i, f = (raw[:, at:] for at in (self.q_off, self.k_off, self.v_off, self.g_off, self.i_off, self.f_off))
        args = (q, k, v, (i, f, self.i_bias, self.f_bias), self.cap, cache.data, ctx.slots_dev, ctx.seq_ids, ctx.cu_seqlens, H, dk, dv,
                ctx.max_q_len)
        if ops.matrix_memory_finishes(ctx.dtype, ctx.all_decode, dk, dv):
            ops.matrix_memory(*args, q_scale=self.scale, finish=(rows, g, self.gate, self.norm_eps, self.weight), alloc=ctx.empty)
            return
        o = ctx.empty((T, H * dv), torch.float32)
        ops.matrix_memory(*args, q_scale=self.scale, out=o, alloc=ctx.empty)
        ops.gated_rmsnorm(o, self.weight, g, rows, H, dv, self.norm_eps, self.gate)

    def forward(self, x, ctx: StepContext, cache: StateView, residual, writes_cache=True, then_norm=None):
        rows = ctx.empty((x.shape[0], self.open_columns()), ctx.dtype)
        self.rows_into(x, ctx, cache, rows, writes_cache)
        return self.o.add_to(rows, residual, then_norm)


register_mixer("mlstm", MatrixMemory)
register_mixer("fixed_decay", FixedDecayAttention)
register_mixer("gla", GatedLinearAttention)
register_mixer("ssd", StateSpaceDuality)
