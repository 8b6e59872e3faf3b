"""A routed feed-forward (mixture of experts): every token runs through a few of many small gated feed-forwards.

    z = W_r h (32-bit) ;  s = softmax(z) over all experts
    the experts form ``groups`` equal groups of neighbours; a group's score is its best expert's; only experts of the
    ``keep_groups`` best groups can be chosen; the ``top`` best of those are
    y = sum over the chosen e of  s_e / (sum of the chosen s + 1e-20) * down_e( act(gate_e h, up_e h) )

With ``router_bias`` a learned vector joins the logits z.  With one group and ``weight_eps`` 0 the weights are the softmax
over the chosen logits alone (s_e over the chosen s is exp(z_e) over the chosen exp(z)).

With ``score="sigmoid"`` every expert's score is the sigmoid of its own logit.  With ``choice_correction`` a learned vector joins the
scores for the choice alone: the experts are chosen by s + correction and weighed by s.  ``weight_scale``: a last factor on the
weights.  ``activation`` may be one without a gate (``relu_squared``): expert e is then down_e( act(up_e h) ).  ``shared_size``: a
further expert of that inner size that every token runs through, its result times sigmoid(w_sg h), one number per token.

With ``router="table"`` there is no router product: row ``token id`` of an integer table [vocabulary, top] names the token's
experts, and every one of them weighs 1 / top.

The router and the weights are 32-bit in both precisions.  The (token, choice) pairs are ordered by expert.  A step of
few tokens then runs every expert's rows as a weight-streaming product whose row counts are read on the device, so a
decode step's launches do not depend on the routing and can be recorded; an expert's weights are read once for all the
tokens that chose it, and not at all when none did.  A prompt's rows are gathered into the order of their experts and
multiplied by one launch of the tcgen05 product over all experts' tiles (gated epilogue included), which reads the runs
on the device as well.  Only where that kernel does not take the operands (the float32 run, sizes off its grid) do
the per-expert row counts come back to the host, for one product per expert through the kernels the dense feed-forward
uses; that wait is why a prompt pass of this part is not replayed from a recording."""
from __future__ import annotations

import torch

from ..config.base import ConfigError
from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import FeedForward, OpenEnded, StepContext, register_feed_forward
from .linear import Linear


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class RoutedFeedForward(FeedForward, OpenEnded):
    graph_safe = True    # (decode steps: the pair kernels read the routing from device memory)
    pad_safe = False     # a prompt pass may read the experts' row counts on the host

    def __init__(self, hidden_size: int, intermediate_size: int, n_experts: int, top: int, groups: int = 1,
                 keep_groups: int | None = None, activation: str = "silu", limit: float | None = None, slope: float = 1.0,
                 weight_eps: float = 1e-20, router: str = "learned", vocab_size: int | None = None,
                 router_bias: bool = False, score: str = "softmax", choice_correction: bool = False, weight_scale: float = 1.0,
                 shared_size: int | None = None):
        keep_groups = groups if keep_groups is None else keep_groups
        if router not in ("learned", "table"):
            raise ConfigError(f"routed feed-forward: router {router!r}; known: learned, table")
        if router == "table" and not vocab_size:
            raise ConfigError("routed feed-forward: a routing table needs the vocabulary's size")
        if router_bias and router != "learned":
            raise ConfigError("routed feed-forward: only a learned router has logits a bias can join")
        self.routing, self.vocab_size, self.router_bias = router, int(vocab_size or 0), bool(router_bias)
        self.gated = activation not in ops.UNGATED_ACTIVATIONS
        if self.gated and activation not in ops.ACTIVATION_CODES:
            raise ConfigError(f"feed-forward activation {activation!r}; known: "
                              f"{', '.join(sorted([*ops.ACTIVATION_CODES, *ops.UNGATED_ACTIVATIONS]))}")
        if score not in ops.ROUTER_SCORES:
            raise ConfigError(f"routed feed-forward: scores {score!r}; known: {', '.join(sorted(ops.ROUTER_SCORES))}")
        if (choice_correction or score != "softmax" or weight_scale != 1.0) and router != "learned":
            raise ConfigError("routed feed-forward: only a learned router has scores")
        if shared_size is not None and (shared_size < 1 or self.gated):
            raise ConfigError("routed feed-forward: a shared expert has a positive size and an activation without a gate")
        self.score, self.choice_correction, self.weight_scale = score, bool(choice_correction), float(weight_scale)
        self.shared_size = int(shared_size or 0)
        self.gives_input = self.shared_size > 0
        if activation == "clamped_sigmoid" and (limit is None or not limit > 0):
            raise ConfigError(f"the clamped feed-forward needs a positive limit, got {limit!r}")
        if not (1 <= n_experts <= ops.MAX_EXPERTS) or not (1 <= top <= min(n_experts, ops.MAX_EXPERTS_PER_TOKEN)):
            raise ConfigError(f"routed feed-forward: {top} of {n_experts} experts (at most {ops.MAX_EXPERTS_PER_TOKEN} of "
                              f"{ops.MAX_EXPERTS})")
        if groups < 1 or n_experts % groups or not (1 <= keep_groups <= groups):
            raise ConfigError(f"routed feed-forward: {n_experts} experts do not form {groups} equal groups of which "
                              f"{keep_groups} are kept")
        if top > keep_groups * (n_experts // groups):
            raise ConfigError(f"routed feed-forward: {top} experts cannot come from {keep_groups} groups of {n_experts // groups}")
        self.hidden_size, self.intermediate_size = int(hidden_size), int(intermediate_size)
        self.n_experts, self.top, self.groups, self.keep_groups = int(n_experts), int(top), int(groups), int(keep_groups)
        self.activation, self.gate_args, self.weight_eps = activation, (float(limit or 0.0), float(slope)), float(weight_eps)

    def parameters(self):
        p = ({"router": ParamSpec((self.n_experts, self.hidden_size))} if self.routing == "learned" else
             {"table": ParamSpec((self.vocab_size, self.top), "int_table", float(self.n_experts))})
        if self.router_bias:
            p["router_bias"] = ParamSpec((self.n_experts,), "normal", 0.0, 0.02)
        if self.choice_correction:
            p["correction"] = ParamSpec((self.n_experts,), "normal", 0.0, 0.1)
        if self.shared_size:
            p.update({"shared.up": ParamSpec((self.shared_size, self.hidden_size)),
                      "shared.down": ParamSpec((self.hidden_size, self.shared_size)), "shared.sg": ParamSpec((1, self.hidden_size))})
        for e in range(self.n_experts):
            if self.gated:
                p[f"e{e}.gate"] = ParamSpec((self.intermediate_size, self.hidden_size))
            p[f"e{e}.up"] = ParamSpec((self.intermediate_size, self.hidden_size))
            p[f"e{e}.down"] = ParamSpec((self.hidden_size, self.intermediate_size))
        return p

    def load(self, tensors, dtype, device):
        run = torch.float32 if dtype == torch.float32 else torch.bfloat16
        E, ff, h = self.n_experts, self.intermediate_size, self.hidden_size
        if self.routing == "learned":
            self.router = tensors["router"].to(device=device, dtype=torch.float32).contiguous()
            self.bias = tensors["router_bias"].to(device=device, dtype=torch.float32).contiguous() if self.router_bias else None
        else:
            self.table = tensors["table"].to(device=device, dtype=torch.int32).contiguous()
        self.correction = tensors["correction"].to(device=device, dtype=torch.float32).contiguous() if self.choice_correction else None
        self.w_up = torch.empty((E, (2 if self.gated else 1) * ff, h), dtype=run, device=device)   # gated: gate and up rows interleaved
        self.w_down = torch.empty((E, h, ff), dtype=run, device=device)
        for e in range(E):
            if self.gated:
                self.w_up[e, 0::2] = tensors[f"e{e}.gate"].to(device=device, dtype=run)
                self.w_up[e, 1::2] = tensors[f"e{e}.up"].to(device=device, dtype=run)
            else:
                self.w_up[e] = tensors[f"e{e}.up"].to(device=device, dtype=run)
            self.w_down[e] = tensors[f"e{e}.down"].to(device=device, dtype=run)
        self.up = [Linear(self.w_up[e]) for e in range(E)]
        self.down = [Linear(self.w_down[e]) for e in range(E)]
        self.shared_up = self.shared_down = None
        if self.shared_size:      # one product for the shared expert's rows and its gate's, each group padded to a multiple of 8 rows
            self.shared_gate_at = _pad8(self.shared_size)
            w = torch.zeros((self.shared_gate_at + 8, h), dtype=run, device=device)
            w[:self.shared_size] = tensors["shared.up"].to(device=device, dtype=run)
            w[self.shared_gate_at] = tensors["shared.sg"].to(device=device, dtype=run)[0]
            self.shared_up, self.shared_down = Linear(w), Linear(tensors["shared.down"].to(device=device, dtype=run).contiguous())
        # a decode step's launches depend on device memory alone when the streaming kernel takes the rows, or else when
        # the grouped product does (the per-expert products need the runs' lengths on the host)
        grouped = run == torch.bfloat16 and E <= ops.MAX_GEMM_GROUPS and h % 8 == 0 and ff % 8 == 0
        self.graph_safe = ops.moe_rows_takes(max(h, ff), run) or grouped

    def route(self, x: torch.Tensor, ctx: StepContext, scores: torch.Tensor | None = None):
        T = x.shape[0]
        chosen = ctx.empty((T, self.top), torch.int32)
        weights = ctx.empty((T, self.top), torch.float32)
        if self.routing == "table":
            ops.moe_table_route(ctx.tokens, self.table, chosen, weights, self.n_experts)
            return chosen, weights
        ops.moe_route(x, self.router, chosen, weights, self.groups, self.keep_groups, self.weight_eps, scores, self.bias,
                      score=self.score, correction=self.correction, scale=self.weight_scale)
        return chosen, weights

    def as_prompt(self, ctx: StepContext, n_tokens: int) -> bool:
        """Whether the experts' rows are gathered and multiplied as dense products (prompts), or streamed past the
        experts' weights a few rows at a time (steps of few tokens)."""
        if not ops.moe_rows_takes(max(self.hidden_size, self.intermediate_size), ctx.dtype):
            return True     # (rows too long to stage for the streaming kernel)
        return (not ctx.all_decode) and n_tokens > 64 and n_tokens * self.top >= 16 * self.n_experts

    def adds_itself(self, x, ctx: StepContext, residual):
        """The routed experts' weighted sum."""
        T = x.shape[0]
        chosen, weights = self.route(x, ctx)
        pairs = T * self.top
        offsets = ctx.empty((self.n_experts + 1,), torch.int32)
        order, place = ctx.empty((pairs,), torch.int32), ctx.empty((pairs,), torch.int32)
        ops.moe_group(chosen, self.n_experts, offsets, order, place)
        y = ctx.empty((pairs, self.intermediate_size), ctx.dtype)
        o = ctx.empty((pairs, self.hidden_size), torch.float32)
        if not self.as_prompt(ctx, T):
            ops.moe_rows(x, self.w_up, offsets, y, order=order, top=self.top, activation=self.activation,
                         gate_args=self.gate_args)
            ops.moe_rows(y, self.w_down, offsets, o)
        else:
            xs = ctx.empty((pairs, self.hidden_size), ctx.dtype)
            ops.moe_gather(x, order, xs, self.top)
            # one launch over all experts' tiles, the runs read on the device; where that kernel does not take the operands
            # (the float32 run, odd sizes) one product per expert, for which the runs' lengths come back to the host
            epilogue = ops.GATED_EPILOGUE_OF[self.activation] if self.gated else ops.EPILOGUE_SQUARED_RELU
            if not (ops.gemm_tcgen05_grouped(xs, self.w_up, offsets, y, epilogue, self.gate_args)
                    and ops.gemm_tcgen05_grouped(y, self.w_down, offsets, o)):
                bounds = offsets.tolist()
                runs = [(e, bounds[e], bounds[e + 1]) for e in range(self.n_experts) if bounds[e + 1] > bounds[e]]
                for e, lo, hi in runs:
                    if self.gated:
                        self.up[e].gated_into(xs[lo:hi], y[lo:hi], self.activation, self.gate_args)
                    else:
                        self.up[e].into(xs[lo:hi], y[lo:hi])
                if not self.gated:
                    ops.bias_act_rows(y, None, self.activation)
                for e, lo, hi in runs:
                    self.down[e].into(y[lo:hi], o[lo:hi])
        ops.moe_combine(o, place, weights, residual)

    # ---- the shared expert: rows before a last product
    def open_columns(self):
        return self.shared_size

    def take_output(self):
        weight, self.shared_down = self.shared_down.weight, None
        return weight, None

    def take_input(self):
        weight, self.shared_up = self.shared_up.weight, None
        return weight

    def rows_into(self, x, ctx: StepContext, cache, rows, writes_cache=True, mul=1.0):
        self.rows_from(self.shared_up.store(x, ctx.dtype, ctx.empty), ctx, cache, rows, writes_cache, mul)

    def rows_from(self, raw, ctx: StepContext, cache, rows, writes_cache=True, mul=1.0):
        assert mul == 1.0
        ops.bias_act_rows(raw[:, :self.shared_size], None, self.activation, out=rows, gate=raw[:, self.shared_gate_at:])

    def forward(self, x, ctx: StepContext, residual, then_norm=None):
        self.adds_itself(x, ctx, residual)
        if self.shared_size:
            rows = ctx.empty((x.shape[0], self.shared_size), ctx.dtype)
            self.rows_into(x, ctx, None, rows)
            self.shared_down.add_to(rows, residual)
        return None


register_feed_forward("routed", RoutedFeedForward)
