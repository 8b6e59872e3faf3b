"""Zanezen's mechanisms alone against their formulas: soft caps, sinks and gates in every attention kernel (prompts, portions,
decoding), a factor on the turned pairs alone, the matrix memory (one token, runs of tokens, portions that continue a memory, gates
at their caps), routing by sigmoid scores with a correction of the choice, experts without a gate in every product, and the shared
expert's gated rows."""
import math

import pytest
import torch

import plain_zanezen as P
from gpullama3.java_b200.kernels import ops

pytestmark = pytest.mark.gpu
F = torch.float64
DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])


def _close(got, want, rel, what=""):
    got, want = got.detach().cpu().to(F), want.detach().cpu().to(F)
    assert got.shape == want.shape, (what, got.shape, want.shape)
    assert torch.isfinite(got).all(), what
    err, scale = float((got - want).abs().max()), float(want.abs().max()) + 1e-30
    assert err <= rel * scale, f"{what}: {err:.3e} vs scale {scale:.3e}"


class _Shape:
    keep_first, slopes, window, chunk, has_terms = 0, None, None, None, True

    def __init__(self, H, G, D, softcap, sinks):
        self.n_heads, self.n_kv_heads, self.head_dim, self.softcap, self.sinks = H, G, D, softcap, sinks

    def plan_decode(self, ctx, cache):
        from gpullama3.java_b200.parts.attention import plan_decode_attention
        return plan_decode_attention(self, ctx, cache)


@DTYPES
@pytest.mark.parametrize("H, G, D", [(4, 2, 32), (8, 1, 64), (2, 2, 96), (4, 4, 128), (20, 1, 16), (12, 1, 128), (3, 1, 144), (76, 2, 64), (40, 20, 128)])
@pytest.mark.parametrize("softcap, sink, gated", [(2.0, None, False), (30.0, 1.5, True), (None, 0.7, True), (0.5, 2.0, False)])
def test_soft_caps_sinks_and_gates(dtype, H, G, D, softcap, sink, gated):
    """Two sequences: one that brings many tokens behind a cached prefix, one shorter; then a portion of two and many tokens, then
    one token each.  Some keys have scores far beyond the cap, on both sides; the sinks differ from head to head."""
    from gpullama3.java_b200.cache.sequence_cache import KVView
    from gpullama3.java_b200.parts.attention import attend
    from gpullama3.java_b200.parts.base import StepContext

    torch.manual_seed(D + H)
    lens, starts = [300, 131], [137, 0]
    ks = [torch.randn(n, G, D) for n in lens]
    vs = [torch.randn(n, G, D) for n in lens]
    for k in ks:
        k[7] *= 6.0
        k[60:130:13] *= 3.0
    qs = [torch.randn(n, H, D) * 1.5 for n in lens]
    gs = [torch.randn(n, H) * 2 for n in lens]
    per = [-(-n // 64) for n in lens]
    k_pool = torch.full((sum(per) + 1, G, 64, D), float("nan"), dtype=dtype, device="cuda")    # (what a page holds beyond a sequence must not matter)
    v_pool = torch.full((sum(per) + 1, G, D, 64), float("nan"), dtype=dtype, device="cuda")
    table = torch.zeros(2, max(per), dtype=torch.int32)
    page = 1
    for s, n in enumerate(lens):
        for p in range(per[s]):
            table[s, p] = page
            lo, hi = p * 64, min(n, p * 64 + 64)
            k_pool[page, :, :hi - lo] = ks[s][lo:hi].transpose(0, 1).to(dtype).cuda()
            v_pool[page, :, :, :hi - lo] = vs[s][lo:hi].permute(1, 2, 0).to(dtype).cuda()
            page += 1
    sinks = (sink + 0.1 * torch.arange(H)).cuda() if sink is not None else None
    shape = _Shape(H, G, D, softcap, sinks)
    view = KVView(group=0, k=k_pool, v=v_pool, window=None)

    def want(s, lo):
        rnd = lambda z: z.to(dtype).to(F)
        k, v = (rnd(z).repeat_interleave(H // G, dim=1) for z in (ks[s], vs[s]))
        sc = P.soft_cap(torch.einsum("ihd,jhd->hij", rnd(qs[s]), k) / math.sqrt(D), softcap)
        pr = P.softmax_over_visible(sc, P.causal_mask(lens[s]), sinks.cpu().to(F) if sink is not None else None)
        o = torch.einsum("hij,jhd->ihd", pr, v)
        return (o * torch.sigmoid(rnd(gs[s]))[:, :, None] if gated else o)[lo:]

    def run(q_lens):
        st = [n - q for n, q in zip(lens, q_lens)]
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
        T = sum(q_lens)
        ctx = StepContext(dtype=dtype, device=torch.device("cuda"), n_seqs=2, n_tokens=T, slots=[0, 1], start_pos=st, q_lens=q_lens,
                          all_decode=all(q == 1 for q in q_lens), max_q_len=max(q_lens), max_kv_len=max(lens), tokens=i32([0] * T),
                          positions=i32([p for s, q in zip(st, q_lens) for p in range(s, s + q)]),
                          seq_ids=i32([i for i, q in enumerate(q_lens) for _ in range(q)]), cu_seqlens=i32([0, q_lens[0], T]),
                          kv_lens=i32(lens), slots_dev=i32([0, 1]), page_tables=[table.cuda()], kv_capacity=[max(per) * 64])
        q = torch.cat([qs[i][st[i]:].reshape(q_lens[i], H * D) for i in range(2)]).to(dtype).cuda().contiguous()
        wide = torch.cat([torch.zeros(T, 5), torch.cat([gs[i][st[i]:] for i in range(2)])], dim=1).to(dtype).cuda()
        out = torch.empty(T, H * D, dtype=dtype, device="cuda")
        attend(shape, q, out, ctx, ctx.page_tables[0], view, wide[:, 5:] if gated else None)
        out = out.view(T, H, D).cpu()
        return out[:q_lens[0]], out[q_lens[0]:], st

    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    wants = [want(s, 0) for s in range(2)]
    for q_lens in ([300, 131], [163, 131], [2, 130], [1, 1]):
        a, b, st = run(q_lens)
        _close(a, wants[0][st[0]:], tol, f"first sequence, {q_lens}")
        _close(b, wants[1][st[1]:], tol, f"second sequence, {q_lens}")
    assert ops.attention_prefill_tc_status() == 0


@DTYPES
@pytest.mark.parametrize("T", [70, 300])      # (few tokens: a warp per row; many: a CTA per tile of tokens)
@pytest.mark.parametrize("d, pairs", [(24, 8), (16, 8), (64, 12)])
def test_the_factor_on_turned_pairs_leaves_the_other_numbers(dtype, T, d, pairs):
    torch.manual_seed(d)
    H, start = 3, 0
    raw = torch.randn(T, H * d, device="cuda").to(dtype)
    f32 = torch.tensor(P.pair_frequencies(100.0, 2 * pairs)[0], dtype=torch.float32)
    segs = ops.head_row_segments(ops.head_row_segment(0, H, d, 0, d + 8, mul=0.7, half_pairs=pairs, turn_mul=1.3))
    q = torch.empty(T, H * (d + 8), dtype=dtype, device="cuda")
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    ops.head_rows(raw, q, segs, rotary=(pos, f32.cuda()))
    x = raw.cpu().to(F).view(T, H, d)
    want = torch.nn.functional.pad(P.turn_halves(x, f32.to(F).tolist(), 1.3) * 0.7, (0, 8))
    _close(q.view(T, H, d + 8), want, 4e-5 if dtype == torch.float32 else 6e-3)


MEMORIES = [  # heads, d_k, d_v, cap, forget bias, input bias
    (2, 16, 24, 15.0, 3.0, 0.0), (3, 10, 9, 2.0, 1.0, 1.0), (2, 64, 64, 8.0, 6.0, -2.0), (1, 128, 192, 15.0, 4.0, 0.0),
    (2, 64, 128, 5.0, 0.0, 3.0), (1, 256, 40, 15.0, 5.0, -3.0), (1, 400, 33, 10.0, 4.0, 0.0), (2, 48, 300, 15.0, 2.0, 0.0), (1, 8, 4, 1.0, 9.0, -9.0)]


@DTYPES
@pytest.mark.parametrize("H, dk, dv, cap, fb, ib", MEMORIES)
@pytest.mark.parametrize("cut", [[(200, 1)], [(65, 64), (1, 1), (1, 2), (130, 3)], [(1, 1)] * 5 + [(64, 64)], [(2300, 100)]], ids=str)
def test_matrix_memory(dtype, H, dk, dv, cap, fb, ib, cut):
    """Two sequences through steps of the given numbers of tokens each, against the recurrence in float64: the read-outs, the memory,
    its key sum (every copy) and its maximum (every copy), in slots that others have used.  The gates' logits are wide: some tokens
    meet the caps on either side.  The bfloat16 run's operands are rounded once (the projections); what the recurrence does with them
    must be 32-bit."""
    torch.manual_seed(dk + dv)
    lens = [sum(c[i] for c in cut) for i in range(2)]
    data = [[torch.randn(n, H, d).to(dtype) for d in (dk, dk, dv, dv)] + [(torch.randn(n, H) * 4).to(dtype) for _ in range(2)] for n in lens]
    b_i, b_f = (torch.randn(H) + ib).cuda(), (torch.randn(H) + fb).cuda()
    weight = (1 + 0.3 * torch.randn(H * dv)).cuda()
    slots = torch.tensor([2, 0], dtype=torch.int32, device="cuda")
    n_state, copies = ops.matrix_memory_state(H, dk, dv), ops.matrix_memory_copies(dv)
    state = torch.full((3, n_state + 4), 7.0, device="cuda")
    state[slots.long()] = 0.0
    got, done_rows, at, scale = [[], []], [[], []], [0, 0], 0.37
    for ns in cut:
        T = sum(ns)
        cols = [torch.cat([data[i][j][at[i]:at[i] + ns[i]].reshape(ns[i], -1) for i in range(2)]) for j in range(6)]
        raw = torch.cat([torch.nn.functional.pad(c, (0, (-c.shape[1]) % 8)) for c in cols], dim=1).cuda()
        offs, o = [], 0
        for c in cols:
            offs.append(o)
            o += c.shape[1] + (-c.shape[1]) % 8
        q, k, v, g, zi, zf = (raw[:, o:] for o in offs)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
        args = (q, k, v, (zi, zf, b_i, b_f), cap, state, slots, i32([0] * ns[0] + [1] * ns[1]), i32([0, ns[0], T]), H, dk, dv, max(ns))
        single, finished = all(n == 1 for n in ns), None
        if ops.matrix_memory_finishes(dtype, single, dk, dv):
            before = state.clone()
            wide = torch.zeros(T, H * dv + 3, dtype=dtype, device="cuda")
            finished = wide[:, 1:1 + H * dv]
            ops.matrix_memory(*args, q_scale=scale, finish=(finished, g, "sigmoid", 1e-5, weight))
            assert float(wide[:, 0].abs().max()) == 0.0 and float(wide[:, 1 + H * dv:].abs().max()) == 0.0
            after = state.clone()
            state.copy_(before)
        out = torch.empty(T, H * dv, device="cuda")
        ops.matrix_memory(*args, q_scale=scale, out=out)
        if finished is not None:
            assert torch.equal(state, after)
        for i in range(2):
            rows = slice(0, ns[0]) if i == 0 else slice(ns[0], T)
            got[i].append(out[rows].cpu())
            done_rows[i].append(finished[rows].cpu() if finished is not None else None)
            at[i] += ns[i]
    assert float((state[1] - 7.0).abs().max()) == 0.0, "another sequence's memory was touched"
    tol = 2e-5 if dtype == torch.float32 else 2e-4
    for i in range(2):
        q, k, v, g, zi, zf = (z.to(F) for z in data[i])
        li = P.soft_cap(zi + b_i.cpu().to(F), cap)
        lf = torch.nn.functional.logsigmoid(P.soft_cap(zf + b_f.cpu().to(F), cap))
        want, S, n, m = P.matrix_memory(q * scale, k, v, li, lf)
        # a divisor is |n . q| at the least: where that sum is small by cancellation, its rounding is not
        terms = P.matrix_memory(q.abs() * scale, k.abs(), torch.ones(lens[i], H, 1, dtype=F), li, lf)
        big = terms[0][..., 0]
        out = torch.cat(got[i]).view(-1, H, dv).to(F)
        assert torch.isfinite(out).all()
        err = (out - want).abs().amax(dim=-1)
        bound = tol * (want.abs().amax(dim=-1) + 1.0) * _cancellation(q * scale, k, li, lf)
        assert bool((err <= bound).all()), (i, float((err / bound).max()), big.shape)
        mine = state[slots[i].item()]
        _close(mine[:H * dk * dv].view(H, dk, dv), S, tol, f"memory of sequence {i}")
        ns_ = mine[H * dk * dv:H * dk * (dv + copies)].view(H, copies, dk)
        ms = mine[H * dk * (dv + copies):H * (dk * (dv + copies) + copies)].view(H, copies)
        for c in range(copies):
            _close(ns_[:, c], n, tol, f"key sum of sequence {i}, copy {c}")
            assert float((ms[:, c].cpu().to(F) - m).abs().max()) <= 2e-5 * (1 + float(m.abs().max())), (i, c)
        done = P.over_root_mean_square(out, 1e-5) * weight.cpu().to(F).view(H, dv) * torch.sigmoid(g)
        a = 0
        for r, nt in zip(done_rows[i], [c[i] for c in cut]):
            if r is not None:
                _close(r.view(nt, H, dv), done[a:a + nt], 3e-4 if dtype == torch.float32 else 2e-2, "finished heads")
            a += nt


def _cancellation(q, k, li, lf):
    """Per token and head: the sum of the magnitudes behind n . q over the divisor."""
    T, H, d = q.shape
    n, m, out = torch.zeros(H, d, dtype=F), torch.zeros(H, dtype=F), []
    size = torch.zeros(H, d, dtype=F)
    for t in range(T):
        new = torch.maximum(lf[t] + m, li[t])
        keep, take = torch.exp(lf[t] + m - new), torch.exp(li[t] - new)
        m = new
        n, size = keep[:, None] * n + take[:, None] * k[t], keep[:, None] * size + take[:, None] * k[t].abs()
        out.append(torch.clamp((size * q[t].abs()).sum(-1) / (torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6), min=1.0))
    return torch.stack(out)


@DTYPES
@pytest.mark.parametrize("T, width, E, top, scale", [(1, 64, 7, 3, 1.0), (33, 100, 16, 4, 2.0), (5, 40, 40, 32, 0.5), (9, 48, 3, 3, 1.5), (300, 256, 64, 6, 2.5)])
def test_sigmoid_scores_with_a_correction_of_the_choice(dtype, T, width, E, top, scale):
    torch.manual_seed(E)
    h, W = torch.randn(T, width, device="cuda").to(dtype), {"router": torch.randn(E, width) / width ** 0.5, "correction": torch.randn(E) * 2 - 1.5}
    chosen = torch.empty(T, top, dtype=torch.int32, device="cuda")
    weights, scores = torch.empty(T, top, device="cuda"), torch.empty(T, E, device="cuda")
    ops.moe_route(h, W["router"].cuda(), chosen, weights, 1, 1, 1e-20, scores, score="sigmoid", correction=W["correction"].cuda(), scale=scale)
    W = {k: v.to(F) for k, v in W.items()}
    ref, w, margin = P.route(h.cpu().to(F), W, "", {"top": top, "scale": scale})
    sure = margin > 1e-5
    assert float(sure.to(F).mean()) > 0.9
    a, b = torch.sort(chosen.cpu().long(), dim=1), torch.sort(ref, dim=1)
    assert torch.equal(a.values[sure], b.values[sure])
    _close(torch.gather(weights.cpu(), 1, a.indices)[sure], torch.gather(w, 1, b.indices)[sure], 1e-5)
    _close(scores, torch.sigmoid(h.cpu().to(F) @ W["router"].T), 1e-5)
    if top < E and T > 5:      # the correction matters: without it other experts would be chosen
        other = P.route(h.cpu().to(F), {**W, "correction": torch.zeros(E, dtype=F)}, "", {"top": top, "scale": scale})[0]
        assert not torch.equal(torch.sort(other, dim=1).values, b.values)


@DTYPES
@pytest.mark.parametrize("T, width, ff, E, top", [(3, 64, 32, 5, 2), (40, 50, 14, 7, 3), (150, 64, 72, 4, 2), (300, 128, 1032, 6, 2), (1, 96, 64, 16, 4)])
def test_experts_without_a_gate_and_the_shared_one(dtype, T, width, ff, E, top):
    """The routed feed-forward by itself: few tokens past streamed weights, many through the grouped product or expert by expert."""
    from gpullama3.java_b200.parts.base import StepContext
    from gpullama3.java_b200.parts.routed_feed_forward import RoutedFeedForward

    torch.manual_seed(T)
    shared = 24
    part = RoutedFeedForward(width, ff, E, top, activation="relu_squared", score="sigmoid", choice_correction=True, weight_scale=1.7,
                             shared_size=shared)
    W = {n: torch.randn(s.shape) / s.shape[-1] ** 0.5 for n, s in part.parameters().items()}
    W["correction"] = torch.randn(E)
    W = {n: w.to(torch.bfloat16) for n, w in W.items()}
    part.load(W, dtype, torch.device("cuda"))
    x = torch.randn(T, width).to(dtype)

    class Ctx:
        n_tokens, all_decode = T, T == 1
        empty = staticmethod(lambda shape, dt: torch.empty(tuple(shape), dtype=dt, device="cuda"))
    Ctx.dtype = dtype
    residual = torch.randn(T, width, device="cuda")
    before = residual.cpu().to(F)
    part.forward(x.cuda(), Ctx(), residual)
    W64 = {n: w.to(F) for n, w in W.items()}
    mlp = {"router": {"experts": E, "top": top, "scale": 1.7}, "shared": {"ff": shared}}
    margins = []
    P._MARGINS[0] = margins
    want = P.mixture(x.to(F), W64, "", mlp)
    P._MARGINS[0] = None
    sure = margins[0] > 1e-5
    _close((residual.cpu().to(F) - before)[sure], want[sure], 2e-5 if dtype == torch.float32 else 2e-2)
    assert ops.gemm_tcgen05_status() == 0


@DTYPES
@pytest.mark.parametrize("T, n", [(3, 40), (70, 256), (5, 13)])
def test_activated_rows_times_a_gate_of_one_number(dtype, T, n):
    torch.manual_seed(n)
    u = torch.randn(T, n + 8, device="cuda").to(dtype)
    wide = torch.zeros(T, n + 16, dtype=dtype, device="cuda")
    for off in (0, 8, 3):
        wide.zero_()
        ops.bias_act_rows(u[:, :n], None, out=wide[:, off:off + n], gate=u[:, n:])
        want = P.squared_relu(u[:, :n].cpu().to(F)) * torch.sigmoid(u[:, n:n + 1].cpu().to(F))
        _close(wide[:, off:off + n], want, 2e-6 if dtype == torch.float32 else 5e-3)
        assert float(wide[:, :off].abs().sum()) == 0.0 and float(wide[:, off + n:].abs().sum()) == 0.0


@DTYPES
@pytest.mark.parametrize("T, H, n, k", [(1, 3, 128, 96), (8, 20, 32, 128), (70, 2, 40, 24), (200, 4, 130, 56), (65, 5, 11, 8), (300, 1, 300, 512), (40, 3, 9, 14)])
def test_products_per_head(dtype, T, H, n, k):
    """Every kernel behind ``gemm_per_head``: sizes on and off the tensor-core kernel's grid, results in columns of a wider buffer."""
    torch.manual_seed(n)
    a, w = torch.randn(T, H * k, device="cuda").to(dtype), (torch.randn(H, n, k, device="cuda") / k ** 0.5).to(dtype)
    want = torch.einsum("thk,hnk->thn", a.cpu().to(F).view(T, H, k), w.cpu().to(F)).reshape(T, H * n)
    for off in (0, 8, 3):
        wide = torch.zeros(T, H * n + 16, dtype=dtype, device="cuda")
        ops.gemm_per_head(a, w, wide[:, off:off + H * n])
        _close(wide[:, off:off + H * n], want, 3e-6 if dtype == torch.float32 else 6e-3)
        assert float(wide[:, :off].abs().sum()) == 0.0 and float(wide[:, off + H * n:].abs().sum()) == 0.0
