"""Fazezen's mechanisms alone against their formulas: product biases in every product kernel and epilogue, one product that
leaves two norms' rows, two norms in one kernel, rotation over halves on the way into the cache, results turned back,
attention within runs of positions with a silent key in every attention kernel (prompts, portions, decoding), fixed decays
(one token, runs of tokens, portions that continue a state), the feed-forward with biases, and the parallel block with
parts that keep their products to themselves."""
import math

import pytest
import torch

import plain_fazezen as P
from gpullama3.java_b200.kernels import ops

pytestmark = pytest.mark.gpu
F = torch.float64
DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])


def _close(got, want, rel, what=""):
    got, want = got.detach().cpu().to(F), want.detach().cpu().to(F)
    assert got.shape == want.shape, (what, got.shape, want.shape)
    err, scale = float((got - want).abs().max()), float(want.abs().max()) + 1e-30
    assert err <= rel * scale, f"{what}: {err:.3e} vs scale {scale:.3e}"


def _gelu_gated(s):
    return P.gelu_tanh(s[:, 0::2]) * s[:, 1::2]


def _epilogue(kind, a, w, bias, c0, silu):
    s = a.cpu().to(F) @ w.cpu().to(F).T + bias.cpu().to(F)
    if kind == "store":
        return torch.cat([P.silu(s[:, :silu]), s[:, silu:]], dim=1)
    return c0.cpu().to(F) + s if kind == "add" else _gelu_gated(s)


EPILOGUES = {"store": ops.EPILOGUE_STORE, "add": ops.EPILOGUE_RESIDUAL_ADD, "gelu": ops.EPILOGUE_GATED_GELU_TANH}


@pytest.mark.parametrize("kind", sorted(EPILOGUES))
@pytest.mark.parametrize("M, N, K", [(1, 48, 64), (5, 130, 96), (16, 40, 32), (30, 96, 64), (64, 4128, 64), (100, 64, 72), (130, 200, 64),
                                     (300, 264, 136), (520, 1032, 512), (200, 72, 4096)])
def test_biases_and_activated_columns_of_every_product(kind, M, N, K):
    torch.manual_seed(M + N)
    silu = N // 2 + 5 if kind == "store" else 0     # (a border inside every kernel's run of columns)
    g = dict(device="cuda")
    a, w = torch.randn(M, K, **g), torch.randn(N, K, **g) / K ** 0.5
    bias = torch.randn(N, **g)
    n_out = N // 2 if kind == "gelu" else N
    from gpullama3.java_b200.parts.linear import Linear

    for dtype in (torch.float32, torch.bfloat16):
        A, W = a.to(dtype), w.to(dtype)
        out_type = torch.float32 if kind == "add" else dtype
        c0 = torch.randn(M, n_out, **g).to(out_type)
        want = _epilogue(kind, A, W, bias, c0, silu)
        rel = 3e-6 if dtype == torch.float32 else 1e-2
        c = c0.clone()
        Linear(W.contiguous(), bias, silu)._run(A, c, EPILOGUES[kind])
        _close(c, want, rel, f"chosen kernel {dtype} {kind}")
        c = c0.clone()
        ops.gemm_generic(A, W, c, EPILOGUES[kind], bias=bias, silu_columns=silu)
        _close(c, want, rel, f"plain kernel {dtype} {kind}")
        if dtype == torch.bfloat16:
            variants = [dict(tile_width=t, cta_pair=-1, k_spans=1) for t in (64, 128, 256)] + [dict(cta_pair=1, tile_width=t) for t in (128, 256)]
            if kind != "gelu" and K >= 256:
                variants += [dict(k_spans=s) for s in (2, 4)]
            for v in variants:
                c = c0.clone()
                if ops.gemm_tcgen05(A, W, c, EPILOGUES[kind], bias=bias, silu_columns=silu, **v):
                    _close(c, want, rel, f"tcgen05 {v} {kind}")
            assert ops.gemm_tcgen05_status() == 0


@pytest.mark.parametrize("M, N, K", [(1, 64, 96), (7, 640, 128), (16, 96, 64), (9, 4200, 64)])
def test_one_product_leaves_two_norms(M, N, K):
    """c += a w^T + b, and the rows under two norms' weights with one set of partial sums; the next product applies the factor
    before its own bias."""
    torch.manual_seed(N)
    g = dict(device="cuda")
    a, w = torch.randn(M, K, **g).bfloat16(), (torch.randn(N, K, **g) / K ** 0.5).bfloat16()
    bias, n1, n2 = torch.randn(N, **g), 1 + 0.2 * torch.randn(N, **g), 1 + 0.2 * torch.randn(N, **g)
    c = torch.randn(M, N, **g)
    x = c.cpu().to(F) + a.cpu().to(F) @ w.cpu().to(F).T + bias.cpu().to(F)
    acts = [torch.empty(M, N, dtype=torch.bfloat16, **g) for _ in range(2)]
    parts = torch.empty(M, ops.gemm_decode_partials(M, N), **g)
    ops.gemm_decode_linked(a, w, c, ops.EPILOGUE_RESIDUAL_ADD, emit=(n1, acts[0], parts), emit_second=(n2, acts[1]), bias=bias)
    _close(c, x, 1e-5, "stream")
    _close(parts.sum(dim=1), (x * x).sum(dim=1), 1e-5, "sums of squares")
    for act, n in zip(acts, (n1, n2)):
        _close(act, x * n.cpu().to(F), 5e-3, "rows under a weight")
    if N % 32 == 0:
        w2, b2 = (torch.randn(40, N, **g) / N ** 0.5).bfloat16(), torch.randn(40, **g)
        out = torch.empty(M, 40, dtype=torch.float32, **g)
        ops.gemm_decode_linked(acts[1], w2, out, ops.EPILOGUE_STORE, row_factors=(parts, 1e-5, N), bias=b2, silu_columns=13)
        want = P.over_root_mean_square(x, 1e-5) * n2.cpu().to(F) @ w2.cpu().to(F).T + b2.cpu().to(F)
        want[:, :13] = P.silu(want[:, :13])
        _close(out, want, 1e-2, "the product behind it")


@DTYPES
@pytest.mark.parametrize("T, dim", [(3, 50), (1, 4100), (1200, 1024), (1100, 2048), (70, 640), (1030, 3072)])
def test_two_norms_in_one_kernel(dtype, T, dim):
    torch.manual_seed(dim)
    x, w1, w2 = torch.randn(T, dim, device="cuda") * 3, torch.randn(dim, device="cuda"), torch.randn(dim, device="cuda")
    outs = [torch.empty(T, dim, dtype=dtype, device="cuda") for _ in range(2)]
    ops.rmsnorm_pair(x, (w1, w2), outs, 1e-5)
    for o, w in zip(outs, (w1, w2)):
        _close(o, P.over_root_mean_square(x.cpu().to(F), 1e-5) * w.cpu().to(F), 2e-6 if dtype == torch.float32 else 5e-3)


def _pages(n_tokens, n_kv, D, dtype, order_seed=0):
    n = -(-n_tokens // 64) + 2
    k = torch.full((n, n_kv, 64, D), 3.0, dtype=dtype, device="cuda")      # (what a page holds beyond a sequence must not matter)
    v = torch.full((n, n_kv, D, 64), -5.0, dtype=dtype, device="cuda")
    perm = torch.randperm(n, generator=torch.Generator().manual_seed(order_seed))[:n - 1].to(torch.int32)
    return k, v, perm.view(1, -1).contiguous().cuda()


@DTYPES
@pytest.mark.parametrize("T", [70, 300])      # (few tokens: a warp per row; many: a CTA per token)
@pytest.mark.parametrize("d, dv, D, pairs, vpairs", [(16, 24, 32, 8, 12), (12, 20, 32, 2, 10), (64, 64, 64, 32, 32), (40, 96, 96, 5, 48), (8, 8, 16, 0, 0)])
def test_rows_turned_over_halves_on_their_way_into_the_cache(dtype, T, d, dv, D, pairs, vpairs):
    torch.manual_seed(d)
    H, G, start = 4, 2, 31
    raw = torch.randn(T, (H + G) * d + G * dv + 3, device="cuda").to(dtype)
    weight = torch.cat([1 + 0.3 * torch.randn(d), 1 + 0.3 * torch.randn(d)]).cuda()
    fk = torch.tensor(P.pair_frequencies(100.0, 2 * pairs), dtype=torch.float32) if pairs else torch.zeros(0)
    fv = torch.tensor(P.pair_frequencies(50.0, 2 * vpairs), dtype=torch.float32) if vpairs else torch.zeros(0)
    freqs = torch.cat([fk, fv]).cuda() if pairs + vpairs else None
    k_pool, v_pool, table = _pages(start + T, G, D, dtype)
    segs = ops.head_row_segments(
        ops.head_row_segment(0, H, d, 0, D, norm=1, weight_off=0, mul=0.7, half_pairs=pairs),
        ops.head_row_segment(H * d, G, d, 0, D, norm=1, weight_off=d, half_pairs=pairs, target=ops.TO_CACHE_KEYS),
        ops.head_row_segment((H + G) * d, G, dv, 0, D, half_pairs=vpairs, freq_off=pairs, target=ops.TO_CACHE_VALUES))
    q = torch.empty(T, H * D, dtype=dtype, device="cuda")
    pos = torch.arange(start, start + T, dtype=torch.int32, device="cuda")
    seq = torch.zeros(T, dtype=torch.int32, device="cuda")
    ops.head_rows(raw, q, segs, 1e-5, None, weight, cache=(pos, seq, table, k_pool, v_pool), rotary=(pos, freqs) if freqs is not None else None)
    x = torch.zeros(start + T, raw.shape[1], dtype=F)
    x[start:] = raw.cpu().to(F)      # (the plain rotation counts positions from the first row)
    tol = 1e-5 if dtype == torch.float32 else 6e-3

    def rows(off, n, size, w, f, mul=1.0):
        z = x[:, off:off + n * size].view(-1, n, size)
        if w is not None:
            z = P.over_root_mean_square(z, 1e-5) * w.cpu().to(F)
        z = torch.nn.functional.pad(P.turn_halves(z, f.to(F).tolist()) * mul, (0, D - size))
        return z[start:]

    _close(q.view(T, H, D), rows(0, H, d, weight[:d], fk, 0.7), tol, "queries")
    got_k = torch.stack([k_pool[table[0, p // 64].item(), :, p % 64] for p in range(start, start + T)])
    got_v = torch.stack([v_pool[table[0, p // 64].item(), :, :, p % 64] for p in range(start, start + T)])
    _close(got_k, rows(H * d, G, d, weight[d:], fk), tol, "keys")
    _close(got_v, rows((H + G) * d, G, dv, None, fv), tol, "values")


@DTYPES
@pytest.mark.parametrize("T, H, d, D", [(3, 5, 14, 32), (600, 4, 64, 64), (33, 2, 96, 96)])
def test_rows_turned_back(dtype, T, H, d, D):
    torch.manual_seed(T)
    x = torch.randn(T, H * D, device="cuda").to(dtype)
    wide = torch.zeros(T, H * d + 11, dtype=dtype, device="cuda")
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    f32 = torch.tensor(P.pair_frequencies(77.0, d), dtype=torch.float32)
    f = f32.to(F).tolist()
    ops.turn_back_rows(x, pos, f32.cuda(), wide[:, 5:5 + H * d], H, d, D, 1.5)
    want = P.turn_halves(x.cpu().to(F).view(T, H, D)[..., :d], f, sign=-1.0) * 1.5
    _close(wide[:, 5:5 + H * d].reshape(T, H, d), want, 4e-5 if dtype == torch.float32 else 5e-3)
    assert float(wide[:, :5].abs().max()) == 0.0 and float(wide[:, 5 + H * d:].abs().max()) == 0.0
    ops.turn_back_rows(x, pos, None, wide[:, 5:5 + H * d], H, d, D, 2.0)
    _close(wide[:, 5:5 + H * d].reshape(T, H, d), x.cpu().to(F).view(T, H, D)[..., :d] * 2.0, 5e-3)


class _Shape:
    keep_first, slopes, window, has_terms = 0, None, None, True

    def __init__(self, H, G, D, chunk, sinks):
        self.n_heads, self.n_kv_heads, self.head_dim, self.chunk, self.sinks = H, G, D, chunk, sinks

    def plan_decode(self, ctx, cache):
        from gpullama3.java_b200.parts.attention import plan_decode_attention
        return plan_decode_attention(self, ctx, cache)


@DTYPES
@pytest.mark.parametrize("H, G, D", [(4, 2, 32), (8, 1, 64), (2, 2, 96), (4, 4, 128), (20, 1, 16), (3, 1, 144)])
@pytest.mark.parametrize("chunk, sink", [(None, 0.0), (1, 0.0), (7, 0.0), (64, 0.0), (130, 1.5), (200, None)])
def test_attention_within_runs(dtype, H, G, D, chunk, sink):
    """Two sequences: one that brings many tokens behind a cached prefix, one shorter; then one token each.  One key stands
    out just inside and one just outside a run's edge, with a score far above the others."""
    from gpullama3.java_b200.cache.sequence_cache import KVView
    from gpullama3.java_b200.parts.attention import attend
    from gpullama3.java_b200.parts.base import StepContext

    torch.manual_seed(D + (chunk or 0))
    lens, starts = [300, 131], [137, 0]
    ks = [torch.randn(n, G, D) for n in lens]
    vs = [torch.randn(n, G, D) for n in lens]
    for k in ks:      # keys next to the edges of runs stand out: every query that may see them leans on them
        for j in ([] if chunk is None else [p for c in range(chunk, len(k), chunk) for p in (c - 1, c)]):
            k[j] *= 2.5
    qs = [torch.randn(n, H, D) * 1.5 for n in lens]
    per = [-(-n // 64) for n in lens]
    pool_n = sum(per) + 1
    k_pool = torch.zeros(pool_n, G, 64, D, dtype=dtype, device="cuda")
    v_pool = torch.zeros(pool_n, G, D, 64, dtype=dtype, device="cuda")
    table = torch.zeros(2, max(per), dtype=torch.int32)
    page = 1
    for s, n in enumerate(lens):
        for p in range(per[s]):
            table[s, p] = page
            lo, hi = p * 64, min(n, p * 64 + 64)
            k_pool[page, :, :hi - lo] = ks[s][lo:hi].transpose(0, 1).to(dtype).cuda()
            v_pool[page, :, :, :hi - lo] = vs[s][lo:hi].permute(1, 2, 0).to(dtype).cuda()
            page += 1
    sinks = torch.full((H,), sink, device="cuda") if sink is not None else None
    shape = _Shape(H, G, D, chunk, sinks)
    view = KVView(group=0, k=k_pool, v=v_pool, window=None)

    def want(s, lo):
        rnd = lambda z: z.to(dtype).to(F)
        k, v = (rnd(z).repeat_interleave(H // G, dim=1) for z in (ks[s], vs[s]))
        sc = torch.einsum("ihd,jhd->hij", rnd(qs[s]), k) / math.sqrt(D)
        mask = P.chunk_mask(lens[s], chunk)
        if sink is None:
            pr = torch.softmax(torch.where(mask, sc, torch.full_like(sc, -math.inf)), dim=-1)
        else:
            e = torch.where(mask, torch.exp(sc), torch.zeros_like(sc))
            pr = e / (math.exp(sink) + e.sum(dim=-1, keepdim=True))
        return torch.einsum("hij,jhd->ihd", pr, v)[lo:]

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
        out = torch.empty(T, H * D, dtype=dtype, device="cuda")
        attend(shape, q, out, ctx, ctx.page_tables[0], view)
        out = out.view(T, H, D).cpu()
        return out[:q_lens[0]], out[q_lens[0]:], st

    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    for q_lens in ([163, 131], [2, 130], [1, 1]):
        a, b, st = run(q_lens)
        _close(a, want(0, st[0]), tol, f"first sequence, {q_lens}")
        _close(b, want(1, st[1]), tol, f"second sequence, {q_lens}")
    assert ops.attention_prefill_tc_status() == 0


CASES = [  # heads, d_k, d_v, pairs, silu, decays
    (2, 16, 24, 0, True, (0.5, 0.999)), (3, 10, 9, 3, False, (0.0, 1.0, 0.9)), (2, 64, 64, 16, False, (0.97, 0.9995)),
    (1, 128, 192, 0, True, (0.99,)), (2, 128, 128, 64, False, (0.9, 0.999)), (2, 256, 40, 8, False, (0.95, 0.99)), (1, 40, 64, 20, True, (0.6,)),
    (1, 8, 33, 4, False, (0.8,))]


@DTYPES
@pytest.mark.parametrize("H, dk, dv, pairs, silu, decays", CASES)
@pytest.mark.parametrize("cut", [[(200, 1)], [(65, 64), (1, 1), (1, 2), (130, 3)], [(1, 1)] * 5 + [(64, 64)]], ids=str)
def test_fixed_decays(dtype, H, dk, dv, pairs, silu, decays, cut):
    """Two sequences through steps of the given numbers of tokens each, against the recurrence in float64: the outputs and the
    state that is left, in slots that others have used.  The bfloat16 run's operands are rounded once (the projections); what
    the recurrence does with them must be 32-bit: the bound is a hundredth of one bfloat16 rounding, unless the operands pass
    through SiLU (an activation of the projections, which is rounded: q, k and v once each)."""
    torch.manual_seed(dk + dv)
    lens = [sum(c[i] for c in cut) for i in range(2)]
    data = [[torch.randn(n, H, d).to(dtype) for d in (dk, dk, dv, dv)] for n in lens]
    freqs = torch.tensor(P.pair_frequencies(30.0, 2 * pairs), dtype=torch.float32, device="cuda") if pairs else None
    slots = torch.tensor([2, 0], dtype=torch.int32, device="cuda")
    state = torch.full((3, H * dk * dv + 4), 7.0, device="cuda")
    state[slots.long()] = 0.0
    decay = torch.tensor(decays, dtype=torch.float32, device="cuda")
    got, done_rows, at = [[], []], [[], []], [0, 0]
    scale = 0.37
    for ns in cut:
        T = sum(ns)
        cols = [torch.cat([data[i][j][at[i]:at[i] + ns[i]].reshape(ns[i], -1) for i in range(2)]) for j in range(4)]
        raw = torch.cat([torch.nn.functional.pad(c, (0, (-c.shape[1]) % 8)) for c in cols], dim=1).cuda()
        offs, o = [], 0
        for c in cols:
            offs.append(o)
            o += c.shape[1] + (-c.shape[1]) % 8
        q, k, v, g = (raw[:, o:] for o in offs)
        cu = torch.tensor([0, ns[0], T], dtype=torch.int32, device="cuda")
        pos = torch.tensor([p for i in range(2) for p in range(at[i], at[i] + ns[i])], dtype=torch.int32, device="cuda")
        single = all(n == 1 for n in ns)
        finished = None
        if ops.fixed_decay_takes(dtype, single, dk, dv):
            kw = dict(q_scale=scale, qk_silu=silu, v_silu=silu, inv_freq=freqs)
            before = state.clone()
            if ops.fixed_decay_finishes(single, dk, dv):
                wide = torch.zeros(T, H * dv + 3, dtype=dtype, device="cuda")
                finished = wide[:, 1:1 + H * dv]
                ops.fixed_decay(q, k, v, decay, state, slots, cu, pos, H, dk, dv, max(ns), finish=(finished, g, "silu", 1e-5, 0.8), **kw)
                assert float(wide[:, 0].abs().max()) == 0.0 and float(wide[:, 1 + H * dv:].abs().max()) == 0.0
                after = state.clone()
                state.copy_(before)
            out = torch.empty(T, H * dv, device="cuda")
            ops.fixed_decay(q, k, v, decay, state, slots, cu, pos, H, dk, dv, max(ns), out=out, **kw)
            if finished is not None:
                assert torch.equal(state, after)
        else:
            out = torch.empty(T, H * dv, device="cuda")
            ops.linear_scan(q, k, v, None, state, slots, cu, out, H, H, dk, dv, decay_kind=ops.DECAY_FIXED, decay_per_head=True,
                            a_log=decay, q_scale=scale, qk_silu=silu, v_silu=silu, rotary=(pos, freqs) if pairs else None)
        for i in range(2):
            rows = slice(0, ns[0]) if i == 0 else slice(ns[0], T)
            got[i].append(out[rows].cpu())
            done_rows[i].append(finished[rows].cpu() if finished is not None else None)
            at[i] += ns[i]
    assert float((state[1] - 7.0).abs().max()) == 0.0, "another sequence's state was touched"
    for i in range(2):
        act = P.silu if silu else (lambda z: z)
        q, k, v, g = (z.to(F) for z in data[i])
        q, k, v = act(q), act(k), act(v)
        if pairs:
            f = freqs.cpu().to(F).tolist()
            q, k = P.turn_halves(q, f), P.turn_halves(k, f)
        want = P.decayed_outer_sum(q * scale, k, v, [float(x) for x in decay.cpu()])
        tol = 1e-5 if dtype == torch.float32 else (8e-3 if silu else 4e-5)
        _close(torch.cat(got[i]).view(-1, H, dv), want, tol, f"outputs of sequence {i}")
        S = torch.zeros(H, dk, dv, dtype=F)
        for t in range(lens[i]):
            S = decay.cpu().to(F)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        _close(state[slots[i].item(), :H * dk * dv].view(H, dk, dv), S, tol, f"state of sequence {i}")
        done = P.over_root_mean_square(want, 1e-5) * P.silu(g) * 0.8
        a = 0
        for r, n in zip(done_rows[i], [c[i] for c in cut]):
            if r is not None:
                _close(r.view(n, H, dv), done[a:a + n], 2e-4 if dtype == torch.float32 else 2e-2, "finished heads")
            a += n


@DTYPES
@pytest.mark.parametrize("gate_first", [False, True])
@pytest.mark.parametrize("T, parts, d, weighted", [(5, 1, 120, True), (3, 2, 512, False), (70, 1, 2048, True), (9, 1, 4100, True), (4, 3, 515, True)])
def test_gated_norms_with_and_without_a_weight(dtype, gate_first, T, parts, d, weighted):
    torch.manual_seed(d)
    x, w = torch.randn(T, parts * d, device="cuda"), torch.randn(parts * d, device="cuda")
    gate = torch.randn(T, parts * d + 4, device="cuda").to(dtype)[:, :parts * d]
    for off in (0, 3):
        wide = torch.zeros(T, parts * d + 8, dtype=dtype, device="cuda")
        ops.gated_rmsnorm(x, w if weighted else None, gate, wide[:, off:off + parts * d], parts, d, 1e-5, "silu", gate_first=gate_first, mul=0.6)
        z, g = (a.cpu().to(F).view(T, parts, d) for a in (x, gate))
        g = P.silu(g)
        n = P.over_root_mean_square(z * g if gate_first else z, 1e-5) * (w.cpu().to(F).view(parts, d) if weighted else 1.0) * 0.6
        _close(wide[:, off:off + parts * d].reshape(T, parts, d), n if gate_first else n * g, 3e-6 if dtype == torch.float32 else 6e-3)
        assert float(wide[:, :off].abs().sum()) == 0.0 and float(wide[:, off + parts * d:].abs().sum()) == 0.0


def test_parts_that_keep_their_products_run_one_after_the_other(session_tmp):
    """The parallel block takes any mixer and feed-forward: a part that does not give its last product away is run as it is,
    on inputs made before anything joins the stream."""
    from gpullama3.java_b200.parts.parallel import ParallelBlock
    from gpullama3.java_b200.parts.base import FeedForward, Mixer
    from gpullama3.java_b200.parts.norm import RMSNorm

    class AddsTwice(Mixer):
        def forward(self, x, ctx, cache, residual, writes_cache=True):
            residual += 2 * x

    class AddsThrice(FeedForward):
        def forward(self, x, ctx, residual):
            residual += 3 * x

    norms = [RMSNorm(40, 1e-5, offset=1.0) for _ in range(2)]
    block = ParallelBlock(AddsTwice(), norms[0], AddsThrice(), norms[1])
    ws = [0.3 * torch.randn(40) for _ in range(2)]
    for n, w in zip(norms, ws):
        n.load({"weight": w}, torch.float32, torch.device("cuda"))
    block.after_load()
    assert block.out is None
    x = torch.randn(6, 40, device="cuda")

    class Ctx:
        dtype = torch.float32
        all_decode = False
        empty = staticmethod(lambda shape, dtype: torch.empty(tuple(shape), dtype=dtype, device="cuda"))

    y = x.clone()
    block.forward(y, Ctx(), None)
    n = [P.rms_norm_around_zero(x.cpu().to(F), w.to(F), 1e-5) for w in ws]
    _close(y, x.cpu().to(F) + 2 * n[0] + 3 * n[1], 1e-5)
