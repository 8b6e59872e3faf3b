"""Keys at the edges of Fazezen's runs of positions (the last key of the run before, the first of the query's own, in prompts
and in decoding, runs shorter than a page and longer than two), keys far back in a long run with peaked scores, page
borders, the first tokens of a sequence, the further key without a value, positions (of keys, of values, of the retention's
keys), slow decays over many runs of the prompt kernels, and long decoding.  Each test first shows on the plain
implementation that the thing it probes moves the logits by far more than the tolerance, so that an engine that got it
wrong could not pass.  The run model's score scale is small: its attention is nearly flat, so every visible key carries
weight and the edge key cannot hide behind a peak; the far-key model's is large, so that single far keys carry the result."""
import copy

import pytest
import torch

import plain_fazezen
from conftest import random_prompts
from fazezen_helpers import _left, _lig, _par, _rec, _rot, assert_logits, make_fazezen_dir, plain_inputs

pytestmark = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])

RUNS = {
    "architecture": "Fazezen", "vocab": 64, "width": 32, "norm": {"eps": 1e-6}, "initializer_range": 0.15,
    "layers": [
        _par(_left(2, 1, 16, 32, 0.05, 17, _rot(100.0, 8)), _rec(8, 16, (0.9, 0.5), _rot(50.0, 8)), 1.5, 0.3, 48),
        _par(_left(3, 1, 32, 16, 0.05, 140, _rot(500.0, 32)), _rec(16, 8, (0.7,), _rot(50.0, 4)), 2.0, 0.2),
    ],
}
FAR = {
    "architecture": "Fazezen", "vocab": 64, "width": 32, "norm": {"eps": 1e-6}, "initializer_range": 0.15,
    "layers": [
        _par(_left(2, 2, 64, 48, 0.9, 660, _rot(3000.0, 64, (8.0, 1.0, 4.0, 128))), _rec(16, 16, (0.6, 0.9), _rot(100.0, 16)), 1.4, 0.3, 48),
        _lig(16, 24, (0.8, 0.5)),
    ],
}
SLOW = {
    "architecture": "Fazezen", "vocab": 64, "width": 32, "norm": {"eps": 1e-6}, "initializer_range": 0.15,
    "layers": [
        _lig(16, 16, (0.9995, 0.99), 48),
        _par(_left(2, 1, 16, 16, 0.3, 20, _rot(100.0, 16)), _rec(32, 24, (0.9998, 0.995, 0.9), _rot(20000.0, 32)), 0.4, 1.6),
    ],
}


def _run(model_dir, dtype, tokens, prompt_len, chunk=None):
    """Logits at every position: the first ``prompt_len`` tokens as a prompt (in portions of ``chunk``), the rest one
    token a step."""
    from gpullama3.java_b200.engine.step import SequenceInput, StepFunction
    from gpullama3.java_b200.engine.trace import load_model

    model = load_model(model_dir, dtype)
    cache = model.new_cache(64 * (len(tokens) // 64 + 2))
    step = StepFunction(model, cache)
    slot = cache.acquire()
    out, at = [], 0
    while at < len(tokens):
        n = 1 if at >= prompt_len else min(chunk or prompt_len, prompt_len - at)
        out.append(step([SequenceInput(slot, tokens[at:at + n], list(range(n)))]).cpu().clone())
        at += n
    cache.release(slot)
    cache.check_invariants()
    return torch.cat(out)


def _moved(a, b, scale):
    """Per position: how far two sets of logits are apart, in units of the float32 tolerance."""
    return (a - b).abs().amax(dim=1) / (5e-5 * scale)


@DTYPES
@pytest.mark.parametrize("prompt_len, chunk", [(330, None), (150, None), (150, 7), (3, None)])
def test_runs_in_prompts_and_in_decoding(session_tmp, dtype, prompt_len, chunk):
    d = make_fazezen_dir(session_tmp, RUNS, seed=2)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [330], seed=3)[0]
    ref = plain_fazezen.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())
    for layer, size in ((0, 17), (1, 140)):
        # a mask that lets the query see one key of the run before, or hides the first of its own
        for shift in (1, -1):
            whole = plain_fazezen.chunk_mask

            def shifted(T, s, _size=size, _shift=shift):
                m = whole(T, s)
                if s != _size:
                    return m
                i = torch.arange(T)
                first = torch.clamp(i - i % s - _shift, min=0)
                return (i[None, :] <= i[:, None]) & (i[None, :] >= first[:, None]) | torch.eye(T, dtype=torch.bool)

            plain_fazezen.chunk_mask = shifted
            try:
                other = plain_fazezen.forward(cfg, weights, tokens)
            finally:
                plain_fazezen.chunk_mask = whole
            moved = _moved(other, ref, scale)[size + 1:]
            assert float((moved > 8).float().mean()) > 0.8, (layer, shift, moved.median())
    assert_logits(_run(d, dtype, tokens, prompt_len, chunk), ref, dtype, f"runs, prompt of {prompt_len}")


@DTYPES
@pytest.mark.parametrize("prompt_len, chunk", [(700, None), (520, 130), (64, None)])
def test_far_keys_over_many_pages(session_tmp, dtype, prompt_len, chunk):
    """A run of 660 positions: eleven pages of keys with peaked scores; behind it a new run begins inside a page."""
    d = make_fazezen_dir(session_tmp, FAR, seed=4)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [700], seed=5)[0]
    ref = plain_fazezen.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())
    hidden = copy.deepcopy(cfg)
    hidden["layers"][0]["mixer"]["left"]["mask"]["size"] = 330          # attention that cannot see far back
    moved = _moved(plain_fazezen.forward(hidden, weights, tokens), ref, scale)[331:650]
    assert float((moved > 20).float().mean()) > 0.9, moved.median()
    got = _run(d, dtype, tokens, prompt_len, chunk)
    assert_logits(got, ref, dtype, f"far keys, prompt of {prompt_len}")
    assert_logits(got[:4], ref[:4], dtype, "the first tokens")
    edges = [63, 64, 65, 127, 128, 129, 191, 192, 193, 659, 660, 661]
    assert_logits(got[edges], ref[edges], dtype, "positions at the borders of pages and of the run")


@DTYPES
def test_positions_the_silent_key_and_the_factors(session_tmp, dtype):
    """What the plain implementation loses when a mechanism is changed, the engine must have."""
    d = make_fazezen_dir(session_tmp, SLOW, seed=6)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [150], seed=7)[0]
    ref = plain_fazezen.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())

    def differs(what, other, least=0.9):
        moved = _moved(other, ref, scale)[4:]
        assert float((moved > 20).float().mean()) > least, (what, moved.median())

    for path, value in ((("left", "rot", "base"), 40.0), (("left", "rot", "dims"), 8), (("left", "scale"), 0.36),
                        (("right", "rot", "base"), 500.0), (("right", "rot", "dims"), 16), (("left_scale",), 0.8),
                        (("right_scale",), 1.2), (("right", "decay"), [0.9, 0.995, 0.9998])):
        c2 = copy.deepcopy(cfg)
        at = c2["layers"][1]["mixer"]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        differs(path, plain_fazezen.forward(c2, weights, tokens))
    # the pairs of the values: what the result is when they are cached as they are
    turn = plain_fazezen.turn_halves
    calls = []

    def without_values(x, freqs, sign=1.0):
        calls.append(x.shape[1:])
        return x if (sign < 0 or (len(calls) - 1) % 6 in (2,)) else turn(x, freqs, sign)   # q, k, v, o back, q, k of a layer

    plain_fazezen.turn_halves = without_values
    try:
        differs("values turned", plain_fazezen.forward(cfg, weights, tokens))
    finally:
        plain_fazezen.turn_halves = turn
    soft = plain_fazezen.softmax_with_silent_key
    plain_fazezen.softmax_with_silent_key = lambda s, m: torch.softmax(torch.where(m, s, torch.full_like(s, -float("inf"))), dim=-1)
    try:
        differs("the silent key", plain_fazezen.forward(cfg, weights, tokens), 0.6)   # (late in a run its weight is one of twenty)
    finally:
        plain_fazezen.softmax_with_silent_key = soft
    for name, change in (("l0.mlp.gate.b", 0.0), ("l0.mlp.up.b", 0.0), ("l0.mlp.down.b", 0.0), ("embed.norm", 0.0), ("l0.norm2", 0.0)):
        differs(name, plain_fazezen.forward(cfg, {n: t * (change if n == name else 1.0) for n, t in weights.items()}, tokens))
    assert_logits(_run(d, dtype, tokens, 90, 31), ref, dtype, "mechanisms")


@DTYPES
@pytest.mark.parametrize("prompt_len, chunk", [(600, None), (590, 65), (450, None)])
def test_slow_decays_over_many_runs(session_tmp, dtype, prompt_len, chunk):
    """Decays so slow that the state at position 600 still holds the first tokens: a state lost at any border shows."""
    d = make_fazezen_dir(session_tmp, SLOW, seed=8)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [600], seed=9)[0]
    ref = plain_fazezen.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())
    other = plain_fazezen.forward(cfg, weights, random_prompts(cfg["vocab"], [40], seed=10)[0] + tokens[40:])
    moved = _moved(other, ref, scale)[100:]
    assert float((moved > 20).float().mean()) > 0.9, moved.median()
    assert_logits(_run(d, dtype, tokens, prompt_len, chunk), ref, dtype, "slow decays")


@DTYPES
def test_long_decoding(session_tmp, dtype):
    """Four tokens of prompt, then 400 decoded one by one: runs of positions end and begin among decoded tokens, pages fill
    and are let go of, and every step reads the state the step before it left."""
    d = make_fazezen_dir(session_tmp, RUNS, seed=8)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [404], seed=9)[0]
    ref = plain_fazezen.forward(cfg, weights, tokens)
    assert_logits(_run(d, dtype, tokens, 4), ref, dtype, "long decoding")
