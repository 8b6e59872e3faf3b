"""Keys far back over many pages (maps with peaked scores, a latent row), page borders, the first tokens of a sequence, memories that
still hold the first tokens after hundreds, gates at their caps, convolutions across the cuts of a prompt, long decoding, and every
constant and optional mechanism.  Each test first shows on the plain implementation that the thing it probes moves the logits by far
more than the tolerance, so that an engine that got it wrong could not pass."""
import copy

import pytest
import torch

import plain_zanezen as P
from conftest import random_prompts
from zanezen_helpers import _model, _rot, assert_logits, att, dense, lat, make_zanezen_dir, mem, moe, plain_inputs

pytestmark = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])

FAR = _model(64, 32, 1e-6, 0.2, 6.0, 0.7, [
    att(2, 1, 32, 40, 0.9, 0.3, 3, 25.0, _rot(3000.0, 16, (4.0, 64, 8.0, 1.0)), dense(48)),
    lat(3, 24, 8, 16, 24, 0.9, 500.0),
])
SLOW = _model(64, 32, 1e-6, 0.15, 5.0, 0.8, [
    mem(2, 16, 24, 12.0, dense(40)),
    mem(3, 8, 16, 12.0),
])
MIX = _model(64, 32, 1e-5, 0.2, 4.0, 0.65, [
    mem(2, 12, 20, 1.5, moe(24, 6, 2, 1.8, 20)),
    att(4, 2, 16, 24, 0.5, 0.35, 4, 1.2, _rot(200.0, 8, (4.0, 64, 8.0, 1.0)), dense(40)),
    lat(4, 12, 6, 16, 18, 0.6, 80.0),
])


def _slow(tensors):
    for n, t in tensors.items():
        if n.endswith("mix.f.b"):
            tensors[n] = torch.linspace(4.5, 8.0, t.numel())
        if n.endswith("mix.i.b"):
            tensors[n] = torch.linspace(-2.0, 0.5, t.numel())
        if n.endswith(("mix.f", "mix.i")):
            tensors[n] = t * 2.0


def _closed(tensors):
    for n, t in tensors.items():
        if n.endswith("mix.i.b"):
            tensors[n] = torch.linspace(-7.5, -6.0, t.numel())
        if n.endswith("mix.f.b"):
            tensors[n] = torch.linspace(1.0, 5.0, t.numel())


def _wide_gates(tensors):
    for n, t in tensors.items():
        if n.endswith(("mix.f", "mix.i")):
            tensors[n] = t * 4.0
        if n.endswith("sink"):
            tensors[n] = torch.linspace(2.5, 5.0, t.numel())


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
@pytest.mark.parametrize("prompt_len, chunk", [(700, None), (520, 130), (520, 67), (64, None)])
def test_far_keys_over_many_pages(session_tmp, dtype, prompt_len, chunk):
    d = make_zanezen_dir(session_tmp, FAR, seed=4)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [700], seed=5)[0]
    ref = P.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())
    whole = P.causal_mask
    for layer in (0, 1):       # the layer cannot see further back than 250 positions
        calls = []

        def near(T):
            calls.append(T)
            i = torch.arange(T)
            m = whole(T)
            return m & (i[:, None] - i[None, :] < 250) if len(calls) - 1 == layer else m

        P.causal_mask = near
        try:
            moved = _moved(P.forward(cfg, weights, tokens), ref, scale)[300:]
        finally:
            P.causal_mask = whole
        assert float((moved > 20).float().mean()) > 0.9, (layer, moved.median())
    got = _run(d, dtype, tokens, prompt_len, chunk)
    assert_logits(got, ref, dtype, f"far keys, prompt of {prompt_len}")
    assert_logits(got[:4], ref[:4], dtype, "the first tokens")
    edges = [63, 64, 65, 127, 128, 129, 191, 192, 193, 519, 520, 521, 639, 640]
    assert_logits(got[edges], ref[edges], dtype, "positions at the borders of pages and of the prompt")


@DTYPES
@pytest.mark.parametrize("prompt_len, chunk", [(600, None), (590, 65), (590, 2), (450, 64), (3, None)])
def test_memories_over_many_runs(session_tmp, dtype, prompt_len, chunk):
    """Forget gates so close to one that the memory at position 600 still holds the first tokens: a memory, key sum or maximum lost
    at any border shows."""
    d = make_zanezen_dir(session_tmp, SLOW, seed=8, edit=_slow)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [600], seed=9)[0]
    ref = P.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())
    other = P.forward(cfg, weights, random_prompts(cfg["vocab"], [40], seed=10)[0] + tokens[40:])
    moved = _moved(other, ref, scale)[100:]
    assert float((moved > 10).float().mean()) > 0.9, moved.median()
    assert_logits(_run(d, dtype, tokens, prompt_len, chunk), ref, dtype, "memories")


@DTYPES
def test_every_constant_and_mechanism(session_tmp, dtype):
    """What the plain implementation loses when a mechanism is changed or dropped, the engine must have."""
    d = make_zanezen_dir(session_tmp, MIX, seed=6, edit=_wide_gates)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [150], seed=7)[0]
    ref = P.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())

    def differs(what, other, least=0.8):
        moved = _moved(other, ref, scale)[4:]
        assert float((moved > 20).float().mean()) > least, (what, moved.median())

    for path, value in ((("layers", 0, "mixer", "gate_cap"), 2.0), (("layers", 0, "mlp", "router", "scale"), 1.0),
                        (("layers", 0, "mlp", "shared"), None), (("layers", 1, "mixer", "scale"), 0.6), (("layers", 1, "mixer", "diff"), 0.45),
                        (("layers", 1, "mixer", "softcap"), 2.0), (("layers", 1, "mixer", "softcap"), None),
                        (("layers", 1, "mixer", "rot", "base"), 20.0), (("layers", 1, "mixer", "rot", "dims"), 12),
                        (("layers", 1, "mixer", "rot", "scaling"), None), (("layers", 1, "mixer", "rot", "scaling", "factor"), 8.0),
                        (("layers", 1, "mixer", "rot", "scaling", "slow"), 4.0), (("layers", 2, "mixer", "scale"), 0.5),
                        (("layers", 2, "mixer", "rot", "base"), 5.0), (("residual_mult",), 0.75), (("embedding", "scale"), 2.0),
                        (("norm", "eps"), 1e-1)):
        c2 = copy.deepcopy(cfg)
        at = c2
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        differs(path, P.forward(c2, weights, tokens))
    for name, change in (("l0.mix.i.b", 0.0), ("l0.mix.f.b", 0.5), ("l0.mix.norm", 0.7), ("l0.mlp.correction", 0.0), ("l1.mix.lq1", 0.0),
                         ("l1.mlp.gate.b", 0.0), ("l1.mlp.up.b", 0.0), ("l1.mlp.down.b", 0.0), ("l2.mix.g", 0.0), ("l2.mix.dkv.norm", 0.6)):
        differs(name, P.forward(cfg, {n: t * (change if n == name else 1.0) for n, t in weights.items()}, tokens), 0.5 if "correction" in name else 0.8)
    for name in ("l1.mix.q.conv", "l1.mix.k.conv", "l1.mix.v.conv"):       # a convolution of which the newest tap alone is left
        kept = torch.zeros_like(weights[name])
        kept[:, -1] = weights[name][:, -1]
        differs(name, P.forward(cfg, {**weights, name: kept}, tokens))
    sinkless = {**weights, "l2.mix.sink": torch.full_like(weights["l2.mix.sink"], -1e4)}
    differs("the sink", P.forward(cfg, sinkless, tokens), 0.6)
    for cut in ((150, None), (90, 31), (149, 3)):
        assert_logits(_run(d, dtype, tokens, *cut), _settled(cfg, weights, tokens, ref), dtype, f"mechanisms, {cut}")


def _settled(cfg, weights, tokens, ref):
    from zanezen_helpers import reference

    r = reference(cfg, weights, tokens)
    assert torch.equal(r.logits, ref)
    return r


@DTYPES
def test_the_divisors_floor(session_tmp, dtype):
    """Input gates far below zero: what a memory returns is then so small that the eps of its head's norm counts, and with it the
    divisor, which is e^(-m) here."""
    d = make_zanezen_dir(session_tmp, SLOW, seed=3, edit=_closed)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [80], seed=4)[0]
    ref = P.forward(cfg, weights, tokens)
    scale = float(ref.abs().max())
    memory = P.matrix_memory
    P.matrix_memory = lambda q, k, v, li, lf: memory(q, k, v, li + 100.0, lf)       # (a divisor that never is e^(-m))
    try:
        moved = _moved(P.forward(cfg, weights, tokens), ref, scale)
    finally:
        P.matrix_memory = memory
    assert float((moved > 20).float().mean()) > 0.8, moved.median()
    for cut in ((80, None), (70, 9), (2, None)):
        assert_logits(_run(d, dtype, tokens, *cut), ref, dtype, f"floor, {cut}")


@DTYPES
def test_long_decoding(session_tmp, dtype):
    """Four tokens of prompt, then 400 decoded one by one: pages fill, and every step reads the memory and the convolution's inputs
    that the step before it left."""
    cfg_json = _model(64, 32, 1e-6, 0.15, 5.0, 0.8, [SLOW["layers"][0], MIX["layers"][1], MIX["layers"][2]])
    d = make_zanezen_dir(session_tmp, cfg_json, seed=8, edit=_slow)
    cfg, weights = plain_inputs(d)
    tokens = random_prompts(cfg["vocab"], [404], seed=9)[0]
    ref = P.forward(cfg, weights, tokens)
    assert_logits(_run(d, dtype, tokens, 4), ref, dtype, "long decoding")


@DTYPES
def test_slots_used_again_start_empty(session_tmp, dtype):
    """A sequence in a slot whose memory, convolution inputs and pages another sequence has left."""
    from gpullama3.java_b200.engine.step import SequenceInput, StepFunction
    from gpullama3.java_b200.engine.trace import load_model

    d = make_zanezen_dir(session_tmp, MIX, seed=6, edit=_wide_gates)
    cfg, weights = plain_inputs(d)
    a, b = random_prompts(cfg["vocab"], [90, 75], seed=12)
    model = load_model(d, dtype)
    cache = model.new_cache(64 * 2, max_slots=1)
    step = StepFunction(model, cache)
    for tokens in (a, b, a[:1], b[:2] + a):
        slot = cache.acquire()
        got = step([SequenceInput(slot, tokens, list(range(len(tokens))))]).cpu()
        assert_logits(got, _settled(cfg, weights, tokens, P.forward(cfg, weights, tokens)), dtype, f"{len(tokens)} tokens")
        cache.release(slot)
    cache.check_invariants()
