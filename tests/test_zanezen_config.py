"""The Zanezen configuration as data: keys read and written back, records that may be absent, the cache every run keeps, checkpoint
names and shapes, what is refused, random weights, the products that a layer joins, the stream that is kept divided by the residual
factor, and the plain implementation on inputs so small that its mechanisms can be checked by hand."""
import copy
import math

import pytest
import torch

import plain_zanezen as P
from zanezen_helpers import CONFIGS, make_zanezen_dir, plain_inputs
from gpullama3.java_b200.cache import EntryNeeds, KVCacheNeed, StateNeed
from gpullama3.java_b200.config import ConfigError, ZanezenConfig, config_from_dict
from gpullama3.java_b200.engine.model import CausalLM, parameter_specs_by_checkpoint_name
from gpullama3.java_b200.parts.position import YarnRotaryPositionEncoding

F = torch.float64


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_round_trip(name):
    d = CONFIGS[name]
    cfg = config_from_dict(d)
    assert isinstance(cfg, ZanezenConfig) and config_from_dict(cfg.to_dict()) == cfg
    assert [e.layer for e in cfg.schedule()] == list(range(len(d["layers"]))) and not cfg.tie_word_embeddings


def test_names_shapes_and_needs():
    cfg = config_from_dict(CONFIGS["A"])
    specs = parameter_specs_by_checkpoint_name(cfg)
    shapes = {"embed": (160, 64), "head": (160, 64), "final.norm": (64,), "l0.norm1": (64,), "l0.mix.q": (48, 64), "l0.mix.v": (72, 64),
              "l0.mix.g": (72, 64), "l0.mix.o": (64, 72), "l0.mix.norm": (72,), "l0.mix.i": (3, 64), "l0.mix.i.b": (3,),
              "l0.mix.f": (3, 64), "l0.mix.f.b": (3,), "l0.mlp.gate.b": (96,), "l0.mlp.down.b": (64,), "l1.mix.q": (96, 64),
              "l1.mix.k": (48, 64), "l1.mix.v": (40, 64), "l1.mix.q.conv": (96, 3), "l1.mix.k.conv": (48, 3), "l1.mix.v.conv": (40, 3),
              "l1.mix.lq1": (12,), "l1.mix.o": (64, 80), "l1.mlp.router": (7, 64), "l1.mlp.correction": (7,), "l1.mlp.e6.up": (32, 64),
              "l1.mlp.e6.down": (64, 32), "l1.mlp.shared.up": (40, 64), "l1.mlp.shared.down": (64, 40), "l1.mlp.shared.sg": (1, 64),
              "l2.mix.q": (56, 64), "l2.mix.dkv": (20, 64), "l2.mix.dkv.norm": (14,), "l2.mix.uk": (32, 14), "l2.mix.uv": (40, 14),
              "l2.mix.sink": (4,), "l2.mix.g": (4, 64), "l2.mix.o": (64, 40)}
    for n, shape in shapes.items():
        assert specs[n].shape == shape, n
    assert not any(n.startswith("l2.mlp") or n.endswith("norm2") for n in specs)
    needs = CausalLM(cfg, torch.bfloat16, "cpu").cache_needs()
    # a memory: S, then one copy of the key sum and of the maximum per head, to a multiple of 4
    assert needs[0] == StateNeed((3 * (16 * 24 + 16 + 1) + 1,), torch.float32)
    assert needs[1] == EntryNeeds((("kv", KVCacheNeed(2, 32)), ("conv", StateNeed((2 * 184,), torch.float32))))
    assert needs[2] == KVCacheNeed(1, 32)


def test_absent_records_build_the_model_without_the_mechanism():
    blocks = CausalLM(config_from_dict(CONFIGS["E"]), torch.bfloat16, "cpu").blocks
    assert blocks[0].mixer.taps == 0 and not blocks[0].mixer.shape.has_terms and blocks[0].mixer.position.rotary_dim == 0
    assert blocks[0].cache_need() == KVCacheNeed(1, 32) and blocks[2].cache_need() == KVCacheNeed(1, 144)   # (one tap keeps nothing)
    assert blocks[2].mixer.taps == 1 and blocks[2].mixer.shape.softcap == 6.0 and blocks[2].mixer.position.rotary_dim == 0
    assert blocks[3].mixer.rot_dim == 0 and blocks[3].feed_forward.shared_size == 0
    d = copy.deepcopy(CONFIGS["A"])
    d["layers"][1]["mixer"]["rot"]["scaling"] = None
    d["layers"][1]["mlp"]["shared"] = None
    for key in ("embedding", "residual_mult"):
        del d[key]
    cfg = config_from_dict(d)
    assert config_from_dict(cfg.to_dict()) == cfg and cfg.embedding_scale() == 1.0
    assert CausalLM(cfg, torch.bfloat16, "cpu").blocks[1].mixer.magnitude == 1.0


def _broken(path, value):
    d = copy.deepcopy(CONFIGS["A"])
    at = d
    for k in path[:-1]:
        at = at[k]
    if value is KeyError:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return d


@pytest.mark.parametrize("path, value", [
    (("layers",), []), (("norm",), {}), (("norm", "eps"), 0.0), (("vocab",), KeyError), (("residual_mult",), 0.0),
    (("embedding",), 3.0), (("layers", 0, "type"), "lightning"), (("layers", 0, "mixer", "gate_cap"), 0.0),
    (("layers", 0, "mixer", "gate_cap"), KeyError), (("layers", 0, "mixer", "dim"), 0), (("layers", 1, "mixer", "kv_heads"), 3),
    (("layers", 1, "mixer", "diff"), KeyError), (("layers", 1, "mixer", "softcap"), -2.0), (("layers", 1, "mixer", "conv"), 2.5),
    (("layers", 1, "mixer", "rot", "dims"), 7), (("layers", 1, "mixer", "rot", "dims"), 14),
    (("layers", 1, "mixer", "rot", "scaling", "fast"), KeyError), (("layers", 1, "mixer", "rot", "scaling", "original"), 0),
    (("layers", 1, "mixer", "scale"), KeyError), (("layers", 2, "mixer", "rot", "dims"), 4), (("layers", 2, "mixer", "kv_rank"), KeyError),
    (("layers", 2, "mixer", "rot"), None), (("layers", 1, "mlp", "router", "top"), 8), (("layers", 1, "mlp", "kind"), "sparse"),
    (("layers", 1, "mlp", "shared"), {}), (("layers", 0, "mlp", "ff"), KeyError)])
def test_malformed_configurations_are_refused(path, value):
    with pytest.raises(ConfigError):
        config_from_dict(_broken(path, value))


@pytest.mark.parametrize("path, value", [
    (("layers", 0, "mixer", "dim"), 513), (("layers", 1, "mixer", "dim"), 257), (("layers", 1, "mixer", "vdim"), 513),
    (("layers", 1, "mixer", "conv"), 17), (("layers", 2, "mixer", "kv_rank"), 507)])
def test_sizes_no_kernel_takes_are_refused_when_the_model_is_built(path, value):
    with pytest.raises(ConfigError):
        CausalLM(config_from_dict(_broken(path, value)), torch.bfloat16, "cpu")


def test_random_weights_fill_every_tensor(tmp_path):
    d = make_zanezen_dir(tmp_path, CONFIGS["C"], seed=1)
    cfg, weights = plain_inputs(d)
    assert set(weights) == set(parameter_specs_by_checkpoint_name(config_from_dict(CONFIGS["C"])))
    assert all(float(w.abs().max()) > 0 for w in weights.values())


def test_joined_products_are_the_parts_products(tmp_path):
    """After loading, a layer has one last product, and one first product where the feed-forward is a mixture with a shared expert."""
    d = make_zanezen_dir(tmp_path, CONFIGS["A"], seed=2)
    cfg, weights = plain_inputs(d)
    model = CausalLM(config_from_dict(CONFIGS["A"]), torch.float32, "cpu")
    model.load_folder(d)
    first, second, third, _ = model.blocks
    assert torch.equal(first.out.weight, torch.cat([weights["l0.mix.o"], weights["l0.mlp.down"]], dim=1)) and first.inputs is None
    assert torch.equal(first.out.bias, weights["l0.mlp.down.b"])
    assert torch.equal(second.out.weight, torch.cat([weights["l1.mix.o"], weights["l1.mlp.shared.down"]], dim=1))
    w = second.inputs.weight
    assert torch.equal(w[:96], weights["l1.mix.q"]) and torch.equal(w[second.input_columns:][:40], weights["l1.mlp.shared.up"])
    assert torch.equal(w[second.input_columns + 40], weights["l1.mlp.shared.sg"][0]) and second.mixer.qkv is None
    assert torch.equal(third.out.weight, weights["l2.mix.o"]) and third.inputs is None


def test_the_stream_is_kept_divided_by_the_residual_factor():
    """x <- x + r y over norms with eps is x' <- x' + y over norms with eps / r^2, x = r x'."""
    cfg = config_from_dict(CONFIGS["A"])
    assert cfg.embedding_scale() == 6.0 / 0.6
    norm = cfg.layer_specs()[0].parts["mixer_norm"].args
    assert norm["eps"] == 1e-5 / 0.6 ** 2
    x = torch.randn(3, 64, dtype=F) * 1e-2
    assert torch.allclose(P.over_root_mean_square(x, 1e-5), P.over_root_mean_square(x / 0.6, norm["eps"]), rtol=1e-12)
    assert cfg.layer_specs()[0].parts["mixer"].args["norm_eps"] == 1e-5      # (norms of heads are not norms of the stream)


# ---------------------------------------------------------------- the plain implementation by hand
def test_stretched_frequencies():
    f, mag = P.pair_frequencies(100.0, 6, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    lo = max(math.floor(6 * math.log(64 / (16 * math.pi)) / (2 * math.log(100.0))), 0)
    hi = min(math.ceil(6 * math.log(64 / (2 * math.pi)) / (2 * math.log(100.0))), 5)
    assert (lo, hi) == (0, 2) and abs(mag - (0.1 * math.log(4.0) + 1)) < 1e-15
    want = [1.0, 100.0 ** (-1 / 3) * (0.5 / 4 + 0.5), 100.0 ** (-2 / 3) / 4]
    assert all(abs(a - b) < 1e-12 for a, b in zip(f, want))
    part = YarnRotaryPositionEncoding(6, 100.0, 4.0, 64, 8.0, 1.0, pairing="half")
    assert all(abs(a - b) < 1e-12 for a, b in zip(part.frequencies(), f)) and part.magnitude == mag


def test_turning_halves_and_the_columns_behind_them():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]], [[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F)
    y = P.turn_halves(x, [0.5, 2.0], 1.5)
    assert torch.allclose(y[0, 0], torch.tensor([1.5, 3.0, 4.5, 6.0, 5.0], dtype=F))
    assert abs(y[1, 0, 0] - 1.5 * (math.cos(0.5) - 3 * math.sin(0.5))) < 1e-12 and abs(y[1, 0, 2] - 1.5 * (3 * math.cos(0.5) + math.sin(0.5))) < 1e-12


def test_convolution_caps_and_sinks_by_hand():
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=F)
    assert P.causal_convolution(u, torch.tensor([[10.0, 1.0]], dtype=F)).flatten().tolist() == [1.0, 12.0, 24.0]
    assert abs(float(P.soft_cap(torch.tensor(3.0, dtype=F), 2.0)) - 2 * math.tanh(1.5)) < 1e-15
    s = torch.tensor([[[0.0, 5.0], [math.log(2.0), math.log(3.0)]]], dtype=F)
    p = P.softmax_over_visible(s, P.causal_mask(2), torch.tensor([0.0], dtype=F))
    assert torch.allclose(p, torch.tensor([[[0.5, 0.0], [2 / 6, 3 / 6]]], dtype=F))


def test_memory_by_hand():
    """One head of one number: gates e^i and e^f without the running maximum give the same quotients where the floor is far."""
    q, k = torch.tensor([[[2.0]], [[1.0]], [[3.0]]], dtype=F), torch.tensor([[[1.0]], [[2.0]], [[1.0]]], dtype=F)
    v = torch.tensor([[[4.0]], [[8.0]], [[-1.0]]], dtype=F)
    li, lf = torch.tensor([[1.0], [-2.0], [3.0]], dtype=F), torch.log(torch.tensor([[0.5], [0.9], [0.2]], dtype=F))
    o, S, n, m = P.matrix_memory(q, k, v, li, lf)
    s = c = 0.0
    for t in range(3):
        s = math.exp(lf[t]) * s + math.exp(li[t]) * float(k[t]) * float(v[t])
        c = math.exp(lf[t]) * c + math.exp(li[t]) * float(k[t])
        want = s * float(q[t]) / (max(abs(c * float(q[t])), 1.0) + 1e-6 * math.exp(_maximum(li, lf, t)))
        assert abs(float(o[t]) - want) < 1e-12
    assert float(m) == 3.0


def _maximum(li, lf, t):
    m = 0.0
    for s in range(t + 1):
        m = max(float(lf[s]) + m, float(li[s]))
    return m


def test_the_maximum_starts_at_zero():
    """With input gates far below zero the first token's maximum is f + 0, not i: the divisor is e^(-m) then."""
    one = torch.ones(1, 1, 1, dtype=F)
    o, _, _, m = P.matrix_memory(one, one, one, torch.tensor([[-9.0]], dtype=F), torch.tensor([[-0.5]], dtype=F))
    assert float(m) == -0.5 and abs(float(o) - math.exp(-8.5) / (math.exp(0.5) + 1e-6)) < 1e-15


def test_routing_by_hand():
    W = {"router": torch.eye(3, dtype=F), "correction": torch.tensor([0.0, 0.5, 0.0], dtype=F)}
    chosen, w, margin = P.route(torch.tensor([[2.0, 0.0, 1.0]], dtype=F), W, "", {"top": 2, "scale": 3.0})
    s = [1 / (1 + math.exp(-z)) for z in (2.0, 0.0, 1.0)]
    assert chosen.tolist() == [[1, 0]]                        # 0.5 + 0.5 leads, and weighs by 0.5 alone
    assert torch.allclose(w, torch.tensor([[3 * 0.5 / (s[0] + 0.5), 3 * s[0] / (s[0] + 0.5)]], dtype=F))
    assert abs(float(margin) - (s[0] - s[2])) < 1e-12
