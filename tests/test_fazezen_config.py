"""The Fazezen configuration as data: keys read and written back, records that may be absent, the cache every run keeps,
checkpoint names and shapes, what is refused, random weights, pages of a cache cut into runs of positions, and the plain
implementation on inputs so small that its mechanisms can be checked by hand."""
import copy
import math

import pytest
import torch

import plain_fazezen as P
from fazezen_helpers import CONFIGS, make_fazezen_dir, plain_inputs
from gpullama3.java_b200.cache import EntryNeeds, KVCacheNeed, SequenceCache, StateNeed
from gpullama3.java_b200.config import ConfigError, FazezenConfig, config_from_dict
from gpullama3.java_b200.engine.model import CausalLM, parameter_specs_by_checkpoint_name
from gpullama3.java_b200.parts.position import llama3_inverse_frequencies

F = torch.float64


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_round_trip(name):
    d = CONFIGS[name]
    cfg = config_from_dict(d)
    assert isinstance(cfg, FazezenConfig) and config_from_dict(cfg.to_dict()) == cfg
    assert [e.layer for e in cfg.schedule()] == list(range(len(d["layers"])))
    assert cfg.tie_word_embeddings and cfg.embedding_scale() == 1.0 and cfg.embedding_norm() is not None


def test_names_shapes_and_needs():
    d = CONFIGS["A"]
    cfg = config_from_dict(d)
    specs = parameter_specs_by_checkpoint_name(cfg)
    shapes = {"embed": (160, 64), "embed.norm": (64,), "final.norm": (64,), "l0.norm1": (64,), "l0.norm2": (64,),
              "l0.mix.left.q": (64, 64), "l0.mix.left.k": (32, 64), "l0.mix.left.v": (48, 64), "l0.mix.left.q.norm": (16,),
              "l0.mix.left.k.norm": (16,), "l0.mix.left.o": (64, 96), "l0.mix.right.q": (48, 64), "l0.mix.right.k": (48, 64),
              "l0.mix.right.v": (96, 64), "l0.mix.right.g": (96, 64), "l0.mix.right.o": (64, 96), "l0.mlp.gate": (96, 64),
              "l0.mlp.gate.b": (96,), "l0.mlp.up": (96, 64), "l0.mlp.up.b": (96,), "l0.mlp.down": (64, 96), "l0.mlp.down.b": (64,),
              "l1.norm1": (64,), "l1.mix.q": (48, 64), "l1.mix.k": (48, 64), "l1.mix.v": (32, 64), "l1.mix.g": (32, 64),
              "l1.mix.o": (64, 32), "l1.mix.norm": (32,), "l2.mix.norm": (120,), "l2.mlp.down.b": (64,)}
    for n, shape in shapes.items():
        assert specs[n].shape == shape, n
    assert "l1.norm2" not in specs and "l1.mlp.gate" not in specs and "head" not in specs
    assert cfg.optional_tensor_names() == {"l1.norm2"}
    needs = CausalLM(cfg, torch.bfloat16, "cpu").cache_needs()
    assert needs[0] == EntryNeeds((("left", KVCacheNeed(2, 32, chunk=40)), ("right", StateNeed((3 * 16 * 32,), torch.float32))))
    assert needs[1] == StateNeed((2 * 24 * 16,), torch.float32) and needs[2] == StateNeed((3 * 8 * 40,), torch.float32)


def test_absent_records_build_the_model_without_the_mechanism():
    cfg = config_from_dict(CONFIGS["E"])
    left = CausalLM(cfg, torch.bfloat16, "cpu").blocks[0].mixer.left
    assert left.shape.chunk is None and left.position.rotary_dim == 0 and left.value_position is None
    d = copy.deepcopy(CONFIGS["A"])
    d["layers"][0]["mixer"]["left"]["mask"] = None
    d["layers"][0]["mixer"]["left"]["rot"]["scaling"] = None
    d["layers"][0]["mixer"]["right"]["rot"] = None
    cfg = config_from_dict(d)
    assert config_from_dict(cfg.to_dict()) == cfg
    block = CausalLM(cfg, torch.bfloat16, "cpu").blocks[0]
    assert block.mixer.left.shape.chunk is None and block.mixer.left.position.scaling is None
    assert block.mixer.right.position.rotary_dim == 0 and block.cache_need().named()["left"].chunk is None


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
    (("layers",), []), (("norm",), {}), (("norm", "eps"), 0.0), (("vocab",), KeyError), (("layers", 0, "type"), "attention"),
    (("layers", 0, "mixer", "left"), KeyError), (("layers", 0, "mixer", "left", "kv_heads"), 3),
    (("layers", 0, "mixer", "left", "mask", "size"), 0), (("layers", 0, "mixer", "left", "rot", "dims"), 7),
    (("layers", 0, "mixer", "left", "rot", "dims"), 18), (("layers", 0, "mixer", "left", "vdim"), 25),
    (("layers", 0, "mixer", "left", "rot", "scaling", "high"), 1.0), (("layers", 0, "mixer", "left", "rot", "scaling", "low"), KeyError),
    (("layers", 0, "mixer", "left", "scale"), -1.0), (("layers", 0, "mixer", "right", "decay"), [0.5, 0.9]),
    (("layers", 0, "mixer", "right", "decay"), [0.5, 0.9, 1.5]), (("layers", 0, "mixer", "left_scale"), "1"),
    (("layers", 1, "mixer", "dim"), 0), (("layers", 0, "mlp", "kind"), "moe"), (("layers", 0, "mlp", "ff"), KeyError)])
def test_malformed_configurations_are_refused(path, value):
    with pytest.raises(ConfigError):
        config_from_dict(_broken(path, value))


def test_sizes_no_kernel_takes_are_refused_when_the_model_is_built():
    with pytest.raises(ConfigError):
        CausalLM(config_from_dict(_broken(("layers", 0, "mixer", "left", "vdim"), 514)), torch.bfloat16, "cpu")
    with pytest.raises(ConfigError):
        CausalLM(config_from_dict(_broken(("layers", 1, "mixer", "dim"), 513)), torch.bfloat16, "cpu")


def test_random_weights_fill_every_tensor(tmp_path):
    d = make_fazezen_dir(tmp_path, CONFIGS["C"], seed=1)
    cfg, weights = plain_inputs(d)
    assert set(weights) == set(parameter_specs_by_checkpoint_name(config_from_dict(CONFIGS["C"])))
    assert all(float(w.abs().max()) > 0 for w in weights.values())


def test_joined_products_are_the_parts_products(tmp_path):
    """After loading, a layer has one last product: the mixers' and the feed-forward's weights side by side."""
    from gpullama3.java_b200.weights.loader import load_checkpoint_tensors

    d = make_fazezen_dir(tmp_path, CONFIGS["A"], seed=2)
    cfg, weights = plain_inputs(d)
    model = CausalLM(config_from_dict(CONFIGS["A"]), torch.float32, "cpu")
    model.load_folder(d)
    block = model.blocks[0]
    want = torch.cat([weights["l0.mix.left.o"], weights["l0.mix.right.o"], weights["l0.mlp.down"]], dim=1)
    assert torch.equal(block.out.weight, want) and torch.equal(block.out.bias, weights["l0.mlp.down.b"])
    q = block.mixer.inputs.weight
    assert torch.equal(q[:64], weights["l0.mix.left.q"]) and block.mixer.left.qkv is None and block.mixer.right.o is None
    assert block.feed_forward.down is None and model.blocks[1].out.bias is None
    assert torch.equal(model.blocks[1].out.weight, weights["l1.mix.o"])


def test_pages_of_a_cache_cut_into_runs():
    """A page is let go as soon as the next query's run of positions starts behind it, and a sequence never holds more
    pages than a run and a portion need."""
    for size in (64, 40, 130, 7):
        cache = SequenceCache({0: KVCacheNeed(1, 16, chunk=size)}, max_tokens=64 * 40, max_slots=2, dtype=torch.float32,
                              device="cpu", window_slack=16)
        g = cache.paged_groups[0]
        slot, other = cache.acquire(), cache.acquire()
        at = 0
        for n in [16, 1, 1, 15, 16, 14, 1, 1] + [13] * 40:
            cache.reserve([(slot, n)])
            cache.commit(slot, n)
            at += n
            first = at - at % size          # the run that position `at` belongs to
            row = g.rows[slot]
            for p, page in enumerate(row):
                needed = (p + 1) * 64 > first
                assert (page >= 0) == needed, (size, at, p)
            cache.check_invariants()
        cache.release(slot)
        cache.release(other)
        assert g.pool.n_held == 0


# ---------------------------------------------------------------- the plain implementation by hand
def test_frequencies_kept_slowed_and_blended():
    freqs = P.pair_frequencies(100.0, 8)
    assert freqs[0] == 1.0 and abs(freqs[2] - 0.1) < 1e-15
    s = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}
    out = P.stretched_frequencies(freqs, s)
    assert out[0] == freqs[0]                                            # wavelength 6.3 < 64 / 4
    assert abs(out[2] - 0.1 * 0.25) < 0.08 and out[3] == freqs[3] / 4.0    # 62.8: almost all slowed; 199 > 64
    blend = (64 / (2 * math.pi / 0.1) - 1.0) / 3.0
    assert abs(out[2] - ((1 - blend) * 0.1 / 4 + blend * 0.1)) < 1e-15
    # the product's frequencies are these to 32-bit rounding
    got = llama3_inverse_frequencies(8, 100.0, {"factor": 4.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                                                 "original_max_position_embeddings": 64})
    assert all(abs(a - b) <= 1e-6 * b for a, b in zip(got, out))


def test_turning_halves():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]], [[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F)
    y = P.turn_halves(x, [0.5, 2.0])
    assert torch.equal(y[0], x[0])
    assert abs(y[1, 0, 0] - (math.cos(0.5) - 3 * math.sin(0.5))) < 1e-12 and abs(y[1, 0, 2] - (3 * math.cos(0.5) + math.sin(0.5))) < 1e-12
    assert abs(y[1, 0, 1] - (2 * math.cos(2.0) - 4 * math.sin(2.0))) < 1e-12 and y[1, 0, 4] == 5.0
    assert torch.allclose(P.turn_halves(y, [0.5, 2.0], sign=-1.0), x, atol=1e-12)


def test_runs_and_the_silent_key():
    m = P.chunk_mask(7, 3)
    assert m.nonzero().tolist() == [[0, 0], [1, 0], [1, 1], [2, 0], [2, 1], [2, 2], [3, 3], [4, 3], [4, 4], [5, 3], [5, 4], [5, 5], [6, 6]]
    s = torch.tensor([[0.0, 5.0], [math.log(2.0), math.log(3.0)]], dtype=F)
    p = P.softmax_with_silent_key(s, torch.tensor([[True, False], [True, True]]))
    assert torch.allclose(p, torch.tensor([[0.5, 0.0], [2 / 6, 3 / 6]], dtype=F))
    far = P.softmax_with_silent_key(torch.tensor([[800.0], [-800.0]], dtype=F), torch.ones(2, 1, dtype=torch.bool))
    assert torch.allclose(far, torch.tensor([[1.0], [0.0]], dtype=F))


def test_values_enter_turned_by_their_distance_alone():
    """Shifting a sequence by whole runs leaves attention's result as it is."""
    torch.manual_seed(0)
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 6, "scale": 0.5, "mask": {"size": 5}, "rot": {"base": 10.0, "dims": 4}}
    W = {n: torch.randn(s, dtype=F) for n, s in (("q", (8, 8)), ("k", (4, 8)), ("v", (6, 8)), ("o", (8, 12)), ("q.norm", (4,)), ("k.norm", (4,)))}
    h = torch.randn(5, 8, dtype=F)
    y = P.chunked_attention(torch.cat([h, h, h]), W, "", m, 1e-6)
    assert torch.allclose(y[:5], y[5:10], atol=1e-10) and torch.allclose(y[:5], y[10:], atol=1e-10)


def test_decayed_sums_by_hand():
    q = torch.tensor([[[1.0]], [[2.0]], [[1.0]]], dtype=F)
    k = torch.tensor([[[1.0]], [[1.0]], [[3.0]]], dtype=F)
    v = torch.tensor([[[4.0]], [[8.0]], [[1.0]]], dtype=F)
    assert P.decayed_outer_sum(q, k, v, [0.5]).flatten().tolist() == [4.0, 20.0, 8.0]
