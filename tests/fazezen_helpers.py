"""Small Fazezen configurations for the tests, and model folders with random weights made so that faults show.

The configurations differ from one another in every size and option: heads per kv head (1 to 20), key sizes smaller than,
as large as and larger than the values, head sizes the tensor-core attention kernels take and ones that are widened, runs of
one position, shorter than a page, a page long, longer than two, and no runs, rotation of a part of a head, of all of it
and none, with and without slowed frequencies (so that pairs are kept, slowed and blended), score scales that are not
1 / sqrt(dim), factors of the two mixers on both sides of one and a negative one, decays from 0 to 1, states larger than one
CTA's columns and keys too long for the runs' tiles, layers without feed-forward, and both layer types in every order."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _rot(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def _left(heads, kv_heads, dim, vdim, scale, size=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = rot
    return m


def _rec(dim, vdim, decay, rot=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot is not None:
        m["rot"] = rot
    return m


def _par(left, right, left_scale, right_scale, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _lig(dim, vdim, decay, ff=None):
    return {"type": "lightning", "mixer": _rec(dim, vdim, decay), "mlp": {"kind": "dense", "ff": ff} if ff else None}


FAZEZEN_A = {
    "architecture": "Fazezen", "vocab": 160, "width": 64, "norm": {"eps": 1e-5}, "initializer_range": 0.1,
    "layers": [
        _par(_left(4, 2, 16, 24, 0.3, 40, _rot(5000.0, 8, (4.0, 1.0, 4.0, 64))), _rec(16, 32, (0.5, 0.9, 0.995), _rot(100.0, 16)), 0.7, 1.3, 96),
        _lig(24, 16, (0.8, 0.99)),
        _lig(8, 40, (0.3, 0.95, 0.999), 64),
    ],
}
FAZEZEN_B = {
    "architecture": "Fazezen", "vocab": 200, "width": 96, "norm": {"eps": 1e-6}, "initializer_range": 0.08,
    "layers": [
        _lig(32, 64, (0.7, 0.97, 0.9995), 64),
        _par(_left(6, 1, 32, 32, 0.2, 64, _rot(300.0, 32)), _rec(64, 16, (0.9, 0.98, 0.99, 0.6), _rot(1000.0, 32)), 1.5, -0.6, 128),
    ],
}
# sizes off every kernel's grid of fast cases
FAZEZEN_C = {
    "architecture": "Fazezen", "vocab": 77, "width": 50, "norm": {"eps": 1e-5}, "initializer_range": 0.12,
    "layers": [
        _par(_left(3, 3, 12, 20, 0.25, 7, _rot(50.0, 4)), _rec(10, 9, (0.85, 0.97), _rot(30.0, 6)), 1.0, 0.8, 30),
        _lig(7, 11, (0.9, 0.4, 0.99, 0.75, 0.999), 22),
        _par(_left(2, 1, 6, 14, 0.5, 65, _rot(10000.0, 6, (2.0, 1.0, 2.0, 40))), _rec(20, 13, (0.95,), _rot(500.0, 2)), 0.4, 1.0),
    ],
}
# heads of 64 and 128 (the tcgen05 prompt attention), rows wide enough for the kernels that take them in several rounds, a
# state of 128 x 128 and one whose values no single CTA holds
FAZEZEN_D = {
    "architecture": "Fazezen", "vocab": 120, "width": 640, "norm": {"eps": 1e-5}, "initializer_range": 0.04,
    "layers": [
        _par(_left(8, 2, 64, 64, 0.15, 130, _rot(10000.0, 64, (8.0, 1.0, 4.0, 128))), _rec(128, 128, (0.99, 0.9), _rot(20000.0, 128)), 1.25, 0.85, 256),
        _lig(128, 192, (0.97, 0.999)),
        _par(_left(4, 4, 128, 96, 0.1, 33, _rot(700.0, 64)), _rec(32, 64, (0.8, 0.95, 0.99), _rot(100.0, 16)), 0.8, 1.1, 128),
    ],
}
# no runs, no rotation, twenty heads on one kv head, runs of one position, decays of 0 and 1, keys too long for the runs' tiles
FAZEZEN_E = {
    "architecture": "Fazezen", "vocab": 96, "width": 48, "norm": {"eps": 1e-6}, "initializer_range": 0.1,
    "layers": [
        _par(_left(20, 1, 16, 8, 0.3), _rec(24, 16, (0.0, 1.0, 0.97)), 1.1, 0.5, 64),
        _par(_left(2, 2, 24, 16, 0.4, 1, _rot(100.0, 24)), _rec(8, 8, (0.9, 0.99), _rot(100.0, 0)), 0.9, 1.0),
        _lig(272, 24, (0.98,), 32),
        _par(_left(2, 1, 144, 40, 0.1, 200, _rot(1000000.0, 100)), _rec(16, 24, (0.95, 0.999), _rot(10.0, 8)), 1.0, 1.0, 48),
    ],
}
CONFIGS = {"A": FAZEZEN_A, "B": FAZEZEN_B, "C": FAZEZEN_C, "D": FAZEZEN_D, "E": FAZEZEN_E}


def make_fazezen_dir(tmp_path: Path, config_json: dict, seed: int = 0, edit=None) -> Path:
    """A model folder with random bfloat16 weights.  Norm weights and biases get a visible spread.
    ``edit(tensors)`` may change the float32 tensors before they are rounded and written."""
    from gpullama3.java_b200.config import config_from_dict
    from gpullama3.java_b200.weights import random_checkpoint, write_safetensors

    cfg = config_from_dict(config_json)
    tag = abs(hash(json.dumps([config_json, seed, getattr(edit, "__name__", None)], sort_keys=True))) % 10 ** 10
    out = Path(tmp_path) / f"fazezen_{tag}"
    if (out / "model.safetensors").is_file():
        return out
    out.mkdir(parents=True, exist_ok=True)
    where = "cuda" if torch.cuda.is_available() else "cpu"
    tensors = {}
    for n, t in random_checkpoint(cfg, seed, dtype=torch.float32, norm_std=0.2, device=where):
        tensors[n] = t.cpu().to(torch.float32)
    for name in tensors:
        if name.endswith((".norm1", ".norm2", "embed.norm", "final.norm")):
            tensors[name] = tensors[name] * (0.2 / cfg.initializer_range)
        if name.endswith(".b"):
            tensors[name] = tensors[name] * 10.0
    if edit is not None:
        edit(tensors)
    (out / "config.json").write_text(json.dumps(cfg.to_dict(), indent=2))
    write_safetensors(out / "model.safetensors", {n: t.to(torch.bfloat16) for n, t in tensors.items()})
    return out


def plain_inputs(model_dir: Path):
    """config.json as a dict and the weights by checkpoint name as float32, read with the safetensors package (not with
    the product's reader)."""
    from safetensors.torch import load_file

    cfg = json.loads((Path(model_dir) / "config.json").read_text())
    weights = {k: v.to(torch.float32) for k, v in load_file(str(Path(model_dir) / "model.safetensors")).items()}
    return cfg, weights


class Reference:
    """The plain implementation's logits of a request and, per position and logit, how far they move when what every
    product reads and returns is rounded to bfloat16: a head's output is divided by its root mean square, so where it is
    small by chance the norm magnifies any rounding; the plain implementation shows that itself."""

    def __init__(self, logits: torch.Tensor, moved: torch.Tensor):
        self.logits, self.moved = logits, moved

    def __getitem__(self, index):
        return Reference(self.logits[index], self.moved[index])


def reference(cfg, weights, tokens) -> Reference:
    import plain_fazezen

    exact = plain_fazezen.forward(cfg, weights, tokens)
    rounded = plain_fazezen.forward(cfg, weights, tokens, reads=lambda h: h.to(torch.bfloat16).to(h.dtype))
    return Reference(exact, (rounded - exact).abs())


def assert_logits(got: torch.Tensor, ref, dtype, what: str = "") -> None:
    """float32: accumulation-order noise only, at every position.  bfloat16: the engine rounds activations between its
    kernels, the plain implementation does not round at all; what is allowed is a few roundings' worth relative to the
    largest logit plus, against a ``Reference``, three times what the roundings of its products move the plain
    implementation's own result at that position; a small share of positions may lie outside."""
    moved = None
    if isinstance(ref, Reference):
        ref, moved = ref.logits, ref.moved.detach().to("cpu", torch.float64)
    got = got.detach().to("cpu", torch.float64)
    ref = ref.detach().to("cpu", torch.float64)
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    scale = float(ref.abs().max()) + 1e-30
    err = (got - ref).abs()
    worst, mean = err.amax(dim=-1), err.mean(dim=-1)
    if dtype == torch.float32:
        allowed = 5e-5 * scale + (1e-3 * moved.amax(dim=-1) if moved is not None else 0.0)
        over = worst - allowed
        assert float(over.max()) <= 0.0, (f"{what}: max err {float(worst.max()):.3e} vs scale {scale:.3e} "
                                          f"(position {int(over.argmax())})")
        return
    if moved is None:
        bad = (worst > 0.06 * scale) | (mean > 0.01 * scale)
    else:
        bad = (worst > 0.04 * scale + 3.0 * moved.amax(dim=-1)) | (mean > 0.008 * scale + 3.0 * moved.mean(dim=-1))
    allowed = max(1, int(0.05 * bad.numel())) if bad.numel() >= 3 else 0
    assert int(bad.sum()) <= allowed, (f"{what}: {int(bad.sum())} of {bad.numel()} positions outside "
                                       f"(max err {float(err.max()):.3e}, scale {scale:.3e})")
    typical = 0.03 * scale + (3.0 * float(moved.amax(dim=-1).median()) if moved is not None else 0.0)
    assert float(worst.median()) <= typical, f"{what}: median of the worst errors {float(worst.median()):.3e} vs scale {scale:.3e}"
