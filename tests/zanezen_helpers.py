"""Small Zanezen configurations for the tests, and model folders with random weights made so that faults show.

The configurations differ from one another in every size and option: heads per kv head (1 to 24 queries' maps on one key row), keys
smaller than, as large as and larger than the values, row sizes the tensor-core attention kernels take and ones that are widened,
convolutions of one tap to five and none, soft caps near the scores and none, rotation of a part of a map, of all of it and none, with
and without stretched frequencies (pairs kept, slowed and blended), latent rows with and without a rotated part, more heads than one
decode launch takes, memories whose values no single CTA holds and keys too long for the runs' tiles, residual factors on both
sides of one, layers with dense, routed and no feed-forward, with and without a shared expert, all experts chosen, and the three
layer types in different orders."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _rot(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def mem(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def att(heads, kv_heads, dim, vdim, scale, diff, conv=None, softcap=None, rot=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    for key, v in (("conv", conv), ("softcap", softcap), ("rot", rot)):
        if v is not None:
            m[key] = v
    return {"type": "attention", "mixer": m, "mlp": mlp}


def lat(heads, dim, rot_dim, vdim, rank, scale, base=100.0, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale}
    if rot_dim:
        m["rot"] = _rot(base, rot_dim)
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _model(vocab, width, eps, std, emb, mult, layers):
    return {"architecture": "Zanezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "initializer_range": std,
            "embedding": {"scale": emb}, "residual_mult": mult, "layers": layers}


ZANEZEN_A = _model(160, 64, 1e-5, 0.1, 6.0, 0.6, [
    mem(3, 16, 24, 5.0, dense(96)),
    att(4, 2, 12, 20, 0.4, 0.3, 3, 4.0, _rot(100.0, 6, (4.0, 64, 8.0, 1.0)), moe(32, 7, 2, 1.7, 40)),
    lat(4, 8, 6, 10, 14, 0.35),
    att(2, 2, 16, 32, 0.3, 0.55, 2, 9.0, _rot(5000.0, 16), dense(48)),
])
ZANEZEN_B = _model(200, 96, 1e-6, 0.08, 1.0, 1.4, [
    att(6, 1, 16, 32, 0.3, 0.2, 5, 3.0, _rot(300.0, 8), dense(64)),
    lat(3, 16, 8, 32, 24, 0.25, 50.0, moe(64, 12, 4, 0.6, 32)),
    mem(2, 32, 64, 15.0, moe(32, 6, 3, 2.5)),
])
# sizes off every kernel's grid of fast cases
ZANEZEN_C = _model(77, 50, 1e-5, 0.12, 3.0, 0.8, [
    lat(3, 7, 4, 9, 11, 0.4, 30.0, moe(14, 5, 2, 1.0, 10)),
    mem(2, 10, 13, 8.0, dense(30)),
    att(3, 3, 9, 11, 0.35, 0.4, 4, 2.5, _rot(50.0, 4, (2.0, 40, 4.0, 1.0)), moe(10, 9, 3, 1.3)),
    mem(3, 7, 33, 3.0),
])
# rows of 128 (the tcgen05 prompt attention), twenty heads on one latent row, memories of 128 x 192 and 64 x 128
ZANEZEN_D = _model(120, 640, 1e-5, 0.04, 8.0, 0.5, [
    att(4, 2, 64, 128, 0.12, 0.35, 4, 12.0, _rot(10000.0, 32, (8.0, 128, 16.0, 1.0)), moe(128, 8, 2, 2.0, 256)),
    mem(2, 128, 192, 10.0, dense(256)),
    lat(20, 64, 32, 32, 96, 0.1, 1000.0, dense(128)),
    mem(4, 64, 128, 15.0, moe(64, 16, 5, 1.0, 64)),
    att(2, 1, 32, 64, 0.2, 0.1, 3, 20.0, _rot(700.0, 32)),
])
# no convolution or one tap, no cap, no rotation, 24 maps on one key row, all experts chosen, keys too long for the runs' tiles
ZANEZEN_E = _model(96, 48, 1e-6, 0.1, 5.0, 1.0, [
    att(12, 1, 8, 12, 0.4, 0.25, None, None, None, moe(16, 5, 5, 1.0, 24)),
    mem(1, 400, 24, 6.0, dense(32)),
    att(2, 1, 72, 40, 0.15, 0.6, 1, 6.0, _rot(1000.0, 0), dense(40)),
    lat(2, 24, 0, 16, 20, 0.3, mlp=moe(24, 4, 1, 3.0)),
    mem(4, 8, 8, 1.5, moe(16, 3, 2, 0.5, 8)),
])
CONFIGS = {"A": ZANEZEN_A, "B": ZANEZEN_B, "C": ZANEZEN_C, "D": ZANEZEN_D, "E": ZANEZEN_E}


def make_zanezen_dir(tmp_path: Path, config_json: dict, seed: int = 0, edit=None) -> Path:
    """A model folder with random bfloat16 weights.  Norm weights and biases get a visible spread, the vectors behind lambda are
    large enough for it to differ from ``diff``, the routers' corrections lie wide apart (few choices are close calls), forget gates
    reach from a few tokens to hundreds.  ``edit(tensors)`` may change the float32 tensors before they are rounded and written."""
    from gpullama3.java_b200.config import config_from_dict
    from gpullama3.java_b200.weights import random_checkpoint, write_safetensors

    cfg = config_from_dict(config_json)
    tag = abs(hash(json.dumps([config_json, seed, getattr(edit, "__name__", None)], sort_keys=True))) % 10 ** 10
    out = Path(tmp_path) / f"zanezen_{tag}"
    if (out / "model.safetensors").is_file():
        return out
    out.mkdir(parents=True, exist_ok=True)
    where = "cuda" if torch.cuda.is_available() else "cpu"
    tensors = {}
    for n, t in random_checkpoint(cfg, seed, dtype=torch.float32, norm_std=0.2, device=where):
        tensors[n] = t.cpu().to(torch.float32)
    for name in tensors:
        last = name.rsplit(".", 1)[-1]
        if last in ("lq1", "lk1", "lq2", "lk2"):
            tensors[name] = tensors[name] * 3.0
        elif last == "correction":
            tensors[name] = tensors[name] * 4.0
        elif name.endswith(("gate.b", "up.b", "down.b")):
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


CLOSE_CALL = 0.01


class Reference:
    """The plain implementation's logits of a request and, per position and logit, how far they move when what every product
    reads and returns is rounded to bfloat16 (heads are divided by their root mean square, so where one is small by chance the
    norm magnifies any rounding).  ``settled`` [T]: no routed layer had a close call at this position or at one before it: behind
    one, a bfloat16 run may have picked the other expert, and attention and memories carry that to every later position."""

    def __init__(self, logits, moved, settled):
        self.logits, self.moved, self.settled = logits, moved, settled

    def __getitem__(self, index):
        return Reference(self.logits[index], self.moved[index], self.settled[index])


def reference(cfg, weights, tokens) -> Reference:
    import plain_zanezen

    margins: list = []
    exact = plain_zanezen.forward(cfg, weights, tokens, margins=margins)
    rounded = plain_zanezen.forward(cfg, weights, tokens, reads=lambda h: h.to(torch.bfloat16).to(h.dtype))
    close = torch.zeros(exact.shape[0], dtype=torch.bool)
    for m in margins:
        close |= m < CLOSE_CALL
    return Reference(exact, (rounded - exact).abs(), torch.cumsum(close.to(torch.int64), dim=0) == 0)


def assert_logits(got: torch.Tensor, ref, dtype, what: str = "") -> None:
    """float32: accumulation-order noise only, at every position.  bfloat16: the engine rounds activations between its
    kernels, the plain implementation does not round at all; what is allowed is a few roundings' worth relative to the
    largest logit plus, against a ``Reference``, three times what the roundings of its products move the plain
    implementation's own result at that position; a small share of positions may lie outside."""
    moved = settled = None
    if isinstance(ref, Reference):
        ref, moved, settled = ref.logits, ref.moved.detach().to("cpu", torch.float64), ref.settled
    got = got.detach().to("cpu", torch.float64)
    ref = ref.detach().to("cpu", torch.float64)
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    scale = float(ref.abs().max()) + 1e-30
    err = (got - ref).abs()
    if dtype == torch.float32:
        worst = err.amax(dim=-1)
        over = worst - (5e-5 * scale + (1e-3 * moved.amax(dim=-1) if moved is not None else 0.0))
        assert float(over.max()) <= 0.0, (f"{what}: max err {float(worst.max()):.3e} vs scale {scale:.3e} "
                                          f"(position {int(over.argmax())})")
        return
    if settled is not None:
        # behind a close call positions must be sane, the ones before it are held to the bound (the float32 run everywhere)
        assert float(err.max()) <= 2.0 * scale, f"{what}: max err {float(err.max()):.3e} vs scale {scale:.3e}"
        if not bool(settled.any()):
            return
        err, moved = err[settled], moved[settled]
    worst, mean = err.amax(dim=-1), err.mean(dim=-1)
    if moved is None:
        bad = (worst > 0.06 * scale) | (mean > 0.01 * scale)
    else:
        bad = (worst > 0.04 * scale + 3.0 * moved.amax(dim=-1)) | (mean > 0.008 * scale + 3.0 * moved.mean(dim=-1))
    allowed = max(1, int(0.05 * bad.numel())) if bad.numel() >= 3 else 0
    assert int(bad.sum()) <= allowed, (f"{what}: {int(bad.sum())} of {bad.numel()} positions outside "
                                       f"(max err {float(err.max()):.3e}, scale {scale:.3e})")
    typical = 0.03 * scale + (3.0 * float(moved.amax(dim=-1).median()) if moved is not None else 0.0)
    assert float(worst.median()) <= typical, f"{what}: median of the worst errors {float(worst.median()):.3e} vs scale {scale:.3e}"
