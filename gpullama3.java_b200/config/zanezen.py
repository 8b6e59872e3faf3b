"""Typed configuration of the Zanezen decoder, read from ``config.json``.

A Zanezen model is a list of layers over one residual stream, which starts as the embedding rows times ``embedding.scale``.  In
a layer one RMS norm (``norm.eps``) is read by the mixer and the feed-forward alike, and both results join the stream times
``residual_mult``.  The output head is a matrix of its own, behind a last such norm.

* ``layers[i].type`` names the mixer, ``layers[i].mixer`` gives its sizes.
  ``mlstm``: a matrix memory with exponential gates (``heads``, ``dim``, ``vdim``, ``gate_cap``), every head normed, with a weight and a
  sigmoid gate;
  ``attention``: differential attention (``heads``, ``kv_heads``, query/key size ``dim`` of one of the two maps, value size ``vdim``, score
  ``scale``, ``softcap`` on the scores, ``diff``, ``conv`` taps of a convolution over time on queries, keys and values, rotation ``rot`` of
  the first ``dims`` numbers of every map over halves: ``base`` and optionally ``scaling`` with ``factor``, ``original``, ``fast``,
  ``slow``);
  ``latent_attention``: keys and values from one cached latent row (``heads``, ``dim`` plain and ``rot_dim`` rotated numbers per head,
  ``vdim``, ``kv_rank``, score ``scale``, ``rot``), with a sink and an output gate per head;
* ``layers[i].mlp`` is null, ``{"kind": "dense", "ff"}`` (SiLU-gated, all three products with biases) or ``{"kind": "moe", "expert":
  {"ff"}, "router": {"experts", "top", "scale"}, "shared": {"ff"}}`` (experts without gate, the square of max(., 0); sigmoid scores, a
  correction that takes part in the choice alone; a shared expert with a gate of one number per token).

A record that is absent (``rot``, ``rot.scaling``, ``conv``, ``softcap``, ``mlp.shared``, ``mlp`` null) builds the model without that mechanism.

The stream is kept divided by ``residual_mult``.  With x = r x', x <- x + r y is x' <- x' + y, and a norm of x is the norm of x' with
eps / r^2 in place of eps; so the embedding rows enter times scale / r and no product has to apply the factor."""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, LayerSpec, ModelConfig, PartSpec, as_float, as_int, require_keys
from .registry import register_architecture

MIXER_TYPES = ("mlstm", "attention", "latent_attention")
MIXER_SIZES = {"mlstm": ("heads", "dim", "vdim"), "attention": ("heads", "kv_heads", "dim", "vdim"),
               "latent_attention": ("heads", "dim", "vdim", "kv_rank")}
ROTARY_MAGNITUDE_SLOPE = 0.1     # cosine and sine are multiplied by 0.1 ln(factor) + 1
ROTARY_MIN_RAMP_WIDTH = 0.001
ROUTING_EPS = 1e-20              # joins the sum of the chosen scores


def _positive(d: dict, key: str, where: str) -> float:
    v = as_float(d, key)
    if not v > 0:
        raise ConfigError(f"{where}: {key} must be positive, got {v}")
    return v


def _record(d: dict, key: str, where: str) -> dict:
    if not isinstance(d.get(key), dict):
        raise ConfigError(f"{where}: {key} must be an object")
    return dict(d[key])


@dataclass(frozen=True)
class ZanezenLayer:
    type: str
    mixer: dict        # the mixer's record as config.json has it (checked when read)
    mlp: dict | None   # the feed-forward's record, None for a layer without one


@dataclass(frozen=True)
class ZanezenConfig(ModelConfig):
    vocab_size: int
    hidden_size: int
    layers: tuple
    norm_eps: float
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    initializer_range: float = 0.02
    tie_word_embeddings: bool = False
    stop_token_ids: tuple[int, ...] = ()

    architecture = "Zanezen"

    # ---- reading
    @classmethod
    def from_dict(cls, d: dict) -> "ZanezenConfig":
        where = "Zanezen config.json"
        require_keys(d, ["vocab", "width", "layers", "norm"], where)
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("Zanezen config.json: 'layers' must be a non-empty list")
        norm = _record(d, "norm", where)
        require_keys(norm, ["eps"], "Zanezen norm")
        layers = []
        for i, L in enumerate(d["layers"]):
            at = f"layer {i}"
            if not isinstance(L, dict) or not isinstance(L.get("mixer"), dict):
                raise ConfigError(f"{at}: needs 'type' and a 'mixer' object")
            kind = L.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{at}: unknown mixer type {kind!r}; known: {', '.join(MIXER_TYPES)}")
            layers.append(ZanezenLayer(kind, cls._checked_mixer(kind, dict(L["mixer"]), at),
                                       cls._checked_mlp(L["mlp"], at + " mlp") if L.get("mlp") is not None else None))
        scale, mult = 1.0, 1.0
        if d.get("embedding") is not None:
            record = _record(d, "embedding", where)
            scale = as_float(record, "scale") if record.get("scale") is not None else 1.0
        if d.get("residual_mult") is not None:
            mult = _positive(d, "residual_mult", where)
        eos = d.get("eos_token_id")
        stop = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab_size=as_int(d, "vocab"), hidden_size=as_int(d, "width"), layers=tuple(layers),
                   norm_eps=_positive(norm, "eps", "norm"), embed_scale=scale, residual_mult=mult,
                   initializer_range=float(d.get("initializer_range", 0.02)), stop_token_ids=stop)

    @staticmethod
    def _checked_rotation(m: dict, most: int, where: str) -> None:
        if m.get("rot") is None:
            m.pop("rot", None)
            return
        rot = m["rot"] = _record(m, "rot", where)
        where += " rot"
        require_keys(rot, ["base", "dims"], where)
        _positive(rot, "base", where)
        dims = as_int(rot, "dims", minimum=0)
        if dims % 2 or dims > most:
            raise ConfigError(f"{where}: dims {dims} must be even and at most {most}")
        if rot.get("scaling") is None:
            rot.pop("scaling", None)
        else:
            s = rot["scaling"] = _record(rot, "scaling", where)
            require_keys(s, ["factor", "original", "fast", "slow"], where + ".scaling")
            for key in ("factor", "original", "fast", "slow"):
                _positive(s, key, where + ".scaling")

    @classmethod
    def _checked_mixer(cls, kind: str, m: dict, where: str) -> dict:
        require_keys(m, list(MIXER_SIZES[kind]), where)
        for key in MIXER_SIZES[kind]:
            as_int(m, key)
        if kind == "mlstm":
            require_keys(m, ["gate_cap"], where)
            _positive(m, "gate_cap", where)
            return m
        require_keys(m, ["scale"], where)
        _positive(m, "scale", where)
        if kind == "latent_attention":
            require_keys(m, ["rot_dim"], where)
            rot_dim = as_int(m, "rot_dim", minimum=0)
            cls._checked_rotation(m, rot_dim, where)
            if rot_dim and (m.get("rot") or {}).get("dims") != rot_dim:
                raise ConfigError(f"{where}: the {rot_dim} rotated numbers are rotated whole (rot.dims)")
            return m
        require_keys(m, ["diff"], where)
        as_float(m, "diff")
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
        if m.get("softcap") is None:
            m.pop("softcap", None)
        else:
            _positive(m, "softcap", where)
        if m.get("conv") is None:
            m.pop("conv", None)
        else:
            as_int(m, "conv", minimum=0)
        cls._checked_rotation(m, m["dim"], where)
        return m

    @staticmethod
    def _checked_mlp(mlp, where: str) -> dict:
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"{where} must be null or an object of kind 'dense' or 'moe', got {mlp!r}")
        if mlp["kind"] == "dense":
            require_keys(mlp, ["ff"], where)
            return {"kind": "dense", "ff": as_int(mlp, "ff")}
        expert, router = _record(mlp, "expert", where), _record(mlp, "router", where)
        require_keys(expert, ["ff"], where + ".expert")
        require_keys(router, ["experts", "top"], where + ".router")
        n, top = as_int(router, "experts"), as_int(router, "top")
        if top > n:
            raise ConfigError(f"{where}.router: {top} of {n} experts")
        scale = as_float(router, "scale") if router.get("scale") is not None else 1.0
        out = {"kind": "moe", "expert": {"ff": as_int(expert, "ff")}, "router": {"experts": n, "top": top, "scale": scale}}
        if mlp.get("shared") is not None:
            shared = _record(mlp, "shared", where)
            require_keys(shared, ["ff"], where + ".shared")
            out["shared"] = {"ff": as_int(shared, "ff")}
        return out

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult, "norm": {"eps": self.norm_eps},
             "initializer_range": self.initializer_range,
             "layers": [{"type": L.type, "mixer": dict(L.mixer), "mlp": dict(L.mlp) if L.mlp else None} for L in self.layers]}
        if self.stop_token_ids:
            d["eos_token_id"] = list(self.stop_token_ids)
        return d

    # ---- the model as data
    def embedding_scale(self) -> float:
        return self.embed_scale / self.residual_mult

    def _stream_norm(self) -> PartSpec:
        return PartSpec("norm", "rmsnorm", {"dim": self.hidden_size, "eps": self.norm_eps / self.residual_mult ** 2})

    @staticmethod
    def _position(m: dict) -> PartSpec:
        rot = m.get("rot") or {}
        if not rot.get("dims"):
            return PartSpec("position", "none", {})
        s = rot.get("scaling") or {}
        return PartSpec("position", "yarn", {
            "rotary_dim": rot["dims"], "base": float(rot["base"]), "factor": s.get("factor"), "original": s.get("original"),
            "fast": s.get("fast", 32.0), "slow": s.get("slow", 1.0), "magnitude_slope": ROTARY_MAGNITUDE_SLOPE,
            "min_ramp_width": ROTARY_MIN_RAMP_WIDTH, "pairing": "half"})

    def _mixer(self, L: ZanezenLayer) -> PartSpec:
        m, h = L.mixer, self.hidden_size
        if L.type == "mlstm":
            return PartSpec("mixer", "mlstm", {"hidden_size": h, "n_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
                                               "gate_cap": float(m["gate_cap"]), "norm_eps": self.norm_eps})
        if L.type == "latent_attention":
            return PartSpec("mixer", "latent_attention", {
                "hidden_size": h, "n_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"], "kv_rank": m["kv_rank"],
                "q_rank": None, "norm_eps": self.norm_eps, "scale": float(m["scale"]), "rot_dim": m["rot_dim"],
                "position": self._position(m) if m["rot_dim"] else None, "head_gate": True, "sink": True})
        return PartSpec("mixer", "differential_attention", {
            "hidden_size": h, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
            "scale": float(m["scale"]), "diff": float(m["diff"]), "norm_eps": self.norm_eps, "position": self._position(m),
            "output_gate": False, "qk_norm": False, "softcap": m.get("softcap"), "conv_taps": m.get("conv") or 0})

    def _feed_forward(self, mlp: dict) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("feed_forward", "gated", {"hidden_size": self.hidden_size, "intermediate_size": mlp["ff"],
                                                      "activation": "silu", "bias": True})
        ro = mlp["router"]
        return PartSpec("feed_forward", "routed", {
            "hidden_size": self.hidden_size, "intermediate_size": mlp["expert"]["ff"], "n_experts": ro["experts"], "top": ro["top"],
            "activation": "relu_squared", "weight_eps": ROUTING_EPS, "score": "sigmoid", "choice_correction": True,
            "weight_scale": ro["scale"], "shared_size": (mlp.get("shared") or {}).get("ff")})

    def layer_specs(self) -> list[LayerSpec]:
        specs = []
        for L in self.layers:
            parts = {"mixer": self._mixer(L), "mixer_norm": self._stream_norm()}
            if L.mlp is not None:
                parts["feed_forward"] = self._feed_forward(L.mlp)
            specs.append(LayerSpec("parallel", parts))
        return specs

    def final_norm(self) -> PartSpec:
        return self._stream_norm()

    def tensor_names(self) -> dict[str, str]:
        names = {"embedding.table": "embed", "final_norm.weight": "final.norm", "head.weight": "head"}
        for i, L in enumerate(self.layers):
            p, c = f"layers.{i}.", f"l{i}."
            names[p + "mixer_norm.weight"] = c + "norm1"
            m, x = p + "mixer.", c + "mix."
            if L.type == "mlstm":
                for w in ("q", "k", "v", "g", "o", "norm", "i", "f"):
                    names[m + w] = x + w
                for w in ("i", "f"):
                    names[m + w + "_bias"] = x + w + ".b"
            elif L.type == "attention":
                for w in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2"):
                    names[m + w] = x + w
                if L.mixer.get("conv"):
                    for w in ("q", "k", "v"):
                        names[m + w + "_conv"] = x + w + ".conv"
            else:
                for w in ("q", "dkv", "uk", "uv", "sink", "g", "o"):
                    names[m + w] = x + w
                names[m + "dkv_norm"] = x + "dkv.norm"
            if L.mlp is None:
                continue
            f, x = p + "feed_forward.", c + "mlp."
            if L.mlp["kind"] == "dense":
                for w in ("gate", "up", "down"):
                    names[f + w], names[f + w + "_bias"] = x + w, x + w + ".b"
                continue
            names[f + "router"], names[f + "correction"] = x + "router", x + "correction"
            for e in [f"e{e}" for e in range(L.mlp["router"]["experts"])] + (["shared"] if L.mlp.get("shared") else []):
                for w in ("up", "down"):
                    names[f"{f}{e}.{w}"] = f"{x}{e}.{w}"
            if L.mlp.get("shared"):
                names[f + "shared.sg"] = x + "shared.sg"
        return names

    def init_std(self) -> float:
        return self.initializer_range


register_architecture("Zanezen", ZanezenConfig)
