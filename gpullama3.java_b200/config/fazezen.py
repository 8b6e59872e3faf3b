"""Typed configuration of the Fazezen decoder, read from ``config.json``.

A Fazezen model is a list of layers over one residual stream.  The stream starts as the RMS-normed embedding rows.  In a
layer the mixer and the feed-forward stand side by side: both read the same stream, each through an RMS norm of its own
(``norm.eps``; weights are stored around zero and applied as 1 + w), and both results join it at once.  The output head is
the embedding table, behind a last such norm.

* ``layers[i].type`` names the mixer, ``layers[i].mixer`` gives its sizes.
  ``lightning``: linear attention with a fixed decay per head over SiLU-ed queries, keys and values (``heads``, ``dim``,
  ``vdim``, ``decay``), all heads normed together, with a sigmoid gate;
  ``parallel``: two mixers side by side, ``left_scale`` and ``right_scale`` their factors.  ``left``: softmax attention within
  runs of ``mask.size`` positions (``heads``, ``kv_heads``, query/key size ``dim``, value size ``vdim``, score ``scale``), an RMS norm
  over every query and key head, rotation ``rot`` of the first ``dims`` numbers over halves (``base``, and optionally ``scaling``
  with ``factor``, ``low``, ``high``, ``original``: slow pairs turn slower), values turned by their distance with frequencies of
  ``rot.base`` over all their numbers, one added to the softmax's denominator.  ``right``: retention (``heads``, ``dim``, ``vdim``,
  ``decay``, ``rot``), every head divided by its root mean square, with a SiLU gate;
* ``layers[i].mlp`` is null or ``{"kind": "dense", "ff"}``: GELU-gated (tanh form), all three products with biases.

A record that is absent (a mixer's ``mask`` or ``rot``, ``mlp`` null) builds the model without that mechanism."""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, LayerSpec, ModelConfig, PartSpec, as_float, as_int, require_keys
from .registry import register_architecture

MIXER_TYPES = ("lightning", "parallel")
SINK_SCORE = 0.0     # the further key without a value that every query of the softmax attention sees


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
class FazezenLayer:
    type: str
    mixer: dict        # the mixer's record as config.json has it (checked when read)
    mlp: dict | None   # the feed-forward's record, None for a layer without one


@dataclass(frozen=True)
class FazezenConfig(ModelConfig):
    vocab_size: int
    hidden_size: int
    layers: tuple
    norm_eps: float
    initializer_range: float = 0.02
    tie_word_embeddings: bool = True
    stop_token_ids: tuple[int, ...] = ()

    architecture = "Fazezen"

    # ---- reading
    @classmethod
    def from_dict(cls, d: dict) -> "FazezenConfig":
        require_keys(d, ["vocab", "width", "layers", "norm"], "Fazezen config.json")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("Fazezen config.json: 'layers' must be a non-empty list")
        norm = _record(d, "norm", "Fazezen config.json")
        require_keys(norm, ["eps"], "Fazezen norm")
        layers = []
        for i, L in enumerate(d["layers"]):
            where = f"layer {i}"
            if not isinstance(L, dict) or not isinstance(L.get("mixer"), dict):
                raise ConfigError(f"{where}: needs 'type' and a 'mixer' object")
            kind, m = L.get("type"), dict(L["mixer"])
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{where}: unknown mixer type {kind!r}; known: {', '.join(MIXER_TYPES)}")
            if kind == "lightning":
                m = cls._checked_recurrence(m, where)
            else:
                require_keys(m, ["left", "right", "left_scale", "right_scale"], where)
                as_float(m, "left_scale"), as_float(m, "right_scale")
                m["left"] = cls._checked_attention(_record(m, "left", where), where + " left")
                m["right"] = cls._checked_recurrence(_record(m, "right", where), where + " right")
            mlp = L.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"{where}: mlp must be null or an object of kind 'dense', got {mlp!r}")
                require_keys(mlp, ["ff"], where + " mlp")
                as_int(mlp, "ff")
                mlp = dict(mlp)
            layers.append(FazezenLayer(kind, m, mlp))
        eos = d.get("eos_token_id")
        stop = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab_size=as_int(d, "vocab"), hidden_size=as_int(d, "width"), layers=tuple(layers),
                   norm_eps=_positive(norm, "eps", "norm"), initializer_range=float(d.get("initializer_range", 0.02)),
                   stop_token_ids=stop)

    @staticmethod
    def _checked_rotation(m: dict, where: str) -> None:
        if m.get("rot") is None:
            m.pop("rot", None)
            return
        rot = m["rot"] = _record(m, "rot", where)
        where += " rot"
        require_keys(rot, ["base", "dims"], where)
        _positive(rot, "base", where)
        dims = as_int(rot, "dims", minimum=0)
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f"{where}: dims {dims} must be even and at most dim {m['dim']}")
        if rot.get("scaling") is None:
            rot.pop("scaling", None)
        else:
            s = rot["scaling"] = _record(rot, "scaling", where)
            require_keys(s, ["factor", "low", "high", "original"], where + ".scaling")
            for key in ("factor", "low", "high", "original"):
                _positive(s, key, where + ".scaling")
            if not s["high"] > s["low"]:
                raise ConfigError(f"{where}.scaling: high {s['high']} must be above low {s['low']}")

    @classmethod
    def _checked_recurrence(cls, m: dict, where: str) -> dict:
        require_keys(m, ["heads", "dim", "vdim", "decay"], where)
        for key in ("heads", "dim", "vdim"):
            as_int(m, key)
        if not isinstance(m["decay"], list) or len(m["decay"]) != m["heads"]:
            raise ConfigError(f"{where}: decay must list one number for each of the {m['heads']} heads")
        for g in m["decay"]:
            if isinstance(g, bool) or not isinstance(g, (int, float)) or not 0.0 <= g <= 1.0:
                raise ConfigError(f"{where}: a decay must lie between 0 and 1, got {g!r}")
        cls._checked_rotation(m, where)
        return m

    @classmethod
    def _checked_attention(cls, m: dict, where: str) -> dict:
        require_keys(m, ["heads", "kv_heads", "dim", "vdim", "scale"], where)
        for key in ("heads", "kv_heads", "dim", "vdim"):
            as_int(m, key)
        _positive(m, "scale", where)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
        if m.get("mask") is None:
            m.pop("mask", None)      # (no mask: every earlier position is visible)
        else:
            m["mask"] = _record(m, "mask", where)
            require_keys(m["mask"], ["size"], where + " mask")
            as_int(m["mask"], "size")
        cls._checked_rotation(m, where)
        if m.get("rot") is not None and m["vdim"] % 2:
            raise ConfigError(f"{where}: values are turned in pairs, vdim {m['vdim']} must be even")
        return m

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "initializer_range": self.initializer_range,
             "layers": [{"type": L.type, "mixer": dict(L.mixer), "mlp": dict(L.mlp) if L.mlp else None} for L in self.layers]}
        if self.stop_token_ids:
            d["eos_token_id"] = list(self.stop_token_ids)
        return d

    # ---- the model as data
    def _norm(self) -> PartSpec:
        return PartSpec("norm", "rmsnorm", {"dim": self.hidden_size, "eps": self.norm_eps, "offset": 1.0})

    @staticmethod
    def _position(m: dict) -> PartSpec:
        rot = m.get("rot") or {}
        if not rot.get("dims"):
            return PartSpec("position", "none", {})
        s = rot.get("scaling")
        scaling = None if s is None else {"factor": s["factor"], "low_freq_factor": s["low"], "high_freq_factor": s["high"],
                                          "original_max_position_embeddings": s["original"]}
        return PartSpec("position", "rope", {"head_dim": m["dim"], "theta": float(rot["base"]), "pairing": "half",
                                             "rotary_dim": rot["dims"], "scaling": scaling})

    def _recurrence(self, m: dict, **more) -> PartSpec:
        return PartSpec("mixer", "fixed_decay", {"hidden_size": self.hidden_size, "n_heads": m["heads"], "head_dim": m["dim"],
                                                 "value_dim": m["vdim"], "decay": list(m["decay"]), "norm_eps": self.norm_eps, **more})

    def _mixer(self, L: FazezenLayer) -> PartSpec:
        if L.type == "lightning":
            return self._recurrence(L.mixer, activation="silu", norm_over="all", norm_weight=True, gate="sigmoid")
        left, right = L.mixer["left"], L.mixer["right"]
        value_position = None
        if left.get("rot") is not None:
            value_position = PartSpec("position", "rope", {"head_dim": left["vdim"], "theta": float(left["rot"]["base"]), "pairing": "half"})
        return PartSpec("mixer", "parallel", {
            "left": PartSpec("mixer", "chunked_attention", {
                "hidden_size": self.hidden_size, "n_heads": left["heads"], "n_kv_heads": left["kv_heads"], "head_dim": left["dim"],
                "value_dim": left["vdim"], "scale": float(left["scale"]), "position": self._position(left),
                "value_position": value_position, "norm_eps": self.norm_eps, "chunk": (left.get("mask") or {}).get("size"),
                "sink": SINK_SCORE}),
            "right": self._recurrence(right, position=self._position(right), scale=right["dim"] ** -0.5, norm_over="head", gate="silu"),
            "left_scale": float(L.mixer["left_scale"]), "right_scale": float(L.mixer["right_scale"])})

    def layer_specs(self) -> list[LayerSpec]:
        specs = []
        for L in self.layers:
            parts = {"mixer": self._mixer(L), "mixer_norm": self._norm()}
            if L.mlp is not None:
                parts["feed_forward"] = PartSpec("feed_forward", "gated", {
                    "hidden_size": self.hidden_size, "intermediate_size": L.mlp["ff"], "activation": "gelu_tanh", "bias": True})
                parts["feed_forward_norm"] = self._norm()
            specs.append(LayerSpec("parallel", parts))
        return specs

    def embedding_norm(self) -> PartSpec:
        return self._norm()

    def final_norm(self) -> PartSpec:
        return self._norm()

    def tensor_names(self) -> dict[str, str]:
        names = {"embedding.table": "embed", "embedding_norm.weight": "embed.norm", "final_norm.weight": "final.norm"}
        for i, L in enumerate(self.layers):
            p, c = f"layers.{i}.", f"l{i}."
            names[p + "mixer_norm.weight"] = c + "norm1"
            if L.mlp is not None:
                names[p + "feed_forward_norm.weight"] = c + "norm2"
                for w in ("gate", "up", "down"):
                    names[p + "feed_forward." + w] = c + f"mlp.{w}"
                    names[p + f"feed_forward.{w}_bias"] = c + f"mlp.{w}.b"
            if L.type == "lightning":
                for w in ("q", "k", "v", "g", "o", "norm"):
                    names[p + "mixer." + w] = c + f"mix.{w}"
                continue
            for w in ("q", "k", "v", "o"):
                names[p + "mixer.left." + w] = c + f"mix.left.{w}"
            for w in ("q", "k"):
                names[p + f"mixer.left.{w}_norm"] = c + f"mix.left.{w}.norm"
            for w in ("q", "k", "v", "g", "o"):
                names[p + "mixer.right." + w] = c + f"mix.right.{w}"
        return names

    def optional_tensor_names(self) -> set[str]:
        """A layer without a feed-forward reads no second norm; a checkpoint may still hold one."""
        return {f"l{i}.norm2" for i, L in enumerate(self.layers) if L.mlp is None}

    def init_std(self) -> float:
        return self.initializer_range


register_architecture("Fazezen", FazezenConfig)
