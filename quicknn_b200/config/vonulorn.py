"""Vonulorn: typed configuration and its layout as parts.

A decoder whose layers are listed one by one in ``config.json``.

    {"architecture": "Vonulorn", "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m,
     "layers": [
       {"type": "delta", "mixer": {"heads", "kv_heads", "dim", "vdim", "conv"}, "mlp": {"kind": "dense", "ff"} | null},
       {"type": "attention",
        "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "diff", "q_temp": {"coef", "every"}}, "mlp": ...},
       {"type": "latent_attention",
        "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot": {"base", "dims"}}, "mlp": ...}]}

Pre-norm layers (RMS norms with plain weights), what a sublayer gives is multiplied by ``residual_mult``.  ``delta``: a gated delta
rule behind short convolutions.  ``attention``: differential attention, soft-capped, with queries that grow with the logarithm of
the position and no rotation.  ``latent_attention``: queries and keys/values through latents, a rotated key part shared by the
heads (interleaved pairs), a sink, no gate.  Feed-forward: a gated one (gelu).  The output matrix is a tensor of its own.

Checkpoint names: ``embed``, ``head``, ``final.norm``; layer i: ``l<i>.norm1``, ``.norm2``; ``l<i>.mix.q|k|v`` (+ ``.conv``),
``.b|a|A_log|dt_bias|norm|g|o``; ``l<i>.mix.q|k|v|lq1|lk1|lq2|lk2|o``; ``l<i>.mix.dq|dkv`` (+ ``.norm``), ``.uq|uk|uv|sink|o``;
``l<i>.mlp.gate|up|down``.
"""
from __future__ import annotations

import dataclasses
import math
from typing import Any, Dict, List, Optional, Tuple

from ..parts.spec import EmbeddingSpec, HeadSpec, LayerSpec, ModelSpec, PartSpec, default_schedule
from .base import Architecture, ModelConfig, as_float, as_int, register_architecture
from .linedra import MAX_POSITIONS, LatentConfig, _at_least_one, _eps, _obj, _req

LAYER_TYPES = ("delta", "attention", "latent_attention")
MLP_KINDS = ("dense",)


def _grouped(rec, where: str) -> List[str]:
    if rec.kv_heads >= 1 and rec.heads % rec.kv_heads:
        return [f"{where}: {rec.kv_heads} kv_heads do not divide {rec.heads} heads"]
    return []


@dataclasses.dataclass(frozen=True)
class DeltaConfig:
    """The ``delta`` mixer."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                        # taps

    @classmethod
    def parse(cls, m: Dict[str, Any]) -> "DeltaConfig":
        return cls(**{f.name: as_int(m.get(f.name)) for f in dataclasses.fields(cls)})

    def to_dict(self) -> Dict[str, Any]:
        return dataclasses.asdict(self)

    def problems(self, where: str) -> List[str]:
        p = _at_least_one(self, ("heads", "kv_heads", "dim", "vdim", "conv"), where) + _grouped(self, where)
        if self.dim > 256:
            p.append(f"{where}.dim must be <= 256 (got {self.dim})")
        return p


@dataclasses.dataclass(frozen=True)
class DifferentialConfig:
    """The ``attention`` mixer."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    softcap: Optional[float] = None
    temp_coef: Optional[float] = None        # q_temp; None: queries as projected
    temp_every: Optional[float] = None

    @classmethod
    def parse(cls, m: Dict[str, Any]) -> "DifferentialConfig":
        t, cap = m.get("q_temp"), m.get("softcap")
        t = None if t is None else _obj(t, "mixer.q_temp")
        return cls(scale=as_float(m.get("scale")), diff=as_float(m.get("diff")), softcap=None if cap is None else as_float(cap),
                   temp_coef=None if t is None else as_float(t.get("coef")),
                   temp_every=None if t is None else as_float(t.get("every")),
                   **{n: as_int(m.get(n)) for n in ("heads", "kv_heads", "dim", "vdim")})

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale, "diff": self.diff}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.temp_coef is not None:
            out["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return out

    def problems(self, where: str) -> List[str]:
        p = _at_least_one(self, ("heads", "kv_heads", "dim", "vdim"), where) + _grouped(self, where)
        for n in ("scale", "diff"):
            if not math.isfinite(getattr(self, n)):
                p.append(f"{where}.{n} must be finite (got {getattr(self, n)})")
        if self.softcap is not None and not (self.softcap > 0 and math.isfinite(self.softcap)):
            p.append(f"{where}.softcap must be > 0 or absent (got {self.softcap})")
        if self.temp_coef is not None:
            if not math.isfinite(self.temp_coef):
                p.append(f"{where}.q_temp.coef must be finite (got {self.temp_coef})")
            if not (self.temp_every > 0 and math.isfinite(self.temp_every)):
                p.append(f"{where}.q_temp.every must be > 0 (got {self.temp_every})")
        return p


MIXERS = {"delta": DeltaConfig, "attention": DifferentialConfig, "latent_attention": LatentConfig}


def _ff(v: Any) -> Optional[int]:
    """The inner width of a layer's feed-forward, None without one."""
    if v is None:
        return None
    v = _obj(v, "mlp")
    if v.get("kind") not in MLP_KINDS:
        raise ValueError(f"mlp.kind must be one of {MLP_KINDS} (got {v.get('kind')!r})")
    return as_int(v.get("ff"))


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: Any                       # DeltaConfig, DifferentialConfig or LatentConfig
    ff: Optional[int]

    @classmethod
    def parse(cls, v: Any) -> "LayerConfig":
        v = _obj(v, "a layer")
        kind = v.get("type")
        if kind not in LAYER_TYPES:
            raise ValueError(f"layer type must be one of {LAYER_TYPES} (got {kind!r})")
        return cls(kind, MIXERS[kind].parse(_obj(v.get("mixer"), "mixer")), _ff(v.get("mlp")))

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.ff is None else {"kind": "dense", "ff": self.ff}}

    def problems(self, where: str) -> List[str]:
        p = self.mixer.problems(where + ".mixer")
        if self.ff is not None and self.ff < 1:
            p.append(f"{where}.mlp.ff must be >= 1 (got {self.ff})")
        return p


def _layers(v: Any) -> Tuple[LayerConfig, ...]:
    if not isinstance(v, (list, tuple)) or not v:
        raise TypeError("layers must be a list with at least one entry")
    return tuple(LayerConfig.parse(x) for x in v)


@dataclasses.dataclass(frozen=True)
class VonulornConfig(ModelConfig):
    vocab: int = _req(as_int)
    width: int = _req(as_int)
    layers: Tuple[LayerConfig, ...] = _req(_layers)
    norm_eps: float = _req(_eps, key="norm")
    residual_mult: float = _req(as_float)
    architecture: str = dataclasses.field(default="Vonulorn", metadata={"convert": str})
    initializer_range: float = dataclasses.field(default=0.02, metadata={"convert": as_float})

    @classmethod
    def architecture_names(cls) -> Tuple[str, ...]:
        return ("Vonulorn",)

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult, "layers": [l.to_dict() for l in self.layers],
                "initializer_range": self.initializer_range}

    def problems(self) -> List[str]:
        p: List[str] = []
        if self.vocab < 1 or self.width < 1:
            p.append(f"vocab and width must be >= 1 (got {self.vocab}, {self.width})")
        if not self.norm_eps > 0:
            p.append(f"norm.eps must be > 0 (got {self.norm_eps})")
        if not math.isfinite(self.residual_mult):
            p.append(f"residual_mult must be finite (got {self.residual_mult})")
        if not (1 <= len(self.layers) <= 1024):
            p.append(f"between 1 and 1024 layers (got {len(self.layers)})")
        for i, layer in enumerate(self.layers):
            p.extend(layer.problems(f"layers[{i}]"))
        if not self.initializer_range > 0:
            p.append(f"initializer_range must be > 0 (got {self.initializer_range})")
        return p


def _delta(cfg: VonulornConfig, m: DeltaConfig, pre: str) -> Tuple[PartSpec, Dict[str, str]]:
    spec = PartSpec("delta_rule", {"hidden_size": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "dim": m.dim,
                                   "vdim": m.vdim, "conv": m.conv, "eps": cfg.norm_eps})
    names = {f"mixer.{n}": pre + n for n in ("q", "k", "v", "b", "a", "A_log", "dt_bias", "norm", "o")}
    names.update({f"mixer.{n}_conv": f"{pre}{n}.conv" for n in ("q", "k", "v")})
    names["mixer.gate"] = pre + "g"
    return spec, names


def _differential(cfg: VonulornConfig, m: DifferentialConfig, pre: str) -> Tuple[PartSpec, Dict[str, str]]:
    temp = None if m.temp_coef is None else {"coef": m.temp_coef, "every": m.temp_every}
    spec = PartSpec("differential_attention", {
        "hidden_size": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
        "softcap": m.softcap, "window": None, "diff": m.diff, "eps": cfg.norm_eps, "query_temperature": temp})
    return spec, {f"mixer.{n}": pre + n for n in ("q", "k", "v", "lq1", "lk1", "lq2", "lk2", "o")}


def _latent(cfg: VonulornConfig, m: LatentConfig, pre: str) -> Tuple[PartSpec, Dict[str, str]]:
    spec = PartSpec("latent_attention", {
        "hidden_size": cfg.width, "n_heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
        "scale": m.scale, "window": None, "eps": cfg.norm_eps, "sink": True, "gate": "none",
        "position": PartSpec("rotary", {"head_dim": m.rot_dim, "theta": m.rot_base, "rotary_dim": m.rot_dims,
                                        "layout": "interleaved"})})
    names = {f"mixer.{local}": pre + name for local, name in (
        ("dq", "dq"), ("dq_norm", "dq.norm"), ("uq", "uq"), ("dkv", "dkv"), ("dkv_norm", "dkv.norm"), ("uk", "uk"), ("uv", "uv"),
        ("sink", "sink"), ("o", "o"))}
    return spec, names


BUILD = {"delta": _delta, "attention": _differential, "latent_attention": _latent}


def vonulorn_spec(cfg: VonulornConfig) -> ModelSpec:
    W = cfg.width
    norm = PartSpec("rmsnorm", {"size": W, "eps": cfg.norm_eps, "unit_offset": False})
    block = PartSpec("prenorm", {"residual_mult": cfg.residual_mult})
    layers, optional = [], []
    for i, lc in enumerate(cfg.layers):
        pre = f"l{i}."
        mixer, tensors = BUILD[lc.type](cfg, lc.mixer, pre + "mix.")
        names = {"pre_mixer": "norm1"}
        ff = None
        if lc.ff is not None:
            ff = PartSpec("gated_mlp", {"hidden_size": W, "intermediate_size": lc.ff, "activation": "gelu_tanh"})
            tensors.update({f"ff.{n}_proj": f"{pre}mlp.{n}" for n in ("gate", "up", "down")})
            names["pre_ff"] = "norm2"
        else:                                    # a layer without a feed-forward may still carry the norm in front of it
            optional.append(pre + "norm2")
        tensors.update({f"norms.{local}.weight": pre + name for local, name in names.items()})
        layers.append(LayerSpec(block=block, mixer=mixer, feed_forward=ff, norms={n: norm for n in names}, tensors=tensors))
    return ModelSpec(
        name="Vonulorn", hidden_size=W, embedding=EmbeddingSpec(cfg.vocab, W, 1.0, "embed"), layers=tuple(layers),
        schedule=default_schedule(len(layers)),
        head=HeadSpec(cfg.vocab, W, tied=False, tensor="head", softcap=None, norm=norm, norm_tensor="final.norm"),
        max_positions=MAX_POSITIONS, stop_ids=(), init_std=cfg.initializer_range, init_norm_std=0.1,
        optional_tensors=tuple(optional))


VONULORN = register_architecture(Architecture(
    name="Vonulorn", config_cls=VonulornConfig, build_spec=vonulorn_spec, aliases=("vonulorn",)))
