"""Linedra: typed configuration and its layout as parts.

A decoder whose layers are listed one by one in ``config.json``.

    {"architecture": "Linedra", "vocab": V, "width": W, "embedding": {"scale": s}, "norm": {"eps": e}, "canon": {"taps": t},
     "residual_mult": m, "logit_softcap": c,
     "layers": [
       {"type": "parallel",
        "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}},
                  "right": {"width", "blocks", "conv"}, "left_scale", "right_scale"},
        "mlp": {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"}} | null},
       {"type": "latent_attention",
        "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot": {"base", "dims"}}, "mlp": ...}]}

Layers have a norm before and after each sublayer (RMS norms whose weights are stored around zero), what a sublayer gives is
multiplied by ``residual_mult``; what the mixer reads is its normed input plus a causal convolution of it (``canon.taps``
taps); after every layer the stream becomes a learned weighted sum of the embedded rows and all layers' results.
``parallel``: a windowed softmax attention with a distance bias, a sink and a gate per head (left) beside a real-gated linear
recurrence (right), summed with fixed numbers.  ``latent_attention``: queries and keys/values through latents, a rotated
key part shared by the heads, a sink, a gate per element.  Feed-forward: experts with a clamped gate, weights by a softmax over
the chosen logits.  The output matrix is the embedding table, with a softcap on the logits.

Checkpoint names: ``embed``, ``final.norm``; layer i: ``l<i>.norm1``, ``.norm1b``, ``.norm2``, ``.norm2b``, ``.canon1``, ``.dwa``;
``l<i>.mix.left.q|k|v|sink|g|o``; ``l<i>.mix.right.y|x|conv|ra|ri`` (+ ``.b``), ``.lam``, ``.o``;
``l<i>.mix.dq|dkv`` (+ ``.norm``), ``.uq|uk|uv|sink|g|o``; ``l<i>.mlp.router``, ``l<i>.mlp.e<n>.gate|up|down``.
"""
from __future__ import annotations

import dataclasses
import math
from typing import Any, Dict, List, Optional, Tuple

from ..parts.spec import EmbeddingSpec, HeadSpec, LayerSpec, ModelSpec, PartSpec, default_schedule
from .base import Architecture, ModelConfig, as_float, as_int, as_opt_float, register_architecture
from .mubasun import distance_slopes

LAYER_TYPES = ("parallel", "latent_attention")
MLP_KINDS = ("moe",)
MAX_POSITIONS = 1 << 20          # rotations have no table; this only bounds a cache's longest sequence


def _obj(v: Any, what: str) -> Dict[str, Any]:
    if not isinstance(v, dict):
        raise TypeError(f"{what} must be an object, got {v!r}")
    return v


def _at_least_one(rec, names, where: str) -> List[str]:
    return [f"{where}.{n} must be >= 1 (got {getattr(rec, n)})" for n in names if getattr(rec, n) < 1]


@dataclasses.dataclass(frozen=True)
class WindowAttentionConfig:
    """The left branch of ``parallel``."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None             # mask.size; None: every earlier position

    @classmethod
    def parse(cls, m: Dict[str, Any], where: str) -> "WindowAttentionConfig":
        mask = m.get("mask")
        size = None if mask is None else _obj(mask, where + ".mask").get("size")
        return cls(heads=as_int(m.get("heads")), kv_heads=as_int(m.get("kv_heads")), dim=as_int(m.get("dim")),
                   vdim=as_int(m.get("vdim")), scale=as_float(m.get("scale")), window=None if size is None else as_int(size))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out

    def problems(self, where: str) -> List[str]:
        p = _at_least_one(self, ("heads", "kv_heads", "dim", "vdim"), where)
        if self.kv_heads >= 1 and self.heads % self.kv_heads:
            p.append(f"{where}: {self.kv_heads} kv_heads do not divide {self.heads} heads")
        if not math.isfinite(self.scale):
            p.append(f"{where}.scale must be finite (got {self.scale})")
        if self.window is not None and self.window < 1:
            p.append(f"{where}.mask.size must be >= 1 (got {self.window})")
        return p


@dataclasses.dataclass(frozen=True)
class RecurrenceConfig:
    """The right branch of ``parallel``."""

    width: int
    blocks: int
    conv: int

    @classmethod
    def parse(cls, m: Dict[str, Any]) -> "RecurrenceConfig":
        return cls(width=as_int(m.get("width")), blocks=as_int(m.get("blocks")), conv=as_int(m.get("conv")))

    def to_dict(self) -> Dict[str, Any]:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}

    def problems(self, where: str) -> List[str]:
        p = _at_least_one(self, ("width", "blocks", "conv"), where)
        if self.blocks >= 1 and self.width % self.blocks:
            p.append(f"{where}: {self.blocks} blocks do not divide the width {self.width}")
        return p


@dataclasses.dataclass(frozen=True)
class LatentConfig:
    """The ``latent_attention`` mixer."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int

    @classmethod
    def parse(cls, m: Dict[str, Any]) -> "LatentConfig":
        rot = _obj(m.get("rot"), "mixer.rot")
        return cls(rot_base=as_float(rot.get("base")), rot_dims=as_int(rot.get("dims")), scale=as_float(m.get("scale")),
                   **{n: as_int(m.get(n)) for n in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")})

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": {"base": self.rot_base, "dims": self.rot_dims}}

    def problems(self, where: str) -> List[str]:
        p = _at_least_one(self, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"), where)
        if self.rot_dims != self.rot_dim or self.rot_dim % 2:
            p.append(f"{where}: rot.dims must equal rot_dim and be even (got {self.rot_dims} and {self.rot_dim})")
        if not (self.rot_base > 0 and math.isfinite(self.rot_base)):
            p.append(f"{where}.rot.base must be > 0 (got {self.rot_base})")
        if not math.isfinite(self.scale):
            p.append(f"{where}.scale must be finite (got {self.scale})")
        return p


@dataclasses.dataclass(frozen=True)
class MlpConfig:
    ff: int                          # inner width of one expert
    limit: float
    experts: int
    top: int

    @classmethod
    def parse(cls, v: Any) -> Optional["MlpConfig"]:
        if v is None:
            return None
        v = _obj(v, "mlp")
        if v.get("kind") not in MLP_KINDS:
            raise ValueError(f"mlp.kind must be one of {MLP_KINDS} (got {v.get('kind')!r})")
        e, r = _obj(v.get("expert"), "mlp.expert"), _obj(v.get("router"), "mlp.router")
        return cls(as_int(e.get("ff")), as_float(e.get("limit")), as_int(r.get("experts")), as_int(r.get("top")))

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit},
                "router": {"experts": self.experts, "top": self.top}}

    def problems(self, where: str) -> List[str]:
        p: List[str] = []
        if self.ff < 1:
            p.append(f"{where}.expert.ff must be >= 1 (got {self.ff})")
        if not (self.limit > 0 and math.isfinite(self.limit)):
            p.append(f"{where}.expert.limit must be > 0 (got {self.limit})")
        if self.experts < 1 or not (1 <= self.top <= min(16, self.experts)):
            p.append(f"{where}.router.top must lie between 1 and min(16, experts) (got {self.top} of {self.experts})")
        return p


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    type: str
    mlp: Optional[MlpConfig]
    left: Optional[WindowAttentionConfig] = None
    right: Optional[RecurrenceConfig] = None
    left_scale: float = 1.0
    right_scale: float = 1.0
    latent: Optional[LatentConfig] = None

    @classmethod
    def parse(cls, v: Any) -> "LayerConfig":
        v = _obj(v, "a layer")
        kind = v.get("type")
        if kind not in LAYER_TYPES:
            raise ValueError(f"layer type must be one of {LAYER_TYPES} (got {kind!r})")
        m, mlp = _obj(v.get("mixer"), "mixer"), MlpConfig.parse(v.get("mlp"))
        if kind == "latent_attention":
            return cls(kind, mlp, latent=LatentConfig.parse(m))
        return cls(kind, mlp, left=WindowAttentionConfig.parse(_obj(m.get("left"), "mixer.left"), "mixer.left"),
                   right=RecurrenceConfig.parse(_obj(m.get("right"), "mixer.right")),
                   left_scale=as_float(m.get("left_scale")), right_scale=as_float(m.get("right_scale")))

    def to_dict(self) -> Dict[str, Any]:
        if self.type == "latent_attention":
            mixer = self.latent.to_dict()
        else:
            mixer = {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                     "right_scale": self.right_scale}
        return {"type": self.type, "mixer": mixer, "mlp": None if self.mlp is None else self.mlp.to_dict()}

    def problems(self, where: str) -> List[str]:
        p: List[str] = []
        if self.latent is not None:
            p.extend(self.latent.problems(where + ".mixer"))
        else:
            p.extend(self.left.problems(where + ".mixer.left"))
            p.extend(self.right.problems(where + ".mixer.right"))
            if not (math.isfinite(self.left_scale) and math.isfinite(self.right_scale)):
                p.append(f"{where}.mixer: left_scale and right_scale must be finite")
        if self.mlp is not None:
            p.extend(self.mlp.problems(where + ".mlp"))
        return p


def _layers(v: Any) -> Tuple[LayerConfig, ...]:
    if not isinstance(v, (list, tuple)) or not v:
        raise TypeError("layers must be a list with at least one entry")
    return tuple(LayerConfig.parse(x) for x in v)


def _eps(v: Any) -> float:
    return as_float(_obj(v, "norm").get("eps"))


def _embedding_scale(v: Any) -> float:
    return as_float(_obj(v, "embedding").get("scale"))


def _taps(v: Any) -> int:
    return as_int(_obj(v, "canon").get("taps"))


def _req(conv, key=None):
    md = {"convert": conv, "required": True}
    if key:
        md["key"] = key
    return dataclasses.field(default=None, metadata=md)


@dataclasses.dataclass(frozen=True)
class LinedraConfig(ModelConfig):
    vocab: int = _req(as_int)
    width: int = _req(as_int)
    layers: Tuple[LayerConfig, ...] = _req(_layers)
    norm_eps: float = _req(_eps, key="norm")
    embedding_scale: float = _req(_embedding_scale, key="embedding")
    canon_taps: int = _req(_taps, key="canon")
    residual_mult: float = _req(as_float)
    logit_softcap: Optional[float] = dataclasses.field(default=None, metadata={"convert": as_opt_float})
    architecture: str = dataclasses.field(default="Linedra", metadata={"convert": str})
    initializer_range: float = dataclasses.field(default=0.02, metadata={"convert": as_float})

    @classmethod
    def architecture_names(cls) -> Tuple[str, ...]:
        return ("Linedra",)

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                "canon": {"taps": self.canon_taps}, "residual_mult": self.residual_mult, "logit_softcap": self.logit_softcap,
                "layers": [l.to_dict() for l in self.layers], "initializer_range": self.initializer_range}

    def problems(self) -> List[str]:
        p: List[str] = []
        if self.vocab < 1 or self.width < 1:
            p.append(f"vocab and width must be >= 1 (got {self.vocab}, {self.width})")
        if not self.norm_eps > 0:
            p.append(f"norm.eps must be > 0 (got {self.norm_eps})")
        if not math.isfinite(self.embedding_scale):
            p.append(f"embedding.scale must be finite (got {self.embedding_scale})")
        if self.canon_taps < 1:
            p.append(f"canon.taps must be >= 1 (got {self.canon_taps})")
        if not math.isfinite(self.residual_mult):
            p.append(f"residual_mult must be finite (got {self.residual_mult})")
        if self.logit_softcap is not None and not (self.logit_softcap > 0 and math.isfinite(self.logit_softcap)):
            p.append(f"logit_softcap must be > 0 or null (got {self.logit_softcap})")
        if not (1 <= len(self.layers) <= 1024):
            p.append(f"between 1 and 1024 layers (got {len(self.layers)})")
        for i, layer in enumerate(self.layers):
            p.extend(layer.problems(f"layers[{i}]"))
        if not self.initializer_range > 0:
            p.append(f"initializer_range must be > 0 (got {self.initializer_range})")
        return p


def _parallel(cfg: LinedraConfig, lc: LayerConfig, pre: str) -> Tuple[PartSpec, Dict[str, str]]:
    W, a, r = cfg.width, lc.left, lc.right
    left = PartSpec("attention", {
        "hidden_size": W, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim,
        "scale": a.scale, "softcap": None, "window": a.window, "position": PartSpec("none", {"head_dim": a.dim}),
        "distance_slopes": distance_slopes(a.heads), "sink": True, "head_gate": True})
    right = PartSpec("rglru", {"hidden_size": W, "width": r.width, "blocks": r.blocks, "conv": r.conv})
    names = {f"mixer.left.{n}_proj": f"{pre}left.{n}" for n in ("q", "k", "v", "o")}
    names.update({"mixer.left.sink": pre + "left.sink", "mixer.left.head_gate": pre + "left.g"})
    for local, name in (("y", "y"), ("x", "x"), ("conv", "conv"), ("r", "ra"), ("i", "ri")):
        names[f"mixer.right.{local}"] = f"{pre}right.{name}"
        names[f"mixer.right.{local}_bias"] = f"{pre}right.{name}.b"
    names.update({"mixer.right.lam": pre + "right.lam", "mixer.right.o": pre + "right.o"})
    spec = PartSpec("parallel", {"hidden_size": W, "eps": cfg.norm_eps, "branches": {"left": left, "right": right},
                                 "scales": {"left": lc.left_scale, "right": lc.right_scale}})
    return spec, names


def _latent(cfg: LinedraConfig, m: LatentConfig, pre: str) -> Tuple[PartSpec, Dict[str, str]]:
    spec = PartSpec("latent_attention", {
        "hidden_size": cfg.width, "n_heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
        "scale": m.scale, "window": None, "eps": cfg.norm_eps, "sink": True, "gate": "element",
        "position": PartSpec("rotary", {"head_dim": m.rot_dim, "theta": m.rot_base, "rotary_dim": m.rot_dims})})
    names = {f"mixer.{local}": pre + name for local, name in (
        ("dq", "dq"), ("dq_norm", "dq.norm"), ("uq", "uq"), ("dkv", "dkv"), ("dkv_norm", "dkv.norm"), ("uk", "uk"), ("uv", "uv"),
        ("sink", "sink"), ("gate", "g"), ("o", "o"))}
    return spec, names


def _experts(cfg: LinedraConfig, m: MlpConfig, pre: str) -> Tuple[PartSpec, Dict[str, str]]:
    names = {"ff.router": pre + "router"}
    for e in range(m.experts):
        for n in ("gate", "up", "down"):
            names[f"ff.experts.{e}.{n}_proj"] = f"{pre}e{e}.{n}"
    # a softmax over the chosen logits is the softmax over all of them, renormalised over the chosen
    spec = PartSpec("routed_experts", {
        "hidden_size": cfg.width, "experts": m.experts, "top": m.top, "intermediate_size": m.ff, "limit": m.limit,
        "score": "softmax", "renormalize": True, "weight_on": "output"})
    return spec, names


def linedra_spec(cfg: LinedraConfig) -> ModelSpec:
    W = cfg.width
    norm = PartSpec("rmsnorm", {"size": W, "eps": cfg.norm_eps, "unit_offset": True})
    layers, optional = [], []
    for i, lc in enumerate(cfg.layers):
        pre = f"l{i}."
        mixer, tensors = (_parallel(cfg, lc, pre + "mix.") if lc.type == "parallel" else _latent(cfg, lc.latent, pre + "mix."))
        names = {"pre_mixer": "norm1", "post_mixer": "norm1b"}
        ff = None
        if lc.mlp is not None:
            ff, more = _experts(cfg, lc.mlp, pre + "mlp.")
            tensors.update(more)
            names.update({"pre_ff": "norm2", "post_ff": "norm2b"})
        else:                                    # a layer without a feed-forward may still carry the norms around it
            optional += [pre + "norm2", pre + "norm2b"]
        tensors.update({f"norms.{local}.weight": pre + name for local, name in names.items()})
        tensors.update({"input_conv": pre + "canon1", "depth_average": pre + "dwa"})
        block = PartSpec("sandwich", {"hidden_size": W, "residual_mult": cfg.residual_mult, "input_conv": cfg.canon_taps,
                                      "depth_average": i + 2})
        layers.append(LayerSpec(block=block, mixer=mixer, feed_forward=ff, norms={n: norm for n in names}, tensors=tensors))
    return ModelSpec(
        name="Linedra", hidden_size=W, embedding=EmbeddingSpec(cfg.vocab, W, cfg.embedding_scale, "embed"),
        layers=tuple(layers), schedule=default_schedule(len(layers)),
        head=HeadSpec(cfg.vocab, W, tied=True, tensor=None, softcap=cfg.logit_softcap, norm=norm, norm_tensor="final.norm"),
        max_positions=MAX_POSITIONS, stop_ids=(), depth_history=True, init_std=cfg.initializer_range, init_norm_std=0.1,
        optional_tensors=tuple(optional))


LINEDRA = register_architecture(Architecture(
    name="Linedra", config_cls=LinedraConfig, build_spec=linedra_spec, aliases=("linedra",)))
