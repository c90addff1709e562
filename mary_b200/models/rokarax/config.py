"""Configuration of the Rokarax decoder: a list of layers, each with its own mixer (type and sizes) and feed-forward (or none)."""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass
class RotationSpec:
    dims: int
    base: float
    factor: float | None = None           # YaRN; None: plain frequencies
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0


@dataclass
class LatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int
    rot: RotationSpec


@dataclass
class StateSpaceSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    bias_max: float
    kv_from: int | None = None            # the layer whose keys and values this layer reads


@dataclass
class LayerSpec:
    mixer: LatentSpec | StateSpaceSpec | AttentionSpec
    ff: int | None                        # width of the dense feed-forward, None for a layer without one


_KINDS = {"latent_attention": LatentSpec, "mamba2": StateSpaceSpec, "attention": AttentionSpec}
_SCALING = ("factor", "original", "fast", "slow")


def _mixer(kind: str, m: dict, what: str):
    try:
        if kind == "mamba2":
            return StateSpaceSpec(**{k: int(m[k]) for k in StateSpaceSpec.__dataclass_fields__})
        window = int(m["mask"]["size"])
        if kind == "attention":
            return AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), window, float(m["bias_max"]),
                                 None if m.get("kv_from") is None else int(m["kv_from"]))
        r = m["rot"]
        scaling = {k: float(r["scaling"][k]) for k in _SCALING} if r.get("scaling") is not None else {}
        return LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]), float(m["scale"]),
                          window, RotationSpec(int(r["dims"]), float(r["base"]), **scaling))
    except KeyError as ex:
        raise ValueError(f"{what}: config entry {ex} is missing") from None


def _divides(n: int, k: int, what: str) -> None:
    if n < 1 or k < 1 or n % k:
        raise ValueError(f"{what}: {n} does not divide into {k} equal parts")


def _check(s, layers: list[LayerSpec], what: str) -> None:
    if isinstance(s, StateSpaceSpec):
        _divides(s.heads, s.groups, f"{what} groups")
        _divides(s.heads * s.vdim, s.norm_groups, f"{what} norm groups")
        return
    if s.window < 1:
        raise ValueError(f"{what}: a window of {s.window} positions")
    if isinstance(s, LatentSpec):
        if s.rot.dims != s.rot_dim or s.rot_dim % 2:
            raise ValueError(f"{what}: {s.rot.dims} rotated dimensions of a part of {s.rot_dim}")
        return
    _divides(s.heads, s.kv_heads, f"{what} heads")
    if s.kv_from is not None:
        src = layers[s.kv_from].mixer if 0 <= s.kv_from < len(layers) else None
        if not isinstance(src, AttentionSpec) or src.kv_from is not None:
            raise ValueError(f"{what}: layer {s.kv_from} has no keys and values of its own before this layer")
        if (src.heads, src.kv_heads, src.dim, src.vdim) != (s.heads, s.kv_heads, s.dim, s.vdim):
            raise ValueError(f"{what}: head sizes differ from those of layer {s.kv_from}")


@dataclass
class RokaraxConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: list[LayerSpec] = field(default_factory=list)
    name: str = "rokarax"

    num_mtp_layers = 0

    @staticmethod
    def from_json(d: dict) -> "RokaraxConfig":
        layers: list[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in _KINDS:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            mixer = _mixer(e["type"], e["mixer"], f"layer {i}")
            _check(mixer, layers, f"layer {i}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(LayerSpec(mixer, None if mlp is None else int(mlp["ff"])))
        return RokaraxConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]), layers)

    def to_json(self) -> dict:
        out = []
        for s in self.layers:
            m = {k: v for k, v in vars(s.mixer).items() if k not in ("window", "rot") and v is not None}
            if not isinstance(s.mixer, StateSpaceSpec):
                m["mask"] = {"size": s.mixer.window}
            if isinstance(s.mixer, LatentSpec):
                r = s.mixer.rot
                m["rot"] = {"dims": r.dims, "base": r.base}
                if r.factor is not None:
                    m["rot"]["scaling"] = {k: getattr(r, k) for k in _SCALING}
            out.append({"type": next(k for k, c in _KINDS.items() if isinstance(s.mixer, c)), "mixer": m,
                        "mlp": None if s.ff is None else {"kind": "dense", "ff": s.ff}})
        return {"architecture": "Rokarax", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "layers": out}
