"""Configuration of the Tatizen decoder: a list of layers, each with its own mixer (type and sizes) and feed-forward (or none)."""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float


@dataclass
class DecayedLinearSpec:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass
class ParallelSpec:
    left: AttentionSpec
    right: DecayedLinearSpec
    left_scale: float
    right_scale: float


@dataclass
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass
class LayerSpec:
    mixer: ParallelSpec | DeltaSpec
    ff: int | None                        # width of the dense feed-forward, None for a layer without one


def _pick(cls, d: dict, what: str):
    try:
        return cls(**{k: d[k] for k in cls.__dataclass_fields__})
    except KeyError as ex:
        raise ValueError(f"{what}: config entry {ex} is missing") from None


def _check_heads(heads: int, kv_heads: int, what: str) -> None:
    if heads < 1 or kv_heads < 1 or heads % kv_heads:
        raise ValueError(f"{what}: {heads} heads do not divide into {kv_heads} key/value heads")


@dataclass
class TatizenConfig:
    vocab: int
    width: int
    eps: float
    layers: list[LayerSpec] = field(default_factory=list)
    name: str = "tatizen"

    num_mtp_layers = 0

    @staticmethod
    def from_json(d: dict) -> "TatizenConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, kind = e["mixer"], e["type"]
            if kind == "parallel":
                mixer = ParallelSpec(_pick(AttentionSpec, m["left"], f"layer {i} left"), _pick(DecayedLinearSpec, m["right"], f"layer {i} right"),
                                     float(m["left_scale"]), float(m["right_scale"]))
                _check_heads(mixer.left.heads, mixer.left.kv_heads, f"layer {i}")
            elif kind == "delta":
                mixer = _pick(DeltaSpec, m, f"layer {i}")
                _check_heads(mixer.heads, mixer.kv_heads, f"layer {i}")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(LayerSpec(mixer, None if mlp is None else int(mlp["ff"])))
        return TatizenConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers)

    def to_json(self) -> dict:
        out = []
        for s in self.layers:
            if isinstance(s.mixer, ParallelSpec):
                m = dict(left=dict(vars(s.mixer.left)), right=dict(vars(s.mixer.right)), left_scale=s.mixer.left_scale, right_scale=s.mixer.right_scale)
            else:
                m = dict(vars(s.mixer))
            out.append({"type": "parallel" if isinstance(s.mixer, ParallelSpec) else "delta", "mixer": m,
                        "mlp": None if s.ff is None else {"kind": "dense", "ff": s.ff}})
        return {"architecture": "Tatizen", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": out}
