"""Configuration of the Kivezen decoder: a list of layers, each with its own mixer (type and sizes) and feed-forward (or none), the number of residual
streams, and a run of layers that is gone through several times."""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass
class RotationSpec:
    dims: int
    base: float
    factor: float | None = None           # None: plain frequencies
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0


@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float                        # 0: none
    rot: RotationSpec


@dataclass
class LightningSpec:
    heads: int
    dim: int
    vdim: int
    decay: list[float]


@dataclass
class DenseSpec:
    ff: int


@dataclass
class GLUSpec:
    ff: int
    limit: float


@dataclass
class ExpertsSpec:
    experts: int
    top: int
    expert: GLUSpec
    shared: GLUSpec | None = None


@dataclass
class LayerSpec:
    mixer: AttentionSpec | LightningSpec
    mlp: DenseSpec | ExpertsSpec | None


@dataclass
class LoopSpec:
    start: int
    stop: int
    times: int


_SCALING = ("factor", "original", "fast", "slow")


def _whole(v, what: str) -> int:
    if int(v) != v:
        raise ValueError(f"{what}: {v} is not a whole number")
    return int(v)


def _mixer(kind: str, m: dict, what: str):
    size = lambda k: _whole(m[k], f"{what} {k}")  # noqa: E731
    if kind == "lightning":
        s = LightningSpec(size("heads"), size("dim"), size("vdim"), [float(d) for d in m["decay"]])
        if len(s.decay) != s.heads or not all(0.0 <= d <= 1.0 for d in s.decay):
            raise ValueError(f"{what}: decays {s.decay} for {s.heads} heads")
        return s
    if kind == "attention":
        r = m["rot"]
        scaling = {k: float(r["scaling"][k]) for k in _SCALING} if r.get("scaling") is not None else {}
        s = AttentionSpec(size("heads"), size("kv_heads"), size("dim"), size("vdim"), float(m["scale"]), float(m.get("softcap") or 0.0),
                          RotationSpec(_whole(r["dims"], f"{what} rotated dimensions"), float(r["base"]), **scaling))
        if s.heads < 1 or s.kv_heads < 1 or s.heads % s.kv_heads:
            raise ValueError(f"{what}: {s.heads} heads do not divide into {s.kv_heads} equal groups")
        if s.rot.dims % 2 or not 0 <= s.rot.dims <= s.dim or s.vdim % 2:
            raise ValueError(f"{what}: {s.rot.dims} rotated dimensions of {s.dim}, values of {s.vdim}")
        return s
    raise ValueError(f"{what}: unknown mixer type {kind!r}")


def _glu(d: dict) -> GLUSpec:
    return GLUSpec(int(d["ff"]), float(d["limit"]))


def _mlp(d: dict | None, what: str):
    if d is None:
        return None
    if d["kind"] == "dense":
        return DenseSpec(_whole(d["ff"], f"{what} ff"))
    if d["kind"] != "moe":
        raise ValueError(f"{what}: unknown feed-forward kind {d['kind']!r}")
    r = d["router"]
    s = ExpertsSpec(int(r["experts"]), int(r["top"]), _glu(d["expert"]), None if d.get("shared") is None else _glu(d["shared"]))
    if not 1 <= s.top <= s.experts:
        raise ValueError(f"{what}: {s.top} of {s.experts} experts")
    return s


@dataclass
class KivezenConfig:
    vocab: int
    width: int
    eps: float
    logit_softcap: float = 0.0            # 0: none
    streams: int | None = None            # None: the plain residual sum
    loop: LoopSpec | None = None
    layers: list[LayerSpec] = field(default_factory=list)
    name: str = "kivezen"

    num_mtp_layers = 0

    @staticmethod
    def from_json(d: dict) -> "KivezenConfig":
        try:
            layers = [LayerSpec(_mixer(e["type"], e["mixer"], f"layer {i}"), _mlp(e.get("mlp"), f"layer {i}")) for i, e in enumerate(d["layers"])]
            loop, streams = d.get("loop"), d.get("streams")
            if loop is not None:
                loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
                if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                    raise ValueError(f"layers {loop.start} to {loop.stop} of {len(layers)}, {loop.times} times")
            if streams is not None and not 1 <= _whole(streams, "residual streams") <= 16:
                raise ValueError(f"{streams} residual streams: 1 to 16 are served")
            return KivezenConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d.get("logit_softcap") or 0.0),
                                 None if streams is None else int(streams), loop, layers)
        except KeyError as ex:
            raise ValueError(f"config entry {ex} is missing") from None

    def to_json(self) -> dict:
        out = []
        for s in self.layers:
            m, e = s.mixer, s.mlp
            if isinstance(m, LightningSpec):
                j = vars(m)
            else:
                rot = {"dims": m.rot.dims, "base": m.rot.base}
                if m.rot.factor is not None:
                    rot["scaling"] = {k: getattr(m.rot, k) for k in _SCALING}
                j = {**vars(m), "rot": rot}
            if isinstance(e, DenseSpec):
                mlp = {"kind": "dense", "ff": e.ff}
            else:
                mlp = None if e is None else {"kind": "moe", "expert": vars(e.expert), "shared": None if e.shared is None else vars(e.shared),
                                              "router": {"experts": e.experts, "top": e.top}}
            out.append({"type": "lightning" if isinstance(m, LightningSpec) else "attention", "mixer": j, "mlp": mlp})
        d = {"architecture": "Kivezen", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": out,
             "logit_softcap": self.logit_softcap, "streams": self.streams}
        return d if self.loop is None else {**d, "loop": vars(self.loop)}

    def runs(self) -> list[int]:
        """The layers in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b = self.loop.start, self.loop.stop
        return [*range(a), *(list(range(a, b)) * self.loop.times), *range(b, n)]
