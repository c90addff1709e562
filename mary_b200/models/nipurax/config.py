"""Configuration of the Nipurax decoder: a list of layers, each with its own mixer (type and sizes) and mixture of experts (or none), and a
run of layers that is gone through several times."""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass
class RotationSpec:
    dims: int
    base: float
    factor: float | None = None           # None: plain frequencies
    low: float = 0.0
    high: float = 0.0
    original: float = 0.0


@dataclass
class DifferentialSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int
    diff: float
    rot: RotationSpec


@dataclass
class CappedSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    temp_coef: float
    temp_every: int


@dataclass
class GLUSpec:
    ff: int
    limit: float


@dataclass
class ExpertsSpec:
    experts: int
    identity: int
    top: int
    scale: float
    expert: GLUSpec
    shared: GLUSpec | None = None


@dataclass
class LayerSpec:
    mixer: DifferentialSpec | CappedSpec
    mlp: ExpertsSpec | None


@dataclass
class PairsSpec:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class LoopSpec:
    start: int
    stop: int
    times: int


_SCALING = ("factor", "low", "high", "original")
_HEADS = ("heads", "kv_heads", "dim", "vdim")


def _whole(v, what: str) -> int:
    if int(v) != v:
        raise ValueError(f"{what}: {v} is not a whole number")
    return int(v)


def _mixer(kind: str, m: dict, what: str):
    heads = [_whole(m[k], f"{what} {k}") for k in _HEADS]
    if kind == "attention":
        r = m["rot"]
        scaling = {k: float(r["scaling"][k]) for k in _SCALING} if r.get("scaling") is not None else {}
        return DifferentialSpec(*heads, float(m["scale"]), _whole(m["mask"]["size"], f"{what} chunk"), float(m["diff"]),
                                RotationSpec(int(r["dims"]), float(r["base"]), **scaling))
    if kind == "attention_2":
        t = m["q_temp"]
        return CappedSpec(*heads, float(m["scale"]), float(m["softcap"]), float(t["coef"]), _whole(t["every"], f"{what} temperature step"))
    raise ValueError(f"{what}: unknown mixer type {kind!r}")


def _glu(d: dict) -> GLUSpec:
    return GLUSpec(int(d["ff"]), float(d["limit"]))


def _mlp(d: dict | None, what: str) -> ExpertsSpec | None:
    if d is None:
        return None
    if d.get("kind") != "moe":
        raise ValueError(f"{what}: unknown feed-forward kind {d.get('kind')!r}")
    r = d["router"]
    return ExpertsSpec(int(r["experts"]), int(r.get("identity", 0)), int(r["top"]), float(r["scale"]), _glu(d["expert"]),
                       None if d.get("shared") is None else _glu(d["shared"]))


def _check(s, what: str) -> None:
    if s.heads < 1 or s.kv_heads < 1 or s.heads % s.kv_heads:
        raise ValueError(f"{what}: {s.heads} heads do not divide into {s.kv_heads} equal groups")
    if isinstance(s, CappedSpec):
        if s.softcap <= 0 or s.temp_every < 1:
            raise ValueError(f"{what}: a cap of {s.softcap}, a temperature step of {s.temp_every}")
    else:
        if s.chunk < 1:
            raise ValueError(f"{what}: chunks of {s.chunk} positions")
        if s.rot.dims % 2 or not 0 <= s.rot.dims <= s.dim:
            raise ValueError(f"{what}: {s.rot.dims} rotated dimensions of {s.dim}")


@dataclass
class NipuraxConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    pairs: PairsSpec
    loop: LoopSpec | None = None
    layers: list[LayerSpec] = field(default_factory=list)
    name: str = "nipurax"

    num_mtp_layers = 0

    @staticmethod
    def from_json(d: dict) -> "NipuraxConfig":
        try:
            layers = [LayerSpec(_mixer(e["type"], e["mixer"], f"layer {i}"), _mlp(e.get("mlp"), f"layer {i}")) for i, e in enumerate(d["layers"])]
            for i, s in enumerate(layers):
                _check(s.mixer, f"layer {i}")
            b, loop = d["embedding"]["bigram"], d.get("loop")
            if loop is not None:
                loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
                if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                    raise ValueError(f"layers {loop.start} to {loop.stop} of {len(layers)}, {loop.times} times")
            return NipuraxConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["residual_mult"]),
                                 PairsSpec(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])), loop, layers)
        except KeyError as ex:
            raise ValueError(f"config entry {ex} is missing") from None

    def to_json(self) -> dict:
        out = []
        for s in self.layers:
            m, e = s.mixer, s.mlp
            j = {**{k: getattr(m, k) for k in _HEADS}, "scale": m.scale}
            if isinstance(m, CappedSpec):
                j.update(softcap=m.softcap, q_temp={"coef": m.temp_coef, "every": m.temp_every})
            else:
                rot = {"dims": m.rot.dims, "base": m.rot.base}
                if m.rot.factor is not None:
                    rot["scaling"] = {k: getattr(m.rot, k) for k in _SCALING}
                j.update(mask={"size": m.chunk}, diff=m.diff, rot=rot)
            mlp = None if e is None else {"kind": "moe", "expert": vars(e.expert), "shared": None if e.shared is None else vars(e.shared),
                                          "router": {"experts": e.experts, "identity": e.identity, "top": e.top, "scale": e.scale}}
            out.append({"type": "attention_2" if isinstance(m, CappedSpec) else "attention", "mixer": j, "mlp": mlp})
        d = {"architecture": "Nipurax", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "residual_mult": self.residual_mult,
             "embedding": {"bigram": vars(self.pairs)}, "layers": out}
        return d if self.loop is None else {**d, "loop": vars(self.loop)}

    def runs(self) -> list[tuple[int, int | None]]:
        """``(layer, pass)`` in the order they run; ``pass`` is set at the first layer of a pass through the loop."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        a, b = self.loop.start, self.loop.stop
        return [(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(self.loop.times) for i in range(a, b)] + \
            [(i, None) for i in range(b, n)]
