"""Typed configuration of the Kasarax decoder, read from its config.json.

Keys: `architecture` ("Kasarax"), `vocab`, `width`, `norm.eps`, optional `logit_scale`, `layers` (a list; each entry has `type`:
"attention" or "parallel", `mixer` with that mixer's sizes and constants, and `mlp`: null, `{kind: dense, ff}` or `{kind: moe, expert:
{ff}, router: {experts, top}}`), optional `max_positions` (the design has no position limit; the engine needs one for its tables of
angles and query temperatures) and optional `eos_token_ids`.

attention mixer: heads, kv_heads, dim, vdim, scale, optional q_temp {coef, every}. parallel mixer: `left` (heads, kv_heads, dim, vdim,
scale, conv (taps), optional rot {dims, base}) and `right` (heads, dim, vdim, decay: a number a head).
A size that the file leaves out and a tensor's shape gives is read from the checkpoint's header when a model folder is opened
(`sizes_from_tensors`).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Dict, FrozenSet, Optional, Tuple, Union

from .files import ConfigError
from .vapelix import DEFAULT_MAX_POSITIONS, _need


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: float


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[QueryTemperature] = None


@dataclass(frozen=True)
class ConvAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    taps: int
    rot_dims: int = 0      # 0: positions do not enter the scores
    rot_base: float = 10000.0


@dataclass(frozen=True)
class LightningMixer:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class ParallelMixer:
    left: ConvAttention
    right: LightningMixer


@dataclass(frozen=True)
class DenseFF:
    ff: int


@dataclass(frozen=True)
class MoEFF:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class KasaraxLayer:
    type: str  # "attention" | "parallel"
    mixer: Union[AttentionMixer, ParallelMixer]
    mlp: Union[None, DenseFF, MoEFF]


def _sizes(m: Dict[str, Any], w: str, keys=("heads", "kv_heads", "dim", "vdim")) -> Dict[str, int]:
    return {k: int(_need(m, k, w)) for k in keys}


@dataclass(frozen=True)
class KasaraxConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: Tuple[KasaraxLayer, ...]
    logit_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: FrozenSet[int] = field(default_factory=frozenset)

    # names shared with the other configurations (the command line and the scheduler read them)
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, j: Dict[str, Any], generation: Optional[Dict[str, Any]] = None) -> "KasaraxConfig":
        width, vocab = int(_need(j, "width", "config.json")), int(_need(j, "vocab", "config.json"))
        eps = float(_need(_need(j, "norm", "config.json"), "eps", "norm"))
        raw_layers = _need(j, "layers", "config.json")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind, m, w = _need(e, "type", where), _need(e, "mixer", where), where + ".mixer"
            if kind == "attention":
                t = m.get("q_temp")
                temp = QueryTemperature(float(_need(t, "coef", w + ".q_temp")), float(_need(t, "every", w + ".q_temp"))) if t else None
                mixer: Union[AttentionMixer, ParallelMixer] = AttentionMixer(**_sizes(m, w), scale=float(_need(m, "scale", w)), q_temp=temp)
            elif kind == "parallel":
                a, r = _need(m, "left", w), _need(m, "right", w)
                rot, decay = a.get("rot"), _need(r, "decay", w + ".right")
                if not isinstance(decay, list):
                    raise ConfigError(f"config.json: {w}.right.decay must be a list with a number a head")
                left = ConvAttention(**_sizes(a, w + ".left"), scale=float(_need(a, "scale", w + ".left")), taps=int(_need(a, "conv", w + ".left")),
                                     rot_dims=int(_need(rot, "dims", w + ".left.rot")) if rot else 0,
                                     rot_base=float(_need(rot, "base", w + ".left.rot")) if rot else 10000.0)
                mixer = ParallelMixer(left, LightningMixer(**_sizes(r, w + ".right", ("heads", "dim", "vdim")), decay=tuple(float(d) for d in decay)))
            else:
                raise ConfigError(f"config.json: {where}: unknown layer type '{kind}' (attention, parallel)")
            f, fw = e.get("mlp"), where + ".mlp"
            mlp: Union[None, DenseFF, MoEFF] = None
            if f:
                fk = _need(f, "kind", fw)
                if fk == "dense":
                    mlp = DenseFF(int(_need(f, "ff", fw)))
                elif fk == "moe":
                    router = _need(f, "router", fw)
                    mlp = MoEFF(ff=int(_need(_need(f, "expert", fw), "ff", fw + ".expert")), experts=int(_need(router, "experts", fw + ".router")),
                                top=int(_need(router, "top", fw + ".router")))
                else:
                    raise ConfigError(f"config.json: {fw}: unknown kind '{fk}' (dense, moe)")
            layers.append(KasaraxLayer(kind, mixer, mlp))
        logit_scale = j.get("logit_scale")
        cfg = cls(architecture=j.get("architecture", "Kasarax"), vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                  logit_scale=1.0 if logit_scale is None else float(logit_scale), max_positions=int(j.get("max_positions") or DEFAULT_MAX_POSITIONS),
                  eos_token_ids=frozenset(int(t) for t in j.get("eos_token_ids") or []))
        cfg.check()
        return cfg

    def check(self) -> None:
        if self.width <= 0 or self.vocab <= 0 or self.eps < 0 or self.max_positions <= 0:
            raise ConfigError("config.json: width, vocab and max_positions must be positive, eps not negative")
        for i, l in enumerate(self.layers):
            where = f"config.json: layers[{i}]"
            a = l.mixer if l.type == "attention" else l.mixer.left
            aw = f"{where}.mixer" if l.type == "attention" else f"{where}.mixer.left"
            if min(a.heads, a.kv_heads, a.dim, a.vdim) <= 0 or a.heads % a.kv_heads:
                raise ConfigError(f"{aw}: sizes must be positive and heads a multiple of kv_heads")
            if l.type == "attention":
                t = a.q_temp
                if t is not None and not t.every > 0:
                    raise ConfigError(f"{aw}.q_temp: every must be positive")
            else:
                r = l.mixer.right
                if a.taps < 1:
                    raise ConfigError(f"{aw}.conv: there is at least one tap")
                if a.rot_dims < 0 or a.rot_dims % 2 or a.rot_dims > a.dim or not a.rot_base > 0:
                    raise ConfigError(f"{aw}.rot: dims must be even and at most dim, base positive")
                if min(r.heads, r.dim, r.vdim) <= 0 or len(r.decay) != r.heads:
                    raise ConfigError(f"{where}.mixer.right: sizes must be positive, and decay has a number a head")
                if not all(0.0 <= d <= 1.0 for d in r.decay):
                    raise ConfigError(f"{where}.mixer.right.decay: every decay lies in [0, 1]")
            f = l.mlp
            if isinstance(f, DenseFF) and f.ff <= 0:
                raise ConfigError(f"{where}.mlp: ff must be positive")
            if isinstance(f, MoEFF) and (f.ff <= 0 or f.experts < 1 or not 1 <= f.top <= f.experts):
                raise ConfigError(f"{where}.mlp: {f.top} of {f.experts} experts of {f.ff}")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for l in self.layers:
            m = l.mixer
            if l.type == "attention":
                mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
                if m.q_temp is not None:
                    mixer["q_temp"] = {"coef": m.q_temp.coef, "every": m.q_temp.every}
            else:
                a, r = m.left, m.right
                left: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "conv": a.taps}
                if a.rot_dims:
                    left["rot"] = {"dims": a.rot_dims, "base": a.rot_base}
                mixer = {"left": left, "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay)}}
            f, mlp = l.mlp, None
            if isinstance(f, DenseFF):
                mlp = {"kind": "dense", "ff": f.ff}
            elif isinstance(f, MoEFF):
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                               "logit_scale": self.logit_scale, "layers": layers, "max_positions": self.max_positions}
        if self.eos_token_ids:
            out["eos_token_ids"] = sorted(self.eos_token_ids)
        return out


def sizes_from_tensors(j: Dict[str, Any], shape_of: Callable[[str], Optional[Tuple[int, ...]]]) -> Dict[str, Any]:
    """Sizes that the file leaves out and a tensor's shape gives, written into a copy of the configuration. shape_of(name) -> the
    checkpoint's shape of that tensor, or None. What the file says is never overruled here (the loader reports a disagreement)."""
    import copy
    j = copy.deepcopy(j)

    def fill(d, key, name, value_of):
        if isinstance(d, dict) and d.get(key) is None:
            shape = shape_of(name)
            if shape is not None:
                v = value_of(shape)
                if v is not None:
                    d[key] = int(v)

    def per(n, axis=0):
        return lambda s: s[axis] // int(n) if len(s) > axis and s[axis] % int(n) == 0 else None

    def head_sizes(m, p, heads_from):
        fill(m, "heads", p + heads_from, lambda s: s[0])
        if m.get("heads"):
            fill(m, "dim", p + "q", per(m["heads"]))
            fill(m, "vdim", p + "o", per(m["heads"], 1))
        if m.get("dim"):
            fill(m, "kv_heads", p + "k", per(m["dim"]))

    fill(j, "vocab", "embed", lambda s: s[0])
    fill(j, "width", "embed", lambda s: s[1] if len(s) > 1 else None)
    for i, e in enumerate(j.get("layers") or []):
        if not isinstance(e, dict):
            continue
        m, p = e.get("mixer"), f"l{i}.mix."
        if isinstance(m, dict) and e.get("type") == "attention":
            head_sizes(m, p, "g")
        elif isinstance(m, dict) and e.get("type") == "parallel":
            a, r = m.get("left"), m.get("right")
            if isinstance(a, dict):
                head_sizes(a, p + "left.", "sink")
                fill(a, "conv", p + "left.q.conv", lambda s: s[1] if len(s) > 1 else None)
            if isinstance(r, dict):
                if r.get("heads") is None and isinstance(r.get("decay"), list):
                    r["heads"] = len(r["decay"])
                if r.get("heads"):
                    fill(r, "dim", p + "right.q", per(r["heads"]))
                    fill(r, "vdim", p + "right.v", per(r["heads"]))
        f = e.get("mlp")
        if isinstance(f, dict):
            if f.get("kind") == "dense":
                fill(f, "ff", f"l{i}.mlp.gate", lambda s: s[0])
            elif f.get("kind") == "moe":
                fill(f.get("expert"), "ff", f"l{i}.mlp.e0.up", lambda s: s[0])
                fill(f.get("router"), "experts", f"l{i}.mlp.router", lambda s: s[0])
    return j
