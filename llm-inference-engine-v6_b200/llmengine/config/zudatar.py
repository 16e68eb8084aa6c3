"""Typed configuration of the Zudatar decoder, read from its config.json.

Keys: `architecture` ("Zudatar"), `vocab`, `width`, `norm.eps`, optional `embedding` {scale, bigram {buckets, mul_prev, mul_cur}},
optional `logit_scale`, `layers` (a list; each entry has `type`: "channel_delta", "attention" or "latent_attention", `mixer` with
that mixer's sizes and constants, and `mlp`: null or `{kind: dense, ff}`), optional `max_positions` (the design has no position
limit; the engine needs one for its rotation tables) and optional `eos_token_ids`.

channel_delta mixer: heads, kv_heads, dim, vdim, conv (taps). The ranks of its two low-rank maps are no keys of the file: they are
the first dimensions of `l<i>.mix.a1` and `l<i>.mix.g1`, read from the checkpoint's header when a model folder is opened
(`decay_rank` and `gate_rank`, which the random-weights mode writes into its config.json, take precedence).
attention mixer: heads, kv_heads, dim, vdim (equal to dim: the values are the keys), scale, optional mask {size}, optional rot
{dims, base}. latent_attention mixer: heads, dim, vdim, kv_rank, q_rank, scale, optional mask {size}, optional kv_from (the index of
an earlier latent_attention layer whose latents this layer reads).
A size that the file leaves out and a tensor's shape gives is read from the checkpoint's header too (`sizes_from_tensors`).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Dict, FrozenSet, Optional, Tuple, Union

from .files import ConfigError
from .vapelix import DEFAULT_MAX_POSITIONS, _need

DEFAULT_RANK = 16  # what the random-weights mode uses when a configuration names no rank


@dataclass(frozen=True)
class PairTable:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0        # mask.size; 0: every earlier position is seen
    rot_dims: int = 0      # 0: positions do not enter the scores
    rot_base: float = 10000.0


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: int = 0
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class DenseFF:
    ff: int


@dataclass(frozen=True)
class ZudatarLayer:
    type: str  # "channel_delta" | "attention" | "latent_attention"
    mixer: Union[DeltaMixer, AttentionMixer, LatentMixer]
    mlp: Optional[DenseFF]


def _window(m: Dict[str, Any], where: str) -> int:
    mask = m.get("mask")
    return int(_need(mask, "size", where + ".mask")) if mask else 0


@dataclass(frozen=True)
class ZudatarConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: Tuple[ZudatarLayer, ...]
    embed_scale: float = 1.0
    pairs: Optional[PairTable] = None
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
    def from_dict(cls, j: Dict[str, Any], generation: Optional[Dict[str, Any]] = None) -> "ZudatarConfig":
        width, vocab = int(_need(j, "width", "config.json")), int(_need(j, "vocab", "config.json"))
        eps = float(_need(_need(j, "norm", "config.json"), "eps", "norm"))
        raw_layers = _need(j, "layers", "config.json")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind, m, w = _need(e, "type", where), _need(e, "mixer", where), where + ".mixer"
            if kind == "channel_delta":
                mixer: Union[DeltaMixer, AttentionMixer, LatentMixer] = DeltaMixer(
                    heads=int(_need(m, "heads", w)), kv_heads=int(_need(m, "kv_heads", w)), dim=int(_need(m, "dim", w)),
                    vdim=int(_need(m, "vdim", w)), taps=int(_need(m, "conv", w)), decay_rank=int(m.get("decay_rank") or DEFAULT_RANK),
                    gate_rank=int(m.get("gate_rank") or DEFAULT_RANK))
            elif kind == "attention":
                rot, dim = m.get("rot"), int(_need(m, "dim", w))
                mixer = AttentionMixer(heads=int(_need(m, "heads", w)), kv_heads=int(_need(m, "kv_heads", w)), dim=dim,
                                       vdim=int(m.get("vdim") or dim), scale=float(_need(m, "scale", w)), window=_window(m, w),
                                       rot_dims=int(_need(rot, "dims", w + ".rot")) if rot else 0,
                                       rot_base=float(_need(rot, "base", w + ".rot")) if rot else 10000.0)
            elif kind == "latent_attention":
                src = m.get("kv_from")
                mixer = LatentMixer(heads=int(_need(m, "heads", w)), dim=int(_need(m, "dim", w)), vdim=int(_need(m, "vdim", w)),
                                    kv_rank=int(_need(m, "kv_rank", w)), q_rank=int(_need(m, "q_rank", w)), scale=float(_need(m, "scale", w)),
                                    window=_window(m, w), kv_from=None if src is None else int(src))
            else:
                raise ConfigError(f"config.json: {where}: unknown layer type '{kind}' (channel_delta, attention, latent_attention)")
            f, mlp = e.get("mlp"), None
            if f:
                fk = _need(f, "kind", where + ".mlp")
                if fk != "dense":
                    raise ConfigError(f"config.json: {where}.mlp: unknown kind '{fk}' (dense)")
                mlp = DenseFF(int(_need(f, "ff", where + ".mlp")))
            layers.append(ZudatarLayer(kind, mixer, mlp))
        emb = j.get("embedding") or {}
        b, pairs = emb.get("bigram"), None
        if b:
            w = "embedding.bigram"
            pairs = PairTable(int(_need(b, "buckets", w)), int(_need(b, "mul_prev", w)), int(_need(b, "mul_cur", w)))
        scale, logit_scale = emb.get("scale"), j.get("logit_scale")
        cfg = cls(architecture=j.get("architecture", "Zudatar"), vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                  embed_scale=1.0 if scale is None else float(scale), pairs=pairs, logit_scale=1.0 if logit_scale is None else float(logit_scale),
                  max_positions=int(j.get("max_positions") or DEFAULT_MAX_POSITIONS),
                  eos_token_ids=frozenset(int(t) for t in j.get("eos_token_ids") or []))
        cfg.check()
        return cfg

    def check(self) -> None:
        if self.width <= 0 or self.vocab <= 0 or self.eps < 0 or self.max_positions <= 0:
            raise ConfigError("config.json: width, vocab and max_positions must be positive, eps not negative")
        b = self.pairs
        if b is not None and (b.buckets < 1 or not 0 <= b.mul_prev < 2 ** 31 or not 0 <= b.mul_cur < 2 ** 31):
            raise ConfigError("config.json: embedding.bigram: buckets must be positive, the multipliers lie in 0 .. 2^31 - 1")
        for i, l in enumerate(self.layers):
            m, where = l.mixer, f"config.json: layers[{i}]"
            if l.type == "channel_delta":
                if min(m.heads, m.kv_heads, m.dim, m.vdim, m.taps, m.decay_rank, m.gate_rank) <= 0 or m.heads % m.kv_heads:
                    raise ConfigError(f"{where}.mixer: sizes must be positive and heads a multiple of kv_heads")
            elif l.type == "attention":
                if min(m.heads, m.kv_heads, m.dim) <= 0 or m.heads % m.kv_heads or m.window < 0:
                    raise ConfigError(f"{where}.mixer: sizes must be positive and heads a multiple of kv_heads")
                if m.vdim != m.dim:
                    raise ConfigError(f"{where}.mixer: the values are the keys, so vdim ({m.vdim}) is dim ({m.dim})")
                if m.rot_dims < 0 or m.rot_dims % 2 or m.rot_dims > m.dim or not m.rot_base > 0:
                    raise ConfigError(f"{where}.mixer.rot: dims must be even and at most dim, base positive")
            else:
                if min(m.heads, m.dim, m.vdim, m.kv_rank, m.q_rank) <= 0 or m.window < 0:
                    raise ConfigError(f"{where}.mixer: sizes must be positive")
                if m.kv_from is not None:
                    if not 0 <= m.kv_from < i or self.layers[m.kv_from].type != "latent_attention":
                        raise ConfigError(f"{where}.mixer.kv_from: {m.kv_from} is no earlier latent_attention layer")
                    o = self.layers[m.kv_from].mixer
                    if o.kv_from is not None:
                        raise ConfigError(f"{where}.mixer.kv_from: layer {m.kv_from} has no latents of its own")
                    if o.kv_rank != m.kv_rank:
                        raise ConfigError(f"{where}.mixer.kv_from: layer {m.kv_from}'s kv_rank ({o.kv_rank}) is not this layer's ({m.kv_rank})")
            if l.mlp is not None and l.mlp.ff <= 0:
                raise ConfigError(f"{where}.mlp: ff must be positive")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for l in self.layers:
            m = l.mixer
            if l.type == "channel_delta":
                mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps,
                                         "decay_rank": m.decay_rank, "gate_rank": m.gate_rank}
            elif l.type == "attention":
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
                if m.rot_dims:
                    mixer["rot"] = {"dims": m.rot_dims, "base": m.rot_base}
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            if l.type != "channel_delta" and m.window:
                mixer["mask"] = {"size": m.window}
            layers.append({"type": l.type, "mixer": mixer, "mlp": None if l.mlp is None else {"kind": "dense", "ff": l.mlp.ff}})
        emb: Dict[str, Any] = {"scale": self.embed_scale}
        if self.pairs is not None:
            emb["bigram"] = {"buckets": self.pairs.buckets, "mul_prev": self.pairs.mul_prev, "mul_cur": self.pairs.mul_cur}
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                               "embedding": emb, "logit_scale": self.logit_scale, "layers": layers, "max_positions": self.max_positions}
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

    fill(j, "vocab", "embed", lambda s: s[0])
    fill(j, "width", "embed", lambda s: s[1] if len(s) > 1 else None)
    fill((j.get("embedding") or {}).get("bigram"), "buckets", "bigram", lambda s: s[0] - 1)
    for i, e in enumerate(j.get("layers") or []):
        if not isinstance(e, dict):
            continue
        m, p = e.get("mixer"), f"l{i}.mix."
        if isinstance(m, dict):
            if e.get("type") == "channel_delta":
                fill(m, "decay_rank", p + "a1", lambda s: s[0])
                fill(m, "gate_rank", p + "g1", lambda s: s[0])
                fill(m, "conv", p + "q.conv", lambda s: s[1] if len(s) > 1 else None)
                fill(m, "heads", p + "A_log", lambda s: s[0])
                fill(m, "vdim", p + "norm", lambda s: s[0])
                if m.get("heads"):
                    fill(m, "dim", p + "dt_bias", per(m["heads"]))
                if m.get("dim"):
                    fill(m, "kv_heads", p + "k", per(m["dim"]))
            elif e.get("type") == "attention":
                fill(m, "heads", p + "g", lambda s: s[0])
                if m.get("heads"):
                    fill(m, "dim", p + "q", per(m["heads"]))
                    fill(m, "vdim", p + "o", per(m["heads"], 1))
                if m.get("dim"):
                    fill(m, "kv_heads", p + "k", per(m["dim"]))
            elif e.get("type") == "latent_attention":
                fill(m, "heads", p + "g", lambda s: s[0])
                fill(m, "q_rank", p + "dq", lambda s: s[0])
                fill(m, "kv_rank", p + "uk", lambda s: s[1] if len(s) > 1 else None)
                if m.get("heads"):
                    fill(m, "dim", p + "uk", per(m["heads"]))
                    fill(m, "vdim", p + "uv", per(m["heads"]))
        fill(e.get("mlp"), "ff", f"l{i}.mlp.gate", lambda s: s[0])
    return j
