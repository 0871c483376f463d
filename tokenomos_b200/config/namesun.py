"""Typed configuration of the Namesun decoder, read from ``config.json``.

The file gives every size and every constant that differs between models of the design:

- ``vocab``, ``width``, ``norm.eps``, ``residual_mult``;
- ``layers``: a list; each entry has ``type`` (``attention`` or ``retention``), ``mixer`` (the mixer's sizes and constants) and
  ``mlp``: null, ``{"kind": "dense", "ff"}`` or ``{"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top",
  "groups": {"count", "keep"}}, "shared": {"ff", "limit"}}`` (``groups`` absent: one group; ``shared`` absent: no shared
  expert);
- mixer ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (the chunk; absent: every earlier
  position), ``v_mix`` (absent: false);
- mixer ``retention``: ``heads``, ``dim``, ``vdim``, ``decay`` (one per head), ``rot`` (``dims``, ``base``; absent: no rotation).

``from_dict`` lists every fault it finds in one ``ConfigError``.
"""

from __future__ import annotations

from dataclasses import dataclass

from tokenomos_b200.config.lfm3 import ConfigError

MIXER_KINDS = ("attention", "retention")


@dataclass(frozen=True)
class ChunkedParams:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None
    v_mix: bool


@dataclass(frozen=True)
class RotParams:
    dims: int
    base: float


@dataclass(frozen=True)
class RetentionParams:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: RotParams | None


@dataclass(frozen=True)
class DenseParams:
    ff: int


@dataclass(frozen=True)
class ExpertsParams:
    experts: int
    top: int
    groups: tuple[int, int] | None      # (count, keep)
    ff: int
    limit: float
    shared_ff: int | None
    shared_limit: float | None


@dataclass(frozen=True)
class LayerParams:
    kind: str
    mixer: ChunkedParams | RetentionParams
    mlp: DenseParams | ExpertsParams | None


@dataclass(frozen=True)
class NamesunConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: tuple[LayerParams, ...]

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def value_source(self) -> int | None:
        """The first layer that mixes values: the one the later ones mix in."""
        return next((i for i, layer in enumerate(self.layers) if layer.kind == "attention" and layer.mixer.v_mix), None)

    @classmethod
    def from_dict(cls, raw: dict) -> "NamesunConfig":
        errors: list[str] = []

        def number(where: str, d, key: str, kind, positive: bool = True, default=None):
            if not isinstance(d, dict) or key not in d or d[key] is None:
                if default is None:
                    errors.append(f"{where}: missing key {key!r}")
                return default
            v = d[key]
            if isinstance(v, bool) or not isinstance(v, (int, float)) or (kind is int and int(v) != v):
                errors.append(f"{where}.{key} must be {'an integer' if kind is int else 'a number'}, got {v!r}")
                return None
            if positive and not v > 0:
                errors.append(f"{where}.{key} = {v!r} must be positive")
                return None
            return kind(v)

        def attention(w: str, m: dict) -> ChunkedParams:
            heads, kv_heads = number(w, m, "heads", int), number(w, m, "kv_heads", int)
            if None not in (heads, kv_heads) and heads % kv_heads:
                errors.append(f"{w}: {heads} heads over {kv_heads} key/value heads")
            mask = m.get("mask")
            v_mix = m.get("v_mix", False)
            if v_mix is not None and not isinstance(v_mix, bool):
                errors.append(f"{w}.v_mix = {v_mix!r}: true or false")
            return ChunkedParams(heads, kv_heads, number(w, m, "dim", int), number(w, m, "vdim", int),
                                 number(w, m, "scale", float, positive=False),
                                 number(f"{w}.mask", mask, "size", int) if mask is not None else None, bool(v_mix))

        def retention(w: str, m: dict) -> RetentionParams:
            heads, dim = number(w, m, "heads", int), number(w, m, "dim", int)
            decay = m.get("decay")
            if (not isinstance(decay, list) or (heads is not None and len(decay) != heads)
                    or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay)):
                errors.append(f"{w}.decay = {decay!r}: one number per head ({heads})")
                decay = []
            rot = None
            if m.get("rot") is not None:
                dims = number(f"{w}.rot", m["rot"], "dims", int, positive=False)
                rot = RotParams(dims, number(f"{w}.rot", m["rot"], "base", float))
                if None not in (dims, dim) and (dims % 2 or not 0 <= dims <= dim):
                    errors.append(f"{w}.rot.dims = {dims}: an even number of the head's {dim} columns")
            return RetentionParams(heads, dim, number(w, m, "vdim", int), tuple(float(d) for d in decay), rot)

        def experts(w: str, f: dict) -> ExpertsParams:
            r, e, s = f.get("router"), f.get("expert"), f.get("shared")
            n, top = number(f"{w}.router", r, "experts", int), number(f"{w}.router", r, "top", int)
            groups = None
            if isinstance(r, dict) and r.get("groups") is not None:
                groups = (number(f"{w}.router.groups", r["groups"], "count", int),
                          number(f"{w}.router.groups", r["groups"], "keep", int))
            if None not in (n, top) and None not in (groups or (1, 1)):
                count, keep = groups or (1, 1)
                if n % count or keep > count or keep * (n // count) < top:
                    errors.append(f"{w}.router: {top} experts out of {keep} of {count} groups of {n}")
            return ExpertsParams(n, top, groups, number(f"{w}.expert", e, "ff", int), number(f"{w}.expert", e, "limit", float),
                                 number(f"{w}.shared", s, "ff", int) if s is not None else None,
                                 number(f"{w}.shared", s, "limit", float) if s is not None else None)

        vocab = number("config", raw, "vocab", int)
        width = number("config", raw, "width", int)
        eps = number("norm", raw.get("norm"), "eps", float)
        mult = number("config", raw, "residual_mult", float, positive=False, default=1.0)
        layers: list[LayerParams] = []
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            errors.append("'layers' must be a non-empty list")
            entries = []
        for i, entry in enumerate(entries):
            at = f"layers[{i}]"
            kind = entry.get("type") if isinstance(entry, dict) else None
            m = entry.get("mixer") if isinstance(entry, dict) else None
            if kind not in MIXER_KINDS or not isinstance(m, dict):
                errors.append(f"{at}.type = {kind!r}: known mixers are {list(MIXER_KINDS)}" if kind not in MIXER_KINDS
                              else f"{at}: missing 'mixer'")
                continue
            mixer = attention(f"{at}.mixer", m) if kind == "attention" else retention(f"{at}.mixer", m)
            mlp, f = None, entry.get("mlp")
            if f is not None:
                fk = f.get("kind") if isinstance(f, dict) else None
                if fk == "dense":
                    mlp = DenseParams(number(f"{at}.mlp", f, "ff", int))
                elif fk == "moe":
                    mlp = experts(f"{at}.mlp", f)
                else:
                    errors.append(f"{at}.mlp.kind = {fk!r}: 'dense', 'moe' or null")
            layers.append(LayerParams(kind, mixer, mlp))
        mixing = [layer.mixer for layer in layers if layer.kind == "attention" and layer.mixer.v_mix]
        if len({(m.kv_heads, m.vdim) for m in mixing}) > 1:
            errors.append("layers that mix values have the same kv_heads and vdim")
        if errors:
            raise ConfigError("config.json: " + "; ".join(errors))
        return cls(str(raw.get("architecture") or "Namesun"), vocab, width, eps, mult, tuple(layers))
