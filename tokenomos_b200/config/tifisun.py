"""Typed configuration of the Tifisun decoder, read from ``config.json``.

The file gives every size and every constant that differs between models of the design:

- ``vocab``, ``width``, ``norm.eps``, ``residual_mult``, ``embedding.scale`` (absent: 1);
- ``layers``: a list; each entry has ``type`` (``delta``, ``channel_delta`` or ``parallel``), ``mixer`` (the mixer's sizes
  and constants), ``mlp``: null or ``{"kind": "dense", "ff"}``, and optionally ``weights_of``: the layer whose tensors
  this one uses (with a cache and state of its own);
- mixer ``delta`` and ``channel_delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps); the inner widths of
  ``channel_delta``'s two low-rank projections are the stored tensors';
- mixer ``parallel``: ``left`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap`` (absent: none), ``bias_max``,
  ``mask.size`` (the sliding window; absent: every earlier position); the bias table's rows are the stored tensor's) and ``right`` (``heads``, ``dim``, ``vdim``, ``decay``,
  one per head).

``from_dict`` lists every fault it finds in one ``ConfigError``.
"""

from __future__ import annotations

from dataclasses import dataclass

from tokenomos_b200.config.lfm3 import ConfigError

MIXER_KINDS = ("delta", "channel_delta", "parallel")


@dataclass(frozen=True)
class DeltaParams:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class WindowedParams:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None
    bias_max: float
    window: int | None


@dataclass(frozen=True)
class LightningParams:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]


@dataclass(frozen=True)
class PairParams:
    left: WindowedParams
    right: LightningParams


@dataclass(frozen=True)
class LayerParams:
    kind: str
    mixer: DeltaParams | PairParams
    ff: int | None             # None: no feed-forward
    weights: int               # the layer whose tensors this one uses (its own index: its own)


@dataclass(frozen=True)
class TifisunConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    embed_scale: float
    layers: tuple[LayerParams, ...]

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: dict) -> "TifisunConfig":
        errors: list[str] = []

        def number(where: str, d, key: str, kind, positive: bool = True):
            if not isinstance(d, dict) or key not in d or d[key] is None:
                errors.append(f"{where}: missing key {key!r}")
                return None
            v = d[key]
            if isinstance(v, bool) or not isinstance(v, (int, float)) or (kind is int and int(v) != v):
                errors.append(f"{where}.{key} must be {'an integer' if kind is int else 'a number'}, got {v!r}")
                return None
            if positive and not v > 0:
                errors.append(f"{where}.{key} = {v!r} must be positive")
                return None
            return kind(v)

        def optional(where: str, d, key: str, kind, positive: bool = True):
            if not isinstance(d, dict) or d.get(key) is None:
                return None
            return number(where, d, key, kind, positive)

        def grouped(where: str, m):
            heads, kv_heads = number(where, m, "heads", int), number(where, m, "kv_heads", int)
            if None not in (heads, kv_heads) and heads % kv_heads:
                errors.append(f"{where}: {heads} heads over {kv_heads} key/value heads")
            return heads, kv_heads

        vocab = number("config", raw, "vocab", int)
        width = number("config", raw, "width", int)
        eps = number("norm", raw.get("norm"), "eps", float)
        mult = number("config", raw, "residual_mult", float, positive=False)
        scale = optional("embedding", raw.get("embedding"), "scale", float, positive=False)
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
                layers.append(LayerParams("invalid", None, None, i))
                continue
            w = f"{at}.mixer"
            if kind == "parallel":
                left, right = m.get("left"), m.get("right")
                heads, kv_heads = grouped(f"{w}.left", left)
                window = optional(f"{w}.left.mask", left.get("mask") if isinstance(left, dict) else None, "size", int)
                a = WindowedParams(heads, kv_heads, number(f"{w}.left", left, "dim", int), number(f"{w}.left", left, "vdim", int),
                                   number(f"{w}.left", left, "scale", float), optional(f"{w}.left", left, "softcap", float),
                                   number(f"{w}.left", left, "bias_max", float), window)
                rh = number(f"{w}.right", right, "heads", int)
                decay = right.get("decay") if isinstance(right, dict) else None
                if (not isinstance(decay, list) or (rh is not None and len(decay) != rh)
                        or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay)):
                    errors.append(f"{w}.right.decay = {decay!r}: one number per head ({rh})")
                    decay = []
                b = LightningParams(rh, number(f"{w}.right", right, "dim", int), number(f"{w}.right", right, "vdim", int),
                                    tuple(float(d) for d in decay))
                mixer = PairParams(a, b)
            else:
                heads, kv_heads = grouped(w, m)
                mixer = DeltaParams(heads, kv_heads, number(w, m, "dim", int), number(w, m, "vdim", int), number(w, m, "conv", int))
            ff = None
            f = entry.get("mlp")
            if f is not None:
                fk = f.get("kind") if isinstance(f, dict) else None
                if fk == "dense":
                    ff = number(f"{at}.mlp", f, "ff", int)
                else:
                    errors.append(f"{at}.mlp.kind = {fk!r}: 'dense' or null")
            source = optional(at, entry, "weights_of", int, positive=False)
            layers.append(LayerParams(kind, mixer, ff, i if source is None else source))
        for i, layer in enumerate(layers):
            # a layer's tensors may be another's, whose may be another's again
            j, seen = layer.weights, {i}
            while 0 <= j < len(layers) and layers[j].weights != j and j not in seen:
                seen.add(j)
                j = layers[j].weights
            if not 0 <= j < len(layers) or layers[j].weights != j:
                errors.append(f"layers[{i}].weights_of = {layer.weights}: no layer with tensors of its own")
            elif j != i and (layer.kind, layer.mixer, layer.ff) != (layers[j].kind, layers[j].mixer, layers[j].ff):
                errors.append(f"layers[{i}].weights_of = {layer.weights}: the two layers' entries differ")
            else:
                layers[i] = LayerParams(layer.kind, layer.mixer, layer.ff, j)
        if errors:
            raise ConfigError("config.json: " + "; ".join(errors))
        return cls(str(raw.get("architecture") or "Tifisun"), vocab, width, eps, mult, 1.0 if scale is None else scale,
                   tuple(layers))
