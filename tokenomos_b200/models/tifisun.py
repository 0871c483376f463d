"""The Tifisun decoder as a declaration: configuration -> ``ModelSpec``.

A decoder on a 32-bit residual stream with a norm before and after each sublayer:

- embedding: ``embed[token] * scale``;
- a layer: ``x <- x + m * n1b(mixer(n1(x)))``, then ``x <- x + m * n2b(ff(n2(x)))``; the norms' weights are stored around
  zero; a layer may use another layer's tensors with a cache and a state of its own (the layer list names that block
  again);
- mixer ``delta``: the gated delta rule with one decay per head and token, a SiLU output gate;
- mixer ``channel_delta``: the same with one decay per key channel from a low-rank projection, a sigmoid output gate
  from another one;
- mixer ``parallel``: sliding-window attention (norms over the whole query and key rows, a soft cap, a learned bias by
  distance) and lightning attention side by side, each brought to unit root mean square, averaged;
- feed-forward: gelu (tanh form) gated, every projection with a bias, or none;
- output: the model's norm, then the head.

Tensor names: ``embed``, ``final.norm``, ``head``, and per layer ``l<i>.``: ``norm1|norm1b|norm2|norm2b``; delta
``mix.q|k|v``, their ``.conv``, ``mix.b|A_log|dt_bias|norm|o`` with ``mix.a|g`` (delta) or ``mix.a1|a2|g1|g2`` (channel
delta); parallel ``mix.left.q|k|v|q.norm|k.norm|rel|o|out``, ``mix.right.q|k|v|g|norm|o|out``; ``mlp.gate|up|down`` and
their ``.b``.
"""

from __future__ import annotations

from tokenomos_b200.config.tifisun import TifisunConfig
from tokenomos_b200.parts.spec import (ROLE_EMBEDDING, ROLE_MATRIX, ROLE_NORM, ROLE_VECTOR, BlockSpec, FreeDim, LayerCall,
                                       ModelSpec, PartSpec, TensorDecl)

NORM_OFFSET = 1.0        # the stream's norm weights are stored around zero
BIAS_ROWS = 32           # rows of a bias table where no stored tensor says


class Tifisun:
    names = ("Tifisun",)
    config_class = TifisunConfig

    def declare(self, cfg: TifisunConfig, tensor_names=()) -> ModelSpec:
        d, eps = cfg.width, cfg.norm_eps

        def norm(name: str, mult: float = 1.0) -> PartSpec:
            return PartSpec("rmsnorm32", {"eps": eps, "offset": NORM_OFFSET, "mult": mult},
                            {"weight": TensorDecl(name, (d,), ROLE_VECTOR)})

        def delta(a: str, m, channel: bool) -> PartSpec:
            nk, nv = m.kv_heads * m.dim, m.heads * m.vdim
            tensors = {n: TensorDecl(a + n, (rows, d)) for n, rows in (("q", nk), ("k", nk), ("v", nv), ("b", m.heads))}
            tensors.update({f"{n}_conv": TensorDecl(f"{a}{n}.conv", (rows, m.taps), ROLE_VECTOR)
                            for n, rows in (("q", nk), ("k", nk), ("v", nv))})
            tensors["a_log"] = TensorDecl(a + "A_log", (m.heads,), ROLE_VECTOR)
            tensors["dt_bias"] = TensorDecl(a + "dt_bias", (m.heads * (m.dim if channel else 1),), ROLE_VECTOR)
            tensors["norm"] = TensorDecl(a + "norm", (m.vdim,), ROLE_NORM)
            tensors["o"] = TensorDecl(a + "o", (d, nv))
            if channel:
                for n, rows, rank in (("a", m.heads * m.dim, m.dim), ("g", nv, m.vdim)):
                    inner = FreeDim(f"{a}{n}.rank", rank)
                    tensors[n + "1"] = TensorDecl(f"{a}{n}1", (inner, d))
                    tensors[n + "2"] = TensorDecl(f"{a}{n}2", (rows, inner))
            else:
                tensors["a"] = TensorDecl(a + "a", (m.heads, d))
                tensors["g"] = TensorDecl(a + "g", (nv, d))
            return PartSpec("delta_rule", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "v_dim": m.vdim, "eps": eps,
                                           "decay": "channel" if channel else "head",
                                           "gate": "sigmoid" if channel else "silu"}, tensors)

        def pair(a: str, m) -> PartSpec:
            lt, rt = m.left, m.right
            left = {n: TensorDecl(f"{a}left.{n}", (rows, d)) for n, rows in (
                ("q", lt.heads * lt.dim), ("k", lt.kv_heads * lt.dim), ("v", lt.kv_heads * lt.vdim))}
            left["o"] = TensorDecl(a + "left.o", (d, lt.heads * lt.vdim))
            left["position.q_norm"] = TensorDecl(a + "left.q.norm", (lt.heads * lt.dim,), ROLE_NORM)
            left["position.k_norm"] = TensorDecl(a + "left.k.norm", (lt.kv_heads * lt.dim,), ROLE_NORM)
            left["rel"] = TensorDecl(a + "left.rel", (FreeDim(a + "left.rel.rows", BIAS_ROWS), lt.heads), ROLE_VECTOR)
            nk, nv = rt.heads * rt.dim, rt.heads * rt.vdim
            right = {n: TensorDecl(f"{a}right.{name}", (rows, d)) for n, name, rows in (
                ("q", "q", nk), ("k", "k", nk), ("v", "v", nv), ("gate", "g", nv))}
            right["norm"] = TensorDecl(a + "right.norm", (nv,), ROLE_NORM)
            right["o"] = TensorDecl(a + "right.o", (d, nv))
            tensors = {f"left.{k}": v for k, v in left.items()}
            tensors.update({f"right.{k}": v for k, v in right.items()})
            tensors["left_norm"] = TensorDecl(a + "left.out", (d,), ROLE_NORM)
            tensors["right_norm"] = TensorDecl(a + "right.out", (d,), ROLE_NORM)
            return PartSpec("mixer_pair", {
                "eps": eps,
                "left": {"kind": "attention", "params": {
                    "heads": lt.heads, "kv_heads": lt.kv_heads, "head_dim": lt.dim, "v_dim": lt.vdim, "scale": lt.scale,
                    "window": lt.window, "exact": True, "position": {"kind": "plain", "params": {"eps": eps}},
                    "shape": {"cap": lt.softcap, "bias_max": lt.bias_max}}},
                "right": {"kind": "lightning", "params": {"heads": rt.heads, "dim": rt.dim, "v_dim": rt.vdim, "eps": eps,
                                                          "decay": list(rt.decay)}},
            }, tensors)

        blocks, block_of, unused = [], {}, []
        for i, layer in enumerate(cfg.layers):
            if layer.weights != i:
                continue
            p = f"l{i}."
            ffn = None
            if layer.ff is not None:
                tensors = {}
                for n, shape in (("gate", (layer.ff, d)), ("up", (layer.ff, d)), ("down", (d, layer.ff))):
                    tensors[n] = TensorDecl(f"{p}mlp.{n}", shape)
                    tensors[n + "_bias"] = TensorDecl(f"{p}mlp.{n}.b", shape[:1], ROLE_VECTOR)
                ffn = PartSpec("glu_gelu", {}, tensors)
            else:
                # a folder may store the second norms of a layer without a feed-forward: nothing reads them
                unused += [(f"unused.{p}{n}", TensorDecl(p + n, (d,), ROLE_VECTOR, optional=True)) for n in ("norm2", "norm2b")]
            block_of[i] = len(blocks)
            blocks.append(BlockSpec("prenorm", {
                "mixer": pair(p + "mix.", layer.mixer) if layer.kind == "parallel"
                else delta(p + "mix.", layer.mixer, layer.kind == "channel_delta"),
                "ffn": ffn,
                "pre_mixer_norm": norm(p + "norm1"),
                "post_mixer_norm": norm(p + "norm1b", cfg.residual_mult),
                "pre_ffn_norm": norm(p + "norm2") if ffn is not None else None,
                "post_ffn_norm": norm(p + "norm2b", cfg.residual_mult) if ffn is not None else None,
            }))
        return ModelSpec(
            width=d,
            vocab=cfg.vocab,
            embedding=TensorDecl("embed", (cfg.vocab, d), ROLE_EMBEDDING),
            blocks=tuple(blocks),
            order=tuple(LayerCall(block_of[layer.weights]) for layer in cfg.layers),
            final_norm=norm("final.norm"),
            head=TensorDecl("head", (cfg.vocab, d), ROLE_MATRIX),
            embed_scale=cfg.embed_scale,
            embed_wide=True,
            extras=tuple(unused),
        )
