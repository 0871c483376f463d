"""The Namesun decoder as a declaration: configuration -> ``ModelSpec``.

A decoder on a 32-bit residual stream with norms behind its sublayers only:

- embedding: ``embed[token]``;
- a layer: ``x <- x + m * ls1 * n1(mixer(x))``, then ``x <- x + m * ls2 * n2(ff(x))``: the sublayers read the stream itself, and
  what they give is RMS-normed and scaled column by column;
- mixer ``attention``: grouped-query attention without a rotation over the query's own chunk of positions, heads of q and k
  brought to unit root mean square, one added to the softmax's denominator, values mixed with those of the first layer that
  mixes;
- mixer ``retention``: linear attention with a fixed decay per head, rotated q and k, a norm per head and a SiLU gate;
- feed-forward: SwiGLU; or a mixture of experts with clamped gates, chosen by softmax scores plus a correction among the best
  groups of experts and weighed by the scores, plus a shared expert; or none;
- output: the model's norm, then the head.

Tensor names: ``embed``, ``final.norm``, ``head``, and per layer ``l<i>.``: ``norm1|norm2|ls1|ls2``; attention ``mix.q|k|v|o|vmix``;
retention ``mix.q|k|v|g|o``; ``mlp.gate|up|down`` or ``mlp.router|correction``, ``mlp.e<k>.gate|up|down``,
``mlp.shared.gate|up|down``.
"""

from __future__ import annotations

from tokenomos_b200.config.namesun import DenseParams, NamesunConfig
from tokenomos_b200.parts.spec import (ROLE_EMBEDDING, ROLE_MATRIX, ROLE_NORM, ROLE_VECTOR, BlockSpec, LayerCall, ModelSpec,
                                       PartSpec, TensorDecl)

# constants the design fixes
GLU_ALPHA = 1.702        # the sigmoid's slope in an expert's activation
GLU_SHIFT = 1.0          # added to an expert's clamped up branch


class Namesun:
    names = ("Namesun",)
    config_class = NamesunConfig

    def declare(self, cfg: NamesunConfig, tensor_names=()) -> ModelSpec:
        d, eps = cfg.width, cfg.norm_eps
        source = cfg.value_source()

        def behind(p: str, q: int) -> PartSpec:
            return PartSpec("rmsnorm32", {"eps": eps, "mult": cfg.residual_mult}, {
                "weight": TensorDecl(f"{p}norm{q}", (d,), ROLE_NORM), "layer_scale": TensorDecl(f"{p}ls{q}", (d,), ROLE_NORM)})

        def gated(prefix: str, role: str, ff: int) -> dict:
            return {f"{role}gate": TensorDecl(prefix + "gate", (ff, d)), f"{role}up": TensorDecl(prefix + "up", (ff, d)),
                    f"{role}down": TensorDecl(prefix + "down", (d, ff))}

        blocks, unused = [], []
        for i, layer in enumerate(cfg.layers):
            m, p = layer.mixer, f"l{i}."
            a = p + "mix."
            if layer.kind == "attention":
                tensors = {"q": TensorDecl(a + "q", (m.heads * m.dim, d)), "k": TensorDecl(a + "k", (m.kv_heads * m.dim, d)),
                           "v": TensorDecl(a + "v", (m.kv_heads * m.vdim, d)), "o": TensorDecl(a + "o", (d, m.heads * m.vdim))}
                mixes = m.v_mix and i != source
                if mixes:
                    tensors["v_mix"] = TensorDecl(a + "vmix", (), ROLE_VECTOR)
                else:            # a folder may store it all the same: nothing reads it
                    unused.append((f"unused.{a}vmix", TensorDecl(a + "vmix", (), ROLE_VECTOR, optional=True)))
                mixer = PartSpec("attention", {
                    "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim, "scale": m.scale,
                    "chunk": m.chunk, "sink": True, "exact": True,
                    "value_mix": {"source": source if mixes else None} if m.v_mix else None,
                    "position": {"kind": "plain", "params": {"head_norm": True, "eps": eps}},
                }, tensors)
            else:
                nk, nv = m.heads * m.dim, m.heads * m.vdim
                mixer = PartSpec("retention", {
                    "heads": m.heads, "dim": m.dim, "v_dim": m.vdim, "decay": list(m.decay), "eps": eps,
                    "rot": {"dims": m.rot.dims, "base": m.rot.base} if m.rot is not None else None,
                }, {"q": TensorDecl(a + "q", (nk, d)), "k": TensorDecl(a + "k", (nk, d)), "v": TensorDecl(a + "v", (nv, d)),
                    "gate": TensorDecl(a + "g", (nv, d)), "o": TensorDecl(a + "o", (d, nv))})
            f, ffn = layer.mlp, None
            if isinstance(f, DenseParams):
                ffn = PartSpec("swiglu", {}, gated(p + "mlp.", "", f.ff))
            elif f is not None:
                tensors = {"router": TensorDecl(p + "mlp.router", (f.experts, d), ROLE_VECTOR),
                           "correction": TensorDecl(p + "mlp.correction", (f.experts,), ROLE_VECTOR)}
                for k in range(f.experts):
                    tensors.update(gated(f"{p}mlp.e{k}.", f"e{k}.", f.ff))
                if f.shared_ff:
                    tensors.update(gated(p + "mlp.shared.", "shared.", f.shared_ff))
                ffn = PartSpec("clamped_moe", {
                    "experts": f.experts, "top": f.top, "groups": f.groups, "renorm": False, "limit": f.limit,
                    "shared_limit": f.shared_limit, "alpha": GLU_ALPHA, "shift": GLU_SHIFT}, tensors)
            else:
                # a folder may store the second norm and scale of a layer without a feed-forward: nothing reads them
                unused += [(f"unused.{p}{n}", TensorDecl(p + n, (d,), ROLE_VECTOR, optional=True)) for n in ("norm2", "ls2")]
            blocks.append(BlockSpec("prenorm", {
                "mixer": mixer,
                "ffn": ffn,
                "pre_mixer_norm": PartSpec("stream32"),
                "post_mixer_norm": behind(p, 1),
                "pre_ffn_norm": PartSpec("stream32") if ffn is not None else None,
                "post_ffn_norm": behind(p, 2) if ffn is not None else None,
            }))
        return ModelSpec(
            width=d,
            vocab=cfg.vocab,
            embedding=TensorDecl("embed", (cfg.vocab, d), ROLE_EMBEDDING),
            blocks=tuple(blocks),
            order=tuple(LayerCall(i) for i in range(len(blocks))),
            final_norm=PartSpec("rmsnorm32", {"eps": eps}, {"weight": TensorDecl("final.norm", (d,), ROLE_NORM)}),
            head=TensorDecl("head", (cfg.vocab, d), ROLE_MATRIX),
            embed_wide=True,
            extras=tuple(unused),
        )
