"""The Namesun decoder against its plain implementation (``plain_namesun``): every mechanism alone (the norm and scale behind a
sublayer with rows of the stream for the next one, attention in chunks with a sink over unit heads, values mixed with
another layer's, retention, routing by corrected scores among groups, clamped experts with a shared one), the whole model
replayed four ways in 32-bit and in bfloat16 on poisoned pools, keys made loud at page borders and on both sides of a chunk's
edge, states carried over portions down to two tokens, long decoding, generation through the entry points. The
configurations are made for the tests: other layer orders, one head, chunks of one and longer than any request, partial
and no rotation, one group, all experts, layers without a feed-forward, layers that do not mix values, sizes no 16-byte
kernel takes and sizes the tensor-core kernels take."""

from __future__ import annotations

import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_namesun as plain
import trace_util
from part_rig import PLANS, Rig, close, cuts_of, rows_for, write_folder

ROOT = Path(__file__).resolve().parents[1]


def attention(heads, kv_heads, dim, vdim, scale, chunk, v_mix=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": chunk}, "v_mix": v_mix}}


def retention(dim, vdim, decay, rot_dims, base=10000.0):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay}
    if rot_dims is not None:
        m["rot"] = {"dims": rot_dims, "base": base}
    return {"type": "retention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": r}
    if shared is not None:
        f["shared"] = {"ff": shared[0], "limit": shared[1]}
    return f


def model(vocab, width, layers, eps=1e-5, mult=0.5):
    return {"architecture": "Namesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": layers}


# A: retention first, the first layer that mixes values behind one that does not, chunks of 11 and 6 over pages of 4 (two cache
#    groups), part of the head rotated, a layer without a feed-forward in the middle and one at the end
NS_A = model(300, 48, [dict(retention(12, 20, [0.5, 0.9, 0.995], 6), mlp=moe(6, 2, 24, 1.5, (3, 2), (16, 0.7))),
                       dict(attention(4, 2, 12, 20, 0.4, 11, False), mlp=dense(40)),
                       dict(attention(2, 1, 16, 24, 0.3, 6), mlp=None),
                       dict(retention(8, 8, [0.97], 8, 100.0), mlp=dense(64)),
                       dict(attention(3, 1, 8, 24, 0.5, 11), mlp=moe(8, 3, 16, 3.0, (4, 2), (40, 2.0))),
                       dict(attention(4, 1, 12, 24, 0.6, 6), mlp=None)], mult=0.7)
# B: one head everywhere, chunks of one, one expert a token, no groups, no rotation, a factor of 1
NS_B = model(200, 64, [dict(attention(1, 1, 16, 40, 0.25, 1), mlp=moe(3, 1, 96, 2.5, None, (8, 1.0))),
                       dict(retention(16, 16, [0.9], None), mlp=None),
                       dict(attention(1, 1, 24, 40, 0.2, 7), mlp=dense(24))], eps=1e-6, mult=1.0)
# C: sizes no 16-byte kernel takes, a chunk longer than any request, a head that never forgets and one that remembers nothing, as
#    many experts as a token takes, no shared expert
NS_C = model(50, 36, [dict(attention(3, 3, 7, 10, 0.5, 500), mlp=moe(5, 5, 21, 2.0, (5, 5))),
                      dict(retention(9, 5, [1.0, 0.0], 2), mlp=dense(9)),
                      dict(attention(6, 3, 5, 10, 0.9, 13), mlp=moe(9, 2, 11, 0.5, (3, 1), (7, 4.0))),
                      dict(retention(5, 7, [0.25, 0.8, 0.99], 4, 5.0), mlp=None)], mult=-0.3)
# D: sizes the tensor-core kernels take in bfloat16 (keys and values of one size and of two), longer requests, chunks of 100 and
#    64 over pages of 16, a scale too large for a softmax without a running maximum
NS_D = model(400, 128, [dict(attention(8, 2, 64, 64, 0.15, 100), mlp=dense(256)),
                        dict(retention(64, 32, [0.9, 0.98, 0.999, 0.6], 64, 1e5), mlp=moe(16, 4, 64, 2.0, (4, 2), (128, 1.5))),
                        dict(attention(4, 2, 24, 64, 0.2, 64), mlp=moe(8, 2, 128, 1.0, None, (64, 3.0))),
                        dict(attention(4, 2, 128, 64, 0.6, 100), mlp=None),
                        dict(retention(32, 64, [0.95, 0.99], 16), mlp=dense(128))])

CASES = {
    "A": dict(config=NS_A, seed=61, page=4, lengths=[1, 2, 7, 30, 61, 45]),
    "B": dict(config=NS_B, seed=62, page=8, lengths=[3, 19, 21, 50, 90, 33]),
    "C": dict(config=NS_C, seed=63, page=4, lengths=[1, 6, 23, 40, 5]),
    "D": dict(config=NS_D, seed=64, page=16, lengths=[2, 31, 150, 65, 300, 90]),
}
# Bounds relative to a request's largest |logit|. The 32-bit model computes what the plain implementation computes, in another
# order; bfloat16 rounds every product's inputs and outputs.
TOL_F32, TOL_F32_SAME, TOL_BF16 = 4e-5, 3e-5, 0.12
CLOSE_CALLS = 0.2         # of a request's positions, in bfloat16 only (see ``compare``)


def make_tensors(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random weights, rounded to bfloat16: norm weights and scales far from one, routers loud enough to tell experts apart,
    corrections of the size of the scores with both signs, a lambda that is neither 0 nor 1."""
    from tokenomos_b200 import models

    arch = models.architecture_of(config)
    spec = arch.declare(arch.config_class.from_dict(config))
    noise = torch.Generator().manual_seed(seed)
    out = {}
    for d in spec.tensor_decls():
        r, u = torch.randn(d.shape, generator=noise), torch.rand(d.shape, generator=noise)
        n = d.name
        if d.optional and not n.endswith("vmix"):
            continue
        if n.endswith(("norm1", "norm2", "ls1", "ls2", "final.norm")):
            t = 1.0 + 0.3 * r
        elif n.endswith("vmix"):
            t = 0.25 + 0.5 * u
        elif n.endswith("correction"):
            t = 0.5 * r
        elif n == "embed":
            t = r
        elif n.endswith("router"):
            t = r * (3.0 / math.sqrt(d.shape[-1]))
        elif n.endswith((".mlp.gate", ".mlp.up")) or (".mlp." in n and n.endswith(("gate", "up"))):
            t = r * (1.5 / math.sqrt(d.shape[-1]))       # (the clamps are met on both sides)
        else:
            t = r / math.sqrt(d.shape[-1])
        out[n] = t.to(torch.bfloat16)
    return out


def rig_for(layers, width, dtype, folder, seed=0, edit=None, **kw) -> Rig:
    config = model(16, width, layers)
    tensors = make_tensors(config, seed)
    if edit is not None:
        edit(tensors)
    return Rig(config, tensors, dtype, folder, **kw)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, case in CASES.items():
        folder = tmp_path_factory.mktemp(f"ns_{name}")
        tensors = make_tensors(case["config"], case["seed"])
        write_folder(folder, case["config"], tensors)
        out[name] = (folder, {k: v.double() for k, v in tensors.items()})
    return out


def requests_for(name: str) -> dict[str, list[int]]:
    g = torch.Generator().manual_seed(511 + ord(name))
    vocab = CASES[name]["config"]["vocab"]
    return {f"r{i}": torch.randint(0, vocab, (n,), generator=g).tolist() for i, n in enumerate(CASES[name]["lengths"])}


_ORACLE: dict = {}


def oracle(name: str, folders, reqs: dict) -> dict[str, torch.Tensor]:
    out = {}
    for rid, ids in reqs.items():
        key = (name, tuple(ids))
        if key not in _ORACLE:
            _ORACLE[key] = plain.forward(CASES[name]["config"], folders[name][1], ids)[0]
        out[rid] = _ORACLE[key]
    return out


def compare(got: dict, want: dict, tol: float, what: str, close_calls: float = 0.0, rare: float = 0.0):
    """``close_calls``: the share of a request's positions (at least one, if not zero) that may lie outside the bound. A 16-bit
    model's router sees inputs that differ from the plain implementation's by rounding; where two experts' scores are that
    close it takes the other one, and the position's logits move by a whole expert's output (and, through a state or a
    cache, so may later ones). The 32-bit model gets none. ``rare``: the share of positions that may be up to ten times the
    bound off: where the read of a state all but cancels, the norm behind it magnifies what rounding leaves."""
    for rid, ref in want.items():
        assert got[rid].shape == ref.shape, (what, rid, got[rid].shape, ref.shape)
        assert torch.isfinite(got[rid]).all(), (what, rid)
        err = (got[rid] - ref).abs().amax(dim=1)
        scale = ref.abs().max().item()
        bad = (err > tol * scale).nonzero()
        allowed = math.ceil(close_calls * len(err)) if close_calls else 0
        if rare and err.max() <= 10 * tol * scale:
            allowed = max(allowed, math.ceil(rare * len(err)))
        assert bad.numel() <= allowed, (f"{what}: request {rid}: {bad.numel()} wrong positions of {len(err)}, the first {int(bad[0])}: "
                                        f"error {err[int(bad[0])].item():.3e}, allowed {tol * scale:.3e}")


# ---------------------------------------------------------------------------------------------
# without a GPU: configuration, declaration, the oracle's own pieces
# ---------------------------------------------------------------------------------------------

def test_configuration_reads_every_size_and_lists_every_fault():
    from tokenomos_b200.config import ConfigError, NamesunConfig

    cfg = NamesunConfig.from_dict(NS_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.residual_mult) == (300, 48, 1e-5, 0.7)
    assert [layer.kind for layer in cfg.layers] == ["retention", "attention", "attention", "retention", "attention", "attention"]
    assert cfg.value_source() == 2
    r, a = cfg.layers[0].mixer, cfg.layers[4].mixer
    assert (r.heads, r.dim, r.vdim, r.decay, r.rot.dims, r.rot.base) == (3, 12, 20, (0.5, 0.9, 0.995), 6, 10000.0)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.v_mix) == (3, 1, 8, 24, 0.5, 11, True)
    f = cfg.layers[4].mlp
    assert (f.experts, f.top, f.groups, f.ff, f.limit, f.shared_ff, f.shared_limit) == (8, 3, (4, 2), 16, 3.0, 40, 2.0)
    assert cfg.layers[1].mlp.ff == 40 and cfg.layers[2].mlp is None
    cfg = NamesunConfig.from_dict(NS_B)
    assert cfg.layers[0].mlp.groups is None and cfg.layers[1].mixer.rot is None and cfg.value_source() == 0
    bare = json.loads(json.dumps(NS_B))
    for layer in (bare["layers"][0], bare["layers"][2]):
        del layer["mixer"]["mask"], layer["mixer"]["v_mix"]
    cfg = NamesunConfig.from_dict(bare)
    assert cfg.value_source() is None and cfg.layers[0].mixer.chunk is None
    bad = json.loads(json.dumps(NS_A))
    del bad["width"]
    bad["layers"][0]["mixer"]["decay"] = [0.5]                           # read as 3 heads
    bad["layers"][0]["mlp"]["router"]["groups"] = {"count": 4, "keep": 1}
    bad["layers"][1]["mixer"]["kv_heads"] = 3                            # 4 heads over 3
    bad["layers"][2]["type"] = "something"
    bad["layers"][3]["mixer"]["rot"]["dims"] = 9
    bad["layers"][4]["mixer"]["vdim"] = 25                               # mixes with values of 24
    bad["layers"][1]["mlp"]["kind"] = "odd"
    bad["layers"][5]["mixer"].pop("scale")
    with pytest.raises(ConfigError) as err:
        NamesunConfig.from_dict(bad)
    text = str(err.value)
    assert all(s in text for s in ("width", "decay", "1 of 4 groups", "4 heads over 3", "something", "rot.dims = 9",
                                   "mix values", "'odd'", "scale"))


def test_declaration_lists_the_tensors_the_order_and_the_state(folders):
    from tokenomos_b200 import models
    from tokenomos_b200.parts import build_model
    from tokenomos_b200.parts.contract import ChunkKV
    from tokenomos_b200.parts.registry import Runtime
    from tokenomos_b200.weights.checkpoint import Checkpoint, check, load_tensors

    arch = models.architecture_of(NS_A)
    spec = arch.declare(arch.config_class.from_dict(NS_A))
    names = {d.name: d for d in spec.tensor_decls()}
    assert names["head"].shape == (300, 48) and names["l0.mix.g"].shape == (60, 48) and names["l0.ls2"].shape == (48,)
    assert names["l4.mix.vmix"].shape == () and not names["l4.mix.vmix"].optional
    assert names["l2.mix.vmix"].optional and names["l1.mix.vmix"].optional          # where values come from; not mixed
    assert names["l4.mlp.correction"].shape == (8,) and names["l4.mlp.shared.down"].shape == (48, 40)
    assert names["l4.mlp.e7.up"].shape == (16, 48) and names["l2.norm2"].optional and names["l5.ls2"].optional
    folder, _ = folders["A"]
    ckpt = Checkpoint(folder)
    check(ckpt, spec.tensor_decls(), spec.scope)
    tensors = load_tensors(ckpt, spec.tensor_decls(), torch.float32, "cpu")
    stack = build_model(spec, tensors, Runtime(torch.float32, torch.device("cpu")))
    states = stack.state_specs()
    assert set(states) == {(0, "S"), (1, "kv"), (2, "kv"), (3, "S"), (4, "kv"), (5, "kv")}
    assert states[(1, "kv")] == ChunkKV(2, 20, 11) and states[(5, "kv")] == ChunkKV(1, 24, 6)
    assert states[(0, "S")].shape == (3, 20, 12) and states[(0, "S")].dtype == torch.float32
    assert stack.capture_safe
    mix = stack.blocks[5].mixer.value_mix
    assert mix.source == 2 and mix.lam == float(tensors["l5.mix.vmix"]) and stack.blocks[1].mixer.value_mix is None


def test_oracle_pieces():
    t = lambda *v: torch.tensor(v, dtype=torch.float64)
    # chunks of 3: position 3 starts anew
    assert plain.same_chunk(5, 3).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [1, 1, 1, 0, 0], [0, 0, 0, 1, 0], [0, 0, 0, 1, 1]]
    p = plain.sink_softmax(t([0.0, math.log(2.0), 50.0]), torch.tensor([[True, True, False]]))
    assert torch.allclose(p, t([0.25, 0.5, 0.0]))                 # 1 / (1 + 1 + 2), 2 / 4
    # the first two columns turn by position times one frequency each with the third and fourth; the fifth stays
    x = torch.ones(3, 1, 5, dtype=torch.float64)
    y = plain.rotate(x, {"dims": 4, "base": 100.0})
    a, b = 2.0, 0.2
    assert torch.allclose(y[2, 0], t(math.cos(a) - math.sin(a), math.cos(b) - math.sin(b), math.cos(a) + math.sin(a),
                                     math.cos(b) + math.sin(b), 1.0))
    # two tokens of retention by hand: the read follows the write
    o = plain.retention_scan(t([[1.0, 2.0]], [[1.0, 1.0]]), t([[3.0, 1.0]], [[0.0, 2.0]]), t([[5.0]], [[7.0]]), [0.5])
    assert o.flatten().tolist() == [25.0, 0.5 * 15 + 0.5 * 5 + 14]
    # a correction chooses but does not weigh; a group is as good as its best expert; scores below zero beat what is left out
    z = t(0.0, 1.0, 2.0, 3.0, 0.5, 0.2)
    s = torch.softmax(z, -1)
    chosen, w = plain.route(z, t(0.0, 0.0, 0.0, -2.0, 0.0, 0.0), {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert chosen == [2, 3] and torch.equal(w, s[[2, 3]])
    chosen, _ = plain.route(z, t(-3.0, -3.0, -3.0, -3.0, -3.0, -1.0), {"experts": 6, "top": 2})
    assert chosen == [5, 3]
    # an expert at both clamps
    W = {"gate": t([10.0]), "up": t([-10.0]), "down": t([1.0])}
    g = 2.0 / (1 + math.exp(-1.702 * 2.0))
    assert abs(plain.expert(t([1.0]), W, "", 2.0).item() - g * (-2.0 + 1.0)) < 1e-12


# ---------------------------------------------------------------------------------------------
# each mechanism alone, on the GPU
# ---------------------------------------------------------------------------------------------

@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 30, 36, 512, 2048, 1027, 6144, 8200])
def test_scaled_norm_behind_a_sublayer_and_the_streams_rows(width, dtype):
    """``stream + m ls n(x)`` in 32-bit and its rows rounded for the next sublayer; the rows that start a stream; the last add
    with the model's norm behind it."""
    from tokenomos_b200.parts.norm import StreamNorm32, StreamRows32

    g = torch.Generator().manual_seed(width)
    T = 5
    stream = torch.randn(T, width, generator=g) * 3
    x = torch.randn(T, width, generator=g).to(dtype)
    w, ls, wf = (1 + 0.3 * torch.randn(width, generator=g) for _ in range(3))
    post = StreamNorm32(w.cuda(), 1e-3, store=dtype, mult=-0.4, layer_scale=ls.cuda())
    rows = StreamRows32(dtype)
    want = stream.double() - 0.4 * plain.rms(x.double(), 1e-3) * w.double() * ls.double()
    y, new = rows.add_norm(x.cuda(), stream.cuda(), post)
    assert new.dtype == torch.float32 and (new.double().cpu() - want).abs().max() <= 2e-6 * want.abs().max()
    assert y.dtype == dtype and torch.equal(y, new.to(dtype))
    y, start = rows.add_norm(stream.cuda(), None, None)
    assert torch.equal(start.cpu(), stream) and torch.equal(y.cpu(), stream.to(dtype))
    y, added = rows.add_norm(x.cuda(), stream.cuda(), None)
    assert torch.equal(added.cpu(), stream + x.float()) and torch.equal(y, added.to(dtype))
    final = StreamNorm32(wf.cuda(), 1e-5, store=dtype)
    y, _ = final.add_norm(x.cuda(), stream.cuda(), post)
    ref = plain.rms(want, 1e-5) * wf.double()
    assert (y.double().cpu() - ref).abs().max() <= (2e-6 if dtype == torch.float32 else 6e-3) * ref.abs().max()
    with pytest.raises(ValueError):
        post.add_norm(x.cuda(), None)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, D, V, row, shift", [(4, 2, 12, 20, 20, 0), (1, 1, 5, 3, 7, 1), (8, 2, 64, 64, 64, 8), (6, 3, 96, 40, 104, 16),
                                                    (3, 1, 250, 8, 256, 0), (40, 20, 16, 16, 16, 8), (2, 2, 256, 256, 256, 0), (16, 2, 8, 24, 24, 0)])
def test_unit_heads_mixed_values_and_the_cache_write(H, G, D, V, row, shift, dtype):
    """The kernel alone: heads of any size over 1 to 32 lanes, more heads than a pass takes, cache rows wider than either size,
    strided rows, pages out of order, with and without weights, with and without other values to mix in."""
    from tokenomos_b200 import ops

    g = torch.Generator().manual_seed(D + V)
    T, P = 7, 4
    n = H * D + G * (D + V)
    wide = torch.randn(T, n + shift + 8, generator=g).to(dtype)
    other = torch.randn(T, G * V + 8, generator=g).to(dtype)
    wq, wk = 1 + 0.3 * torch.randn(D, generator=g), 1 + 0.3 * torch.randn(D, generator=g)
    pos = torch.tensor([3, 4, 5, 6, 0, 1, 9], dtype=torch.int32)
    seq = torch.tensor([0, 0, 0, 0, 1, 1, 1], dtype=torch.int32)
    table = torch.tensor([[5, 2, 0], [3, 1, 6]], dtype=torch.int32)
    src = wide[:, shift:shift + n].double()
    q = plain.rms(src[:, :H * D].view(T, H, D), 1e-4)
    k = plain.rms(src[:, H * D:(H + G) * D].view(T, G, D), 1e-4)
    v = src[:, (H + G) * D:]
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    for weights in (False, True):
        for lam in (None, 0.3):
            pool = torch.full((8, 2, G, P, row), 7.0, dtype=dtype, device="cuda")
            got = ops.qkv_head_norm_write(
                wide.cuda()[:, shift:shift + n], wq.cuda() if weights else None, wk.cuda() if weights else None, 1e-4, pos.cuda(),
                seq.cuda(), table.cuda(), pool, H, G, D, V, other.cuda()[:, 8:] if lam else None, lam or 0.0).double().cpu()
            cached = pool.double().cpu()
            vv = v if lam is None else plain.mix_values(v, other[:, 8:].double(), lam)
            assert (got - q * (wq.double() if weights else 1)).abs().max() <= tol * 4
            for t in range(T):
                page = int(table[seq[t], pos[t] // P])
                slot = cached[page, :, :, int(pos[t]) % P]
                assert (slot[0, :, :D] - k[t] * (wk.double() if weights else 1)).abs().max() <= tol * 4
                assert (slot[1, :, :V] - vv[t].view(G, V)).abs().max() <= tol * 4
                assert (slot[0, :, D:] == 7.0).all() and (slot[1, :, V:] == 7.0).all()
            assert (cached[[0, 1, 4, 7]] == 7.0).all()           # pages of no token stay as they were
    alone = ops.qkv_head_norm_write(wide.cuda()[:, shift:shift + n], None, None, 1e-4, pos.cuda(), seq.cuda(), None, None, H, G, D, V)
    assert (alone.double().cpu() - q).abs().max() <= tol * 4


ATTENTION = [dict(heads=4, kv_heads=2, dim=12, vdim=20, chunk=11, scale=0.4), dict(heads=1, kv_heads=1, dim=6, vdim=40, chunk=1, scale=0.5),
             dict(heads=3, kv_heads=3, dim=24, vdim=8, chunk=500, scale=0.2), dict(heads=8, kv_heads=2, dim=64, vdim=64, chunk=70, scale=0.1),
             dict(heads=6, kv_heads=2, dim=128, vdim=64, chunk=33, scale=0.05), dict(heads=4, kv_heads=4, dim=48, vdim=96, chunk=65, scale=0.9),
             dict(heads=16, kv_heads=1, dim=104, vdim=128, chunk=64, scale=0.08), dict(heads=4, kv_heads=1, dim=128, vdim=128, chunk=47, scale=0.09),
             dict(heads=6, kv_heads=2, dim=64, vdim=64, chunk=128, scale=0.2), dict(heads=40, kv_heads=2, dim=16, vdim=32, chunk=9, scale=0.3)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "decoded", "portions", "tokens"])
@pytest.mark.parametrize("case", ATTENTION)
def test_chunked_attention_with_mixed_values_alone(case, how, dtype, tmp_path):
    """Two layers, the second one's values mixed with the first one's: values wider and narrower than the keys, one head, chunks
    of one and longer than any request, scales with and without a bounded softmax, sizes each of the tensor-core kernels takes
    and sizes none takes; requests side by side."""
    layer = dict(attention(**case), mlp=None)
    rig = rig_for([layer, layer], 32, dtype, tmp_path, seed=3, page=4, pages=140)
    first, second = (rig.model.blocks[i].mixer for i in (0, 1))
    lengths = {"a": 97, "b": 38, "c": 140}
    x = rows_for(lengths, 32, 5)
    want = {rid: torch.cat((plain.attention(x[rid], rig.w, "l0.mix.", layer["mixer"], 1e-5),
                            plain.attention(x[rid], rig.w, "l1.mix.", layer["mixer"], 1e-5, x[rid] @ rig.w["l0.mix.v"].T)), -1)
            for rid in x}
    # the mix shows
    assert (want["a"][:, 32:] - plain.attention(x["a"], rig.w, "l1.mix.", layer["mixer"], 1e-5)).abs().max() > 0.1 * want["a"].abs().max()
    got = rig.run(x, {rid: PLANS[how](n) for rid, n in lengths.items()},
                  lambda rows, ctx: torch.cat((first.forward(rows, ctx, 0), second.forward(rows, ctx, 1)), -1))
    close(got, want, 2e-5 if dtype == "float32" else 4e-2, f"attention {case} {how} {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("how", ["whole", "decoded", "portions"])
@pytest.mark.parametrize("chunk, T, dim, vdim, dtype", [
    (chunk, T, 16, 24, dtype) for chunk, T in ((9, 90), (9, 91), (64, 320), (64, 257), (150, 299), (400, 330))
    for dtype in ("float32", "bfloat16")] + [
    (chunk, T, dim, dim, "bfloat16") for chunk, T in ((64, 320), (150, 301), (400, 330)) for dim in (64, 128)])
def test_one_loud_key_at_page_borders_and_at_a_chunks_edge(chunk, T, dim, vdim, dtype, how, tmp_path):
    """One key that the last queries lean towards, everything else quiet: the query's own, around a page border, hundreds of
    positions back, the first of the last query's chunk and the last of the chunk before it. A key that is dropped, read
    from a wrong page or let in across the edge changes the output by its own size; the plain implementation with another
    chunk is the control. (T: the last query is its chunk's last, its first, or in between.)"""
    page, width = 8, 32
    layer = dict(attention(2, 1, dim, vdim, 16.0 / dim, chunk), mlp=None)

    def edit(t):
        # keys read the first half of the input's channels alone, and both query heads read the second half as the key head
        # reads the first: a query row [0 | l] scores high against a key row [l | 0] and against no other query row
        k = t["l0.mix.k"].clone()
        k[:, width // 2:] = 0
        t["l0.mix.k"] = k
        t["l0.mix.q"] = torch.cat((k.roll(width // 2, dims=1), k.roll(width // 2, dims=1)))

    rig = rig_for([layer], width, dtype, tmp_path, seed=9, page=page, pages=60, edit=edit)
    mixer = rig.model.blocks[0].mixer
    tol = 2e-5 if dtype == "float32" else 4e-2
    last = T - 1
    start = last // chunk * chunk
    places = {last, last - 1, start, start + 1, start - 1, start - 2, start - chunk}
    places |= {p for p in (0, 1, page - 1, page, 2 * page, T - 257) if p >= start}
    for loud in sorted(p for p in places if 0 <= p <= last):
        g = torch.Generator().manual_seed(loud)
        # (unit heads bring every key to one size: quiet keys point away from the lean instead)
        lean = torch.randn(width // 2, generator=g).to(torch.bfloat16).double()
        x = torch.randn(T, width, generator=g).to(torch.bfloat16).double()
        x[:, :width // 2] = (x[:, :width // 2] - 1.5 * lean).to(torch.bfloat16).double()
        x[loud, :width // 2] = 3.0 * lean
        x[T - 3:, width // 2:] = 3.0 * lean
        want = plain.attention(x, rig.w, "l0.mix.", layer["mixer"], 1e-5)
        if loud == start - 1 or (loud == start and last > start):
            # the control at the edge: chunks that begin one position earlier or later for the last query (by their size, where
            # that is one that divides the place it should begin at)
            seen = plain.same_chunk(T, chunk)
            seen[-1] = (torch.arange(T) >= (start - 1 if loud < start else start + 1))
            real, plain.same_chunk = plain.same_chunk, lambda *_: seen
            try:
                other = plain.attention(x, rig.w, "l0.mix.", layer["mixer"], 1e-5)
            finally:
                plain.same_chunk = real
            assert (want[-1] - other[-1]).abs().max() > 0.3 * max(want[-1].abs().max(), other[-1].abs().max()), loud
        got = rig.run({"x": x}, {"x": PLANS[how](T)}, lambda rows, ctx: mixer.forward(rows, ctx, 0))
        close(got, {"x": want}, tol, f"loud key at {loud}, chunks of {chunk}, {how}, {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("how", ["whole", "tokens"])
def test_a_chunks_first_queries_lean_on_the_sink(how, tmp_path):
    """The first query of a chunk sees one key (its own): its weight is e^s / (1 + e^s), far from the 1 that a softmax without the
    sink gives, in every chunk."""
    for dim, vdim, dtype in ((12, 8, "float32"), (12, 8, "bfloat16"), (64, 64, "bfloat16"), (128, 128, "bfloat16"), (48, 16, "bfloat16")):
        layer = dict(attention(2, 2, dim, vdim, 0.5 / dim, 8), mlp=None)
        rig = rig_for([layer], 32, dtype, tmp_path / f"{dim}{dtype}", seed=4, page=4, pages=40)
        x = rows_for({"a": 41}, 32, 6)
        want = plain.attention(x["a"], rig.w, "l0.mix.", layer["mixer"], 1e-5)
        real = plain.sink_softmax
        plain.sink_softmax = lambda s, seen: torch.softmax(s.masked_fill(~seen, -math.inf), -1)
        try:
            without = plain.attention(x["a"], rig.w, "l0.mix.", layer["mixer"], 1e-5)
        finally:
            plain.sink_softmax = real
        for t in range(0, 41, 8):
            assert (without[t] - want[t]).abs().max() > 0.3 * want[t].abs().max()
        got = rig.run(x, {"a": PLANS[how](41)}, lambda rows, ctx: rig.model.blocks[0].mixer.forward(rows, ctx, 0))
        close(got, {"a": want}, 2e-5 if dtype == "float32" else 4e-2, f"sink {dim} {dtype} {how}")


RETENTION = [dict(dim=8, vdim=12, decay=[0.5, 0.9, 0.995], rot_dims=8), dict(dim=5, vdim=3, decay=[1.0], rot_dims=4, base=3.0),
             dict(dim=100, vdim=70, decay=[0.99, 0.0], rot_dims=66, base=1e6), dict(dim=32, vdim=32, decay=[0.6, 0.8, 0.9, 0.999], rot_dims=2),
             dict(dim=160, vdim=16, decay=[0.9, 0.7], rot_dims=160), dict(dim=64, vdim=64, decay=[0.98, 0.999], rot_dims=64),
             dict(dim=128, vdim=33, decay=[0.97], rot_dims=None), dict(dim=12, vdim=9, decay=[0.9, 0.8], rot_dims=0)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "decoded", "portions", "tokens"])
@pytest.mark.parametrize("case", RETENTION)
def test_retention_alone(case, how, dtype, tmp_path):
    """Key sizes in every register layout of the walk, values that do not fill a block's columns, the whole head, a part of it and
    nothing of it rotated; three requests in unequal portions over two state rows."""
    rig = rig_for([dict(retention(**case), mlp=None)], 40, dtype, tmp_path, seed=13, page=4, pages=90)
    mixer, m = rig.model.blocks[0].mixer, rig.config["layers"][0]["mixer"]
    lengths = {"a": 75, "b": 41, "c": 9}
    x = rows_for(lengths, 40, 7)
    want = {rid: plain.retention(x[rid], rig.w, "l0.mix.", m, 1e-5) for rid in x}
    got = rig.run(x, {rid: PLANS[how](n) for rid, n in lengths.items()}, lambda rows, ctx: mixer.forward(rows, ctx, 0))
    # (bfloat16: a norm over three values magnifies the rounding of each)
    tol = 3e-5 if dtype == "float32" else (4e-2 if case["vdim"] > 3 else 0.15)
    close(got, want, tol, f"retention {case} {how} {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_retention_reads_by_distance_over_hundreds_of_tokens(dtype, tmp_path):
    """A head that all but never forgets, what it was told once, far back: the read at each later token depends on the distance
    through the rotation, whether the tokens come at once, in portions or one by one."""
    layer = dict(retention(16, 8, [0.9999, 0.999], 16, 1e4), mlp=None)
    rig = rig_for([layer], 24, dtype, tmp_path, seed=13, page=8, pages=70)
    mixer, m = rig.model.blocks[0].mixer, rig.config["layers"][0]["mixer"]
    x = rows_for({"a": 420}, 24, 17)
    x["a"][1:300] *= 1e-3                      # one loud token, then hundreds of quiet ones
    want = plain.retention(x["a"], rig.w, "l0.mix.", m, 1e-5)
    short = x["a"].clone()
    short[0] = 0
    assert (plain.retention(short, rig.w, "l0.mix.", m, 1e-5)[290:300] - want[290:300]).abs().max() > 0.3 * want[290:300].abs().max()
    for plan in ([(0, 20)] + [(i, i + 1) for i in range(20, 420)], [(0, 420)], cuts_of(420, (64, 2, 31, 2, 2))):
        got = rig.run(x, {"a": plan}, lambda rows, ctx: mixer.forward(rows, ctx, 0))
        close(got, {"a": want}, 1e-4 if dtype == "float32" else 4e-2, "far write")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", [dict(dim=8, vdim=12, decay=[0.5, 0.99, 1.0], rot_dims=8), dict(dim=40, vdim=33, decay=[0.999, 0.95], rot_dims=8),
                                  dict(dim=100, vdim=70, decay=[0.9995], rot_dims=66, base=1e6),
                                  dict(dim=130, vdim=9, decay=[0.98], rot_dims=None)])
def test_retention_over_long_portions_walked_in_segments(case, dtype, tmp_path):
    """Portions long enough to be walked in segments side by side: whole segments and a rest, one token more than a segment,
    beside short portions and single tokens, from zeros and from a carried state, heads that soon forget and never."""
    rig = rig_for([dict(retention(**case), mlp=None)], 40, dtype, tmp_path, seed=13, page=16, pages=260, slots=4)
    mixer, m = rig.model.blocks[0].mixer, rig.config["layers"][0]["mixer"]
    lengths = {"a": 1024, "b": 1300, "c": 700, "d": 515, "e": 800}
    plans = {"a": [(0, 1024)], "b": [(0, 3), (3, 772), (772, 1029), (1029, 1030), (1030, 1300)], "c": [(0, 513), (513, 514), (514, 700)],
             "d": [(0, 1), (1, 515)], "e": [(0, 256), (256, 768), (768, 800)]}
    x = rows_for(lengths, 40, 7)
    want = {rid: plain.retention(x[rid], rig.w, "l0.mix.", m, 1e-5) for rid in x}
    got = rig.run(x, plans, lambda rows, ctx: mixer.forward(rows, ctx, 0), live=4)
    close(got, want, 1e-4 if dtype == "float32" else 4e-2, f"segments {case} {dtype}")


ROUTES = [dict(E=6, top=2, groups=(3, 2)), dict(E=12, top=3, groups=(3, 1)), dict(E=5, top=5, groups=None), dict(E=40, top=8, groups=(8, 3)),
          dict(E=64, top=1, groups=(64, 2)), dict(E=96, top=6, groups=(2, 1)), dict(E=33, top=32, groups=None), dict(E=1, top=1, groups=(1, 1)),
          dict(E=128, top=4, groups=(4, 4))]


@pytest.mark.gpu
@pytest.mark.parametrize("correction", [False, True])
@pytest.mark.parametrize("case", ROUTES)
def test_routing_alone(case, correction):
    """Choice among the best groups by corrected scores (negative ones too), weights without the correction, over their sum or not;
    one expert to 128, one group to as many as experts."""
    from tokenomos_b200 import ops

    E, top, groups = case["E"], case["top"], case["groups"]
    g = torch.Generator().manual_seed(E)
    T = 37
    z = 2.0 * torch.randn(T, E + 3, generator=g)
    c = torch.randn(E, generator=g) * 0.3 - 0.4 if correction else torch.zeros(E)
    rule = {"experts": E, "top": top}
    if groups is not None:
        rule["groups"] = {"count": groups[0], "keep": groups[1]}
    for renorm in (False, True):
        idx, w, _ = ops.moe_route(z.cuda(), E, top, 1.5, False, c.cuda() if correction else None, groups, renorm)
        for t in range(T):
            chosen, s = plain.route(z[t, :E].double(), c.double(), rule)
            assert idx[t].tolist() == chosen, (t, idx[t].tolist(), chosen)
            ref = 1.5 * (s / s.sum() if renorm else s)
            assert (w[t].double().cpu() - ref).abs().max() <= 2e-6


@pytest.mark.gpu
def test_routing_takes_the_lowest_index_among_equals_and_stays_inside_the_table():
    from tokenomos_b200 import ops

    z = torch.zeros(2, 8)
    z[1] = float("nan")                          # a padded row of a recorded step: any experts, but real ones
    idx, w, _ = ops.moe_route(z.cuda(), 8, 3, 1.0, False, torch.zeros(8).cuda(), (4, 2), False)
    assert idx[0].tolist() == [0, 1, 2] and (w[0].cpu() - 0.125).abs().max() < 1e-7
    assert ((idx[1] >= 0) & (idx[1] < 8)).all()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E, top, ff, limit, groups, shared, T", [
    (6, 2, 24, 1.5, (3, 2), (16, 0.6), 40), (5, 1, 40, 0.4, None, None, 33), (4, 4, 16, 2.0, (2, 2), (24, 5.0), 9),
    (40, 3, 8, 1.0, (8, 2), (8, 1.0), 70), (3, 2, 21, 0.8, (1, 1), (13, 2.0), 1), (8, 4, 64, 1.0, (4, 3), (64, 0.5), 300),
    (8, 2, 64, 1.2, (2, 1), None, 1100)])
def test_clamped_experts_with_a_shared_one_alone(dtype, E, top, ff, limit, groups, shared, T, tmp_path):
    """Experts and shared expert with limits of their own (met on both sides), few tokens, many (128-row tiles), and so many that
    the products are the library's; feed-forward sizes with and without whole runs of 8."""
    layer = dict(retention(8, 8, [0.5], 4), mlp=moe(E, top, ff, limit, groups, shared))
    rig = rig_for([layer], 32, dtype, tmp_path, seed=E + top)
    part = rig.model.blocks[0].ffn
    x = rows_for({"a": T}, 32, 29)["a"]
    f = rig.config["layers"][0]["mlp"]
    want = plain.experts(x, rig.w, "l0.mlp.", f)
    loose = json.loads(json.dumps(f))
    loose["expert"]["limit"] = 1e9
    assert (plain.experts(x, rig.w, "l0.mlp.", loose) - want).abs().max() > 0.1 * want.abs().max()
    got = part.forward(x.to(rig.dtype).cuda()).double().cpu()
    if dtype == "float32":
        assert (got - want).abs().max() <= 3e-5 * want.abs().max()
    else:
        # a close call of the router moves a row by a whole expert's output: most rows are within rounding
        err = (got - want).abs().amax(dim=1)
        assert (err <= 4e-2 * want.abs().max()).float().mean() >= 0.85 and torch.isfinite(got).all()


# ---------------------------------------------------------------------------------------------
# the whole model
# ---------------------------------------------------------------------------------------------

@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_every_way_of_cutting(name, dtype, folders):
    folder, _ = folders[name]
    page = CASES[name]["page"]
    reqs = requests_for(name)
    want = oracle(name, folders, reqs)
    results = {}
    for mode, steps in (("whole", trace_util.whole(reqs)),
                        ("tail", trace_util.tail_decoded(reqs, 48)),
                        ("portions", trace_util.portions(reqs)),
                        ("mixed", trace_util.mixed(reqs, live=4, seed=ord(name)))):
        # exactly the pages the trace's live requests need at its worst moment, all others and every page and state row
        # given back full of NaN
        max_tokens = trace_util.max_live_tokens(steps, page)
        per_step = trace_util.run_in_process(folder, dtype, steps, max_tokens, page, max_requests=4)
        got = trace_util.collect(steps, per_step)
        compare(got, want, TOL_F32 if dtype == "float32" else TOL_BF16, f"{name} {dtype} {mode}",
                close_calls=0.0 if dtype == "float32" else CLOSE_CALLS)
        results[mode] = got
    if dtype == "float32":
        for mode in ("tail", "portions", "mixed"):
            compare(results[mode], results["whole"], TOL_F32_SAME, f"{name} {dtype} {mode} vs whole")


def random_config(seed: int, wide: bool = False) -> tuple[dict, int]:
    """A configuration drawn from everything the design lets vary, and a page size. ``wide``: among the sizes the tensor-core
    kernels take in bfloat16, mixed with sizes they do not."""
    import random

    rng = random.Random(seed + (2000 if wide else 0))
    pick = rng.choice
    width = pick([128, 192, 256]) if wide else pick([16, 24, 30, 40, 64])
    dims = [32, 48, 64, 96, 128] if wide else [4, 8, 10, 16, 24]
    ffs = [64, 128, 192] if wide else [8, 20, 33, 64]
    kv, vdim = pick([1, 2, 3]), pick(dims)               # what layers that mix values have in common
    layers = []
    for i in range(rng.randint(3, 5) if wide else rng.randint(1, 6)):
        if rng.random() < 0.55:
            dim, mixes = pick(dims), rng.random() < 0.7
            layer = attention(kv * pick([1, 2, 4]), kv, dim, vdim if mixes else pick(dims), pick([2.0, 8.0, 40.0]) / dim,
                              pick([16, 63, 64, 65, 130, 500]) if wide else pick([1, 2, 7, 33, 64, 1000]), mixes)
            if not mixes:
                layer["mixer"].update(kv_heads=1)
        else:
            dim = pick(dims)
            layer = retention(dim, pick(dims), [pick([0.3, 0.9, 0.99, 0.999]) for _ in range(pick([1, 2, 4]))],
                              pick([dim, dim // 4 * 2, 2, None]), pick([10.0, 1e4, 1e6]))
        draw = rng.random()
        if draw < 0.15:
            layer["mlp"] = None
        elif draw < 0.4:
            layer["mlp"] = dense(pick(ffs))
        else:
            per, count = pick([1, 2, 4, 5]), pick([1, 2, 3, 4])
            keep = rng.randint(1, count)
            layer["mlp"] = moe(per * count, rng.randint(1, min(4, keep * per)), pick(ffs), pick([0.5, 1.0, 7.0]),
                               None if count == keep == 1 else (count, keep), pick([None, (pick(ffs), pick([0.5, 3.0]))]))
        layers.append(layer)
    return model(rng.randint(40, 300), width, layers, pick([1e-5, 1e-6]), pick([0.2, 0.5, 1.0])), 16 if wide else pick([4, 8, 16])


@pytest.mark.gpu
@pytest.mark.parametrize("wide", [False, True])
@pytest.mark.parametrize("seed", range(12))
def test_random_configurations(seed, wide, tmp_path):
    """Configurations nobody chose: whatever the draw gives, the 32-bit model meets the plain implementation however the requests
    are cut, and the 16-bit one stays close to it."""
    config, page = random_config(seed, wide)
    tensors = make_tensors(config, 300 + seed)
    write_folder(tmp_path, config, tensors)
    w = {k: v.double() for k, v in tensors.items()}
    g = torch.Generator().manual_seed(seed)
    reqs = {f"r{i}": torch.randint(0, config["vocab"], (n,), generator=g).tolist()
            for i, n in enumerate([2, 33, 70, 150] if wide else [1, 2, 17, 45, 80])}
    want = {rid: plain.forward(config, w, ids)[0] for rid, ids in reqs.items()}
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 0.2)):
        for steps in (trace_util.tail_decoded(reqs, 40) if wide else trace_util.portions(reqs), trace_util.mixed(reqs, live=4, seed=seed)):
            per_step = trace_util.run_in_process(tmp_path, dtype, steps, trace_util.max_live_tokens(steps, page), page,
                                                 max_requests=4)
            compare(trace_util.collect(steps, per_step), want, tol, f"random configuration {seed} {dtype}: {config}",
                    close_calls=0.0 if dtype == "float32" else 0.25, rare=0.02)


@pytest.mark.gpu
def test_layers_one_by_one(folders):
    """The residual stream after every layer, in 32-bit: a fault shows at the layer that has it."""
    from tokenomos_b200 import models
    from tokenomos_b200.cache.manager import CacheManager
    from tokenomos_b200.engine.step import StepEntry, StepFunction

    for name in ("A", "B", "C", "D"):
        folder, w = folders[name]
        ids = requests_for(name)["r3"]
        _, want = plain.forward(CASES[name]["config"], w, ids)
        conf = models.configure(folder, work="float32")
        stack = models.load(folder, "cuda", conf)
        cache = CacheManager(stack.state_specs(), 8, 40, 2, conf.work, "cuda", max_len=256, poison=True)
        seen = []
        for block in stack.blocks:
            def wrapped(h, residual, pending, ctx, call, inner=block.forward):
                y, stream, post = inner(h, residual, pending, ctx, call)
                seen.append((stream.double() + plain.rms(y.double(), post.eps) * post.scaled.double()).cpu())
                return y, stream, post
            block.forward = wrapped
        cache.admit("x")
        StepFunction(stack, cache).run([StepEntry("x", ids, [0])])
        assert len(seen) == want.shape[0]
        for layer, (got, ref) in enumerate(zip(seen, want)):
            assert (got - ref).abs().max() <= 2e-5 * ref.abs().max(), (name, layer)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_first_tokens(dtype, folders):
    """One and two token prompts, and 300 tokens decoded one by one: across many pages and chunks, the recurrent states carried
    all the way."""
    for name in ("A", "D"):
        folder, w = folders[name]
        g = torch.Generator().manual_seed(99)
        vocab = CASES[name]["config"]["vocab"]
        reqs = {"one": torch.randint(0, vocab, (1,), generator=g).tolist(),
                "two": torch.randint(0, vocab, (2,), generator=g).tolist(),
                "long": torch.randint(0, vocab, (303,), generator=g).tolist()}
        want = oracle(name, folders, reqs)
        steps = trace_util.tail_decoded(reqs, tail=300)
        page = CASES[name]["page"]
        per_step = trace_util.run_in_process(folder, dtype, steps, trace_util.max_live_tokens(steps, page), page,
                                             max_requests=4)
        compare(trace_util.collect(steps, per_step), want, TOL_F32 if dtype == "float32" else TOL_BF16,
                f"long decoding {name} {dtype}", close_calls=0.0 if dtype == "float32" else CLOSE_CALLS)


def test_a_changed_design_shows_in_the_plain_implementation(folders, monkeypatch):
    """Negative controls, planted in the plain implementation: chunks one longer, no sink, no unit heads, values not mixed or mixed
    with the wrong weight, another head's decay, no rotation, a read before the write, weights renormalized, the correction
    in the weights, groups ignored, another limit, no shared expert, another factor on the residual, no layer scale: all
    move the logits far beyond the bound that the engine meets."""
    name = "A"
    config, w = CASES[name]["config"], folders[name][1]
    ids = requests_for(name)["r4"]
    want = plain.forward(config, w, ids)[0]

    def moved(cfg=config, weights=w):
        got = plain.forward(cfg, weights, ids)[0]
        return ((got - want).abs().max() / want.abs().max()).item() / TOL_F32

    def changed(edit):
        c = json.loads(json.dumps(config))
        edit(c["layers"])
        return c

    assert moved() == 0
    assert moved(changed(lambda ls: ls[5]["mixer"].update(mask={"size": 7}))) > 100
    assert moved(changed(lambda ls: ls[5]["mixer"].update(v_mix=False))) > 100
    assert moved(changed(lambda ls: ls[2]["mixer"].update(v_mix=False))) > 100
    assert moved(changed(lambda ls: ls[0]["mixer"].update(decay=[0.9, 0.5, 0.995]))) > 100
    assert moved(changed(lambda ls: ls[0]["mixer"].pop("rot"))) > 100
    assert moved(changed(lambda ls: ls[0]["mixer"].update(rot={"dims": 12, "base": 10000.0}))) > 100
    assert moved(changed(lambda ls: ls[4]["mlp"]["router"].pop("groups"))) > 100
    assert moved(changed(lambda ls: ls[4]["mlp"]["expert"].update(limit=1.0))) > 100
    assert moved(changed(lambda ls: ls[4]["mlp"]["shared"].update(limit=1.0))) > 100
    assert moved(changed(lambda ls: ls[4]["mlp"].pop("shared"))) > 100
    assert moved(dict(config, residual_mult=1.0)) > 100
    for tensor in ("l3.ls1", "l3.ls2", "l5.norm1"):
        assert moved(weights={**w, tensor: torch.ones_like(w[tensor])}) > 100
    monkeypatch.setattr(plain, "mix_values", lambda v, first, lam: lam * v + (1 - lam) * first)
    assert moved() > 100
    monkeypatch.undo()
    monkeypatch.setattr(plain, "sink_softmax", lambda s, seen: torch.softmax(s.masked_fill(~seen, -math.inf), -1))
    assert moved() > 100
    monkeypatch.undo()
    real_route, real_scan = plain.route, plain.retention_scan

    def renormalized(z, c, r):
        chosen, s = real_route(z, c, r)
        return chosen, s / s.sum()

    def corrected(z, c, r):
        chosen, s = real_route(z, c, r)
        return chosen, s + c[chosen]

    for fault in (renormalized, corrected):
        monkeypatch.setattr(plain, "route", fault)
        assert moved() > 100
        monkeypatch.undo()
    # (a read before the write: what the tokens up to the one before have left)
    monkeypatch.setattr(plain, "retention_scan", lambda q, k, v, g: torch.cat((torch.zeros_like(v[:1]),
                                                                               real_scan(q[1:], k[:-1], v[:-1], g))))
    assert moved() > 100


@pytest.mark.gpu
def test_a_lost_state_shows(folders, monkeypatch):
    """The same replay without the recurrent states is far outside the bound that the real model meets (every index stays in
    bounds: the portions start from zeros)."""
    from tokenomos_b200 import ops

    name = "A"
    folder, _ = folders[name]
    reqs = {k: v for k, v in requests_for(name).items() if k in ("r3", "r4")}
    want = oracle(name, folders, reqs)
    steps = trace_util.portions(reqs)
    page = CASES[name]["page"]

    def worst():
        per_step = trace_util.run_in_process(folder, "float32", steps, trace_util.max_live_tokens(steps, page), page, poison=False)
        got = trace_util.collect(steps, per_step)
        return max(((got[rid] - want[rid]).abs().max() / want[rid].abs().max()).item() for rid in reqs)

    assert worst() <= TOL_F32
    real_scan = ops.linmem_scan

    def forgetful(*args, **kw):
        args = list(args)
        args[7] = torch.zeros_like(args[7])              # seq_ctx: every portion starts from zero
        return real_scan(*args, **kw)
    monkeypatch.setattr(ops, "linmem_scan", forgetful)
    assert worst() > 100 * TOL_F32


@pytest.mark.gpu
@pytest.mark.parametrize("page", [4, 16])
def test_pages_of_a_left_chunk_are_used_again(page, folders):
    """A pool with room for one chunk's pages beside a portion's, not for the request: decoding goes on because chunks that were
    left give their pages back, and the logits stay right on pages that were poisoned in between."""
    from tokenomos_b200 import models
    from tokenomos_b200.cache.manager import CacheManager
    from tokenomos_b200.engine.step import StepEntry, StepFunction

    name = "D"
    folder, _ = folders[name]
    ids = requests_for(name)["r4"]
    want = oracle(name, folders, {"r4": ids})["r4"]
    conf = models.configure(folder, work="float32")
    stack = models.load(folder, "cuda", conf)
    pages = 2 + (100 + 30) // page + 1
    cache = CacheManager(stack.state_specs(), page, pages, 1, conf.work, "cuda", max_len=320, poison=True)
    assert (pages - 1) * page < 200
    fn, rows = StepFunction(stack, cache), []
    cache.admit("x")
    for a, b in cuts_of(len(ids), (30, 1, 1, 17, 2)):
        rows.append(fn.run([StepEntry("x", ids[a:b], list(range(b - a)))]).double().cpu())
        cache.check()
    compare({"r4": torch.cat(rows)}, {"r4": want}, TOL_F32, "a small pool")


# ---------------------------------------------------------------------------------------------
# the entry points: LLM.generate through the scheduler, the command line, the trace program
# ---------------------------------------------------------------------------------------------

def teacher_forced_ok(config, w, prompt, reply, margin, close_calls: int = 0):
    """Every token of ``reply`` is the plain implementation's best, or within ``margin`` of it, but for ``close_calls`` tokens
    (16-bit runs only: a router's close call)."""
    logits, _ = plain.forward(config, w, prompt + reply)
    missed = 0
    for i, tok in enumerate(reply):
        row = logits[len(prompt) + i - 1]
        if int(row.argmax()) != tok and row.max().item() - row[tok].item() > margin:
            missed += 1
    assert missed <= close_calls, (missed, close_calls)


@pytest.mark.gpu
@pytest.mark.parametrize("name, work, graphs", [("A", "fp32", False), ("B", "fp32", True), ("D", "bf16", True),
                                                ("C", "fp32", True), ("D", "fp32", False), ("A", "bf16", True), ("A", "fp32", True)])
def test_greedy_generation_through_llm(name, work, graphs, folders):
    from tokenomos_b200 import LLM, SamplingParams

    folder, w = folders[name]
    config = CASES[name]["config"]
    g = torch.Generator().manual_seed(5)
    prompts = [torch.randint(0, config["vocab"], (n,), generator=g).tolist() for n in (1, 9, 40, 64, 23)]
    steps = 40
    with LLM(str(folder), work=work, page=CASES[name]["page"], max_len=256, slots=4, pages=120,
             prefill_budget=48, poison=True, graphs=graphs) as llm:
        outs = llm.generate(prompts, SamplingParams(max_tokens=steps))
    for prompt, out in zip(prompts, outs):
        assert out.prompt_tokens == len(prompt) and len(out.token_ids) == steps
        teacher_forced_ok(config, w, prompt, out.token_ids, 1e-3 if work == "fp32" else 0.3,
                          close_calls=0 if work == "fp32" else 6)


@pytest.mark.gpu
def test_trace_program_and_command_line(folders, tmp_path):
    name = "A"
    folder, _ = folders[name]
    reqs = requests_for(name)
    want = oracle(name, folders, reqs)
    steps = trace_util.mixed(reqs, live=4, seed=3)
    per_step = trace_util.run_program(folder, "float32", steps, trace_util.max_live_tokens(steps, 64), tmp_path,
                                      CASES[name]["config"]["vocab"])
    compare(trace_util.collect(steps, per_step), want, TOL_F32, "trace program")
    cmd = [sys.executable, "-m", "tokenomos_b200.generate", "--model", str(folder), "--prompt-ids", "1,2,3,4",
           "--max-tokens", "5", "--arch-kw", '{"work": "fp32"}',
           "--engine-kw", '{"page": 4, "max_len": 64, "slots": 2, "pages": 40}']
    proc = subprocess.run(cmd, capture_output=True, text=True, cwd=ROOT, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [json.loads(ln) for ln in proc.stdout.splitlines() if ln.startswith("{")]
    assert len(lines) == 1 and len(lines[0]["token_ids"]) == 5
    teacher_forced_ok(CASES[name]["config"], folders[name][1], [1, 2, 3, 4], lines[0]["token_ids"], 1e-3)
