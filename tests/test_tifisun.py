"""The Tifisun decoder against its plain implementation (``plain_tifisun``): every mechanism alone (the norm behind a
sublayer, norms over whole query and key rows, attention with a soft cap and a bias by distance in a window, the
gated delta rule with one decay per head and with one per key channel, lightning attention, the pair of mixers, the
gelu-gated feed-forward), the whole model replayed four ways in 32-bit and in bfloat16 on poisoned pools, keys made
loud far back, at page borders and at the window's edge, states carried over portions down to two tokens, layers that
use another layer's weights with a cache and state of their own, long decoding, generation through the entry points.
The configurations are made for the tests: other layer orders, one head, one tap, a window of one, a table of two
rows, layers without a feed-forward, caps too wide for the form without a running maximum, sizes no 16-byte kernel
takes and sizes the tensor-core kernels take."""

from __future__ import annotations

import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_tifisun as plain
import trace_util

ROOT = Path(__file__).resolve().parents[1]


def delta(heads, kv_heads, dim, vdim, conv, channel=False):
    return {"type": "channel_delta" if channel else "delta",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def windowed(heads, kv_heads, dim, vdim, scale, softcap, bias_max, window):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
            "bias_max": bias_max, "mask": {"size": window}}


def memory(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def parallel(left, right):
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def model(vocab, width, layers, eps=1e-5, mult=0.5, scale=2.0):
    return {"architecture": "Tifisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale}, "layers": layers}


def dense(ff):
    return {"kind": "dense", "ff": ff}


# A: the channel delta rule first, with q/k heads shared; a window of 11 positions over pages of 4; a layer that uses the
#    first one's weights, one that uses the pair's, one that uses a layer that comes later; a layer without a feed-forward
_A0 = dict(delta(4, 2, 12, 8, 3, channel=True), mlp=dense(40))
_A1 = dict(parallel(windowed(4, 2, 12, 20, 0.4, 12.0, 9, 11), memory(3, 8, 12, [0.5, 0.9, 0.995])), mlp=dense(64))
_A2 = dict(delta(3, 1, 8, 12, 4), mlp=None)
TF_A = model(300, 48, [_A0, _A1, dict(_A2, weights_of=5), dict(_A0, weights_of=0), dict(_A1, weights_of=1), _A2], mult=0.7)
# B: one head everywhere, one tap, a window of one position, a factor and a scale of 1
TF_B = model(200, 64, [dict(delta(1, 1, 16, 40, 1), mlp=dense(96)),
                       dict(parallel(windowed(1, 1, 16, 8, 0.25, 30.0, 20, 1), memory(1, 16, 16, [0.97])), mlp=None),
                       dict(delta(1, 1, 40, 8, 2, channel=True), mlp=dense(24))], eps=1e-6, mult=1.0, scale=1.0)
# C: sizes no 16-byte kernel takes; five taps (more than the shortest portions); a window longer than any request; a cap too
#    wide for a softmax without a running maximum; more rows in the bias table than distances told apart
TF_C = model(50, 36, [dict(delta(3, 3, 5, 7, 5), mlp=dense(30)),
                      dict(parallel(windowed(3, 3, 7, 10, 0.5, 60.0, 4, 500), memory(2, 9, 3, [1.0, 0.25])), mlp=dense(21)),
                      dict(delta(2, 1, 9, 6, 5, channel=True), mlp=dense(9))], mult=0.3, scale=3.5)
# D: sizes the tensor-core kernels take in bfloat16 (keys of 64 and of 24 in one 64-wide tile, values of another size), longer
#    requests, windows of 100 and 40 over pages of 16
TF_D = model(400, 128, [dict(delta(4, 2, 32, 64, 4), mlp=dense(256)),
                        dict(parallel(windowed(8, 2, 64, 64, 0.125, 20.0, 90, 100), memory(4, 32, 32, [0.6, 0.9, 0.98, 0.999])),
                             mlp=dense(128)),
                        dict(delta(4, 4, 64, 32, 4, channel=True), mlp=dense(128)),
                        dict(parallel(windowed(4, 4, 24, 128, 0.2, 55.0, 64, 40), memory(2, 64, 72, [0.8, 0.99])), mlp=None),
                        dict(delta(4, 2, 32, 64, 4), mlp=dense(256), weights_of=0)])

CASES = {
    "A": dict(config=TF_A, seed=51, page=4, lengths=[1, 2, 7, 30, 61, 45], free=(5, 9, 8)),
    "B": dict(config=TF_B, seed=52, page=8, lengths=[3, 19, 21, 50, 90, 33], free=(1, 3, 2)),
    "C": dict(config=TF_C, seed=53, page=4, lengths=[1, 6, 23, 40, 5], free=(3, 2, 6)),
    "D": dict(config=TF_D, seed=54, page=16, lengths=[2, 31, 150, 65, 300, 90], free=(16, 24, 16)),
}
# Bounds relative to a request's largest |logit|. The 32-bit model computes what the plain implementation computes, in
# another order; bfloat16 rounds every product's inputs and outputs.
TOL_F32 = {"A": 4e-5, "B": 4e-5, "C": 4e-5, "D": 4e-5}
TOL_F32_SAME = {"A": 3e-5, "B": 3e-5, "C": 3e-5, "D": 3e-5}
TOL_BF16 = {"A": 0.12, "B": 0.12, "C": 0.12, "D": 0.12}


def make_tensors(config: dict, seed: int, free=(4, 6, 8)) -> dict[str, torch.Tensor]:
    """Random weights, rounded to bfloat16: queries and keys loud enough that a key more or less moves the logits far
    beyond rounding, norm weights far from one, taps of the size of the signal, decays spread from fast to slow. ``free``:
    the sizes only the tensors give (inner widths of the decay's and the gate's projections, rows of the bias table)."""
    from tokenomos_b200 import models

    arch = models.architecture_of(config)
    spec = arch.declare(arch.config_class.from_dict(config))
    noise = torch.Generator().manual_seed(seed)
    sizes = {"a": free[0], "g": free[1], "rel": free[2]}
    out = {}
    for d in spec.tensor_decls():
        if d.optional:
            continue
        shape = [sizes[s.name.split(".rank")[0].split(".rows")[0].rsplit(".", 1)[-1]] if hasattr(s, "name") else s for s in d.shape]
        r, u = torch.randn(shape, generator=noise), torch.rand(shape, generator=noise)
        n = d.name
        if n.endswith((".norm1", ".norm2", ".norm1b", ".norm2b")) or n == "final.norm":
            t = 0.3 * r
        elif n.endswith((".norm", ".out")):
            t = 1.0 + 0.3 * r
        elif n.endswith(".conv"):
            t = 0.7 * r
        elif n.endswith(".dt_bias"):
            t = -4.0 + 5.0 * u
        elif n.endswith(".A_log"):
            t = -3.0 + 4.0 * u
        elif n.endswith(".b") and ".mlp." in n:
            t = 0.5 * r
        elif n.endswith(".rel") or n == "embed":
            t = r
        elif n.endswith((".a", ".b")):
            t = r * (2.0 / math.sqrt(shape[-1]))
        else:
            t = r / math.sqrt(shape[-1])
        out[n] = t.to(torch.bfloat16)
    return out


def write_folder(folder: Path, config: dict, tensors: dict) -> None:
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, case in CASES.items():
        folder = tmp_path_factory.mktemp(f"tf_{name}")
        tensors = make_tensors(case["config"], case["seed"], case["free"])
        write_folder(folder, case["config"], tensors)
        out[name] = (folder, {k: v.double() for k, v in tensors.items()})
    return out


def requests_for(name: str) -> dict[str, list[int]]:
    g = torch.Generator().manual_seed(411 + ord(name))
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


def compare(got: dict, want: dict, tol: float, what: str):
    for rid, ref in want.items():
        assert got[rid].shape == ref.shape, (what, rid, got[rid].shape, ref.shape)
        assert torch.isfinite(got[rid]).all(), (what, rid)
        err = (got[rid] - ref).abs().amax(dim=1)
        scale = ref.abs().max().item()
        bad = (err > tol * scale).nonzero()
        assert bad.numel() == 0, (f"{what}: request {rid}: first wrong position {int(bad[0])} of {len(err)}: error "
                                  f"{err[int(bad[0])].item():.3e}, allowed {tol * scale:.3e}")


# ---------------------------------------------------------------------------------------------
# without a GPU: configuration, declaration, the oracle's own pieces
# ---------------------------------------------------------------------------------------------

def test_configuration_reads_every_size_and_lists_every_fault():
    from tokenomos_b200.config import ConfigError, TifisunConfig

    cfg = TifisunConfig.from_dict(TF_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.residual_mult, cfg.embed_scale) == (300, 48, 1e-5, 0.7, 2.0)
    assert [layer.kind for layer in cfg.layers] == ["channel_delta", "parallel", "delta", "channel_delta", "parallel", "delta"]
    assert [layer.weights for layer in cfg.layers] == [0, 1, 5, 0, 1, 5] and [layer.ff for layer in cfg.layers] == [
        40, 64, None, 40, 64, None]
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.taps) == (4, 2, 12, 8, 3)
    lt, rt = cfg.layers[1].mixer.left, cfg.layers[1].mixer.right
    assert (lt.heads, lt.kv_heads, lt.dim, lt.vdim, lt.scale, lt.softcap, lt.bias_max, lt.window) == (4, 2, 12, 20, 0.4, 12.0, 9, 11)
    assert (rt.heads, rt.dim, rt.vdim, rt.decay) == (3, 8, 12, (0.5, 0.9, 0.995))
    bare = json.loads(json.dumps(TF_B))
    del bare["embedding"], bare["layers"][1]["mixer"]["left"]["softcap"], bare["layers"][1]["mixer"]["left"]["mask"]
    cfg = TifisunConfig.from_dict(bare)
    assert cfg.embed_scale == 1.0 and cfg.layers[1].mixer.left.softcap is None and cfg.layers[1].mixer.left.window is None
    # weights borrowed through a chain end at the layer that has them
    chain = json.loads(json.dumps(TF_A))
    chain["layers"][3]["weights_of"] = 0
    chain["layers"].append(dict(chain["layers"][3], weights_of=3))
    assert TifisunConfig.from_dict(chain).layers[6].weights == 0
    bad = json.loads(json.dumps(TF_A))
    del bad["width"]
    bad["layers"][0]["mixer"]["kv_heads"] = 3                            # 4 heads over 3
    bad["layers"][1]["mixer"]["right"]["decay"] = [0.5]                  # 3 heads
    bad["layers"][2]["type"] = "something"
    bad["layers"][4]["mlp"]["kind"] = "odd"
    bad["layers"][5]["mixer"].pop("conv")
    with pytest.raises(ConfigError) as err:
        TifisunConfig.from_dict(bad)
    text = str(err.value)
    assert all(s in text for s in ("width", "4 heads over 3", "decay", "something", "'odd'", "conv"))
    worse = json.loads(json.dumps(TF_A))
    worse["layers"][3]["mixer"]["dim"] = 16                              # not the entry whose weights it uses
    worse["layers"][4]["weights_of"] = 9
    worse["layers"][1]["weights_of"] = 4
    with pytest.raises(ConfigError) as err:
        TifisunConfig.from_dict(worse)
    assert "entries differ" in str(err.value) and "weights_of = 9" in str(err.value)


def test_declaration_lists_the_tensors_the_order_and_the_state(folders):
    from tokenomos_b200 import models
    from tokenomos_b200.parts import build_model
    from tokenomos_b200.parts.contract import WindowKV
    from tokenomos_b200.parts.registry import Runtime
    from tokenomos_b200.weights.checkpoint import Checkpoint, WeightError, check, load_tensors

    arch = models.architecture_of(TF_A)
    spec = arch.declare(arch.config_class.from_dict(TF_A))
    names = {d.name: d for d in spec.tensor_decls()}
    assert names["head"].shape == (300, 48) and names["l0.mix.dt_bias"].shape == (48,) and names["l5.mix.dt_bias"].shape == (3,)
    assert names["l0.mix.q"].shape == (24, 48) and names["l0.mix.v.conv"].shape == (32, 3) and names["l0.mix.norm"].shape == (8,)
    assert names["l1.mix.left.k.norm"].shape == (24,) and names["l1.mix.right.norm"].shape == (36,)
    assert names["l1.mix.left.o"].shape == (48, 80) and names["l1.mlp.down.b"].shape == (48,)
    assert "l5.mix.g" in names and "l5.mix.g1" not in names and names["l5.norm2b"].optional
    assert not any(n.startswith(("l2.", "l3.", "l4.")) for n in names)
    assert [call.block for call in spec.order] == [0, 1, 2, 0, 1, 2]
    # sizes that only the tensors give are whatever is stored, the same on both sides of an inner width
    folder, _ = folders["A"]
    ckpt = Checkpoint(folder)
    check(ckpt, spec.tensor_decls(), spec.scope)
    assert ckpt.shape("l0.mix.a1") == (5, 48) and ckpt.shape("l0.mix.g2") == (32, 9) and ckpt.shape("l1.mix.left.rel") == (8, 4)

    class Other:
        def names(self):
            return ckpt.names()

        def shape(self, name):
            return (32, 7) if name == "l0.mix.g2" else ckpt.shape(name)

    with pytest.raises(WeightError) as err:
        check(Other(), spec.tensor_decls(), spec.scope)
    assert "l0.mix.g2" in str(err.value) and "[32, 9]" in str(err.value)
    tensors = load_tensors(ckpt, spec.tensor_decls(), torch.float32, "cpu")
    stack = build_model(spec, tensors, Runtime(torch.float32, torch.device("cpu")))
    states = stack.state_specs()
    assert set(states) == {(0, "S"), (0, "conv"), (1, "left.kv"), (1, "right.S"), (2, "S"), (2, "conv"), (3, "S"), (3, "conv"),
                           (4, "left.kv"), (4, "right.S"), (5, "S"), (5, "conv")}
    assert states[(4, "left.kv")] == WindowKV(2, 20, 11) and states[(3, "conv")].shape == (2, 80)
    assert stack.capture_safe


def test_distance_buckets_are_the_plain_ones():
    from tokenomos_b200.parts.attention import distance_bucket

    for rows, far in ((8, 9), (2, 20), (6, 4), (16, 90), (32, 1000), (10, 64)):
        got = [distance_bucket(n, rows, far) for n in range(2 * int(far) + rows)]
        assert got == [plain.bucket(n, rows, far) for n in range(len(got))]
        assert got[0] == 0 and got[-1] == rows - 1 and all(0 <= b - a <= rows for a, b in zip(got, got[1:]))
    # eight rows up to 32: four single distances, then steps of a factor of 8^(1/4)
    assert [plain.bucket(n, 8, 32) for n in (0, 3, 4, 6, 7, 11, 12, 19, 20, 32, 500)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7]


def test_oracle_pieces():
    u = torch.arange(8, dtype=torch.float64).view(4, 2)
    taps = torch.tensor([[1.0, 0.0, 2.0], [0.0, 1.0, 0.0]], dtype=torch.float64)
    out = plain.causal_conv(u, taps)           # the last column is the current token's
    assert out[:, 0].tolist() == [0.0, 4.0, 8.0, 14.0] and out[:, 1].tolist() == [0.0, 1.0, 3.0, 5.0]
    z = torch.tensor([0.5, -2.0], dtype=torch.float64)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert torch.allclose(plain.softplus(z * 30), torch.nn.functional.softplus(z * 30))
    # two tokens of the delta rule by hand: the second reads what the first left, decayed, before it moves it
    t = lambda *v: torch.tensor(v, dtype=torch.float64)
    q, k = t([[1.0, 0.0]], [[0.5, 1.0]]), t([[0.6, 0.8]], [[1.0, 0.0]])
    v, g, beta = t([[2.0]], [[5.0]]), t([[1.0, 1.0]], [[0.5, 0.25]]), t([0.5], [0.25])
    S = [0.6 * 1.0, 0.8 * 1.0]                 # u = 0.5 * 2
    out = [S[0]]
    S = [0.5 * S[0], 0.25 * S[1]]
    u = 0.25 * (5.0 - S[0])
    S = [S[0] + u, S[1]]
    out.append(0.5 * S[0] + S[1])
    assert torch.allclose(plain.delta_scan(q, k, v, g, beta).flatten(), t(*out))


# ---------------------------------------------------------------------------------------------
# each mechanism alone, on the GPU
# ---------------------------------------------------------------------------------------------

def cuts_of(n: int, sizes) -> list[tuple[int, int]]:
    out, a, k = [], 0, 0
    while a < n:
        b = min(n, a + sizes[k % len(sizes)])
        out.append((a, b))
        a, k = b, k + 1
    return out


class Rig:
    """A few layers loaded as the framework loads a folder, over a NaN-poisoned pool of pages and state rows; ``run``
    lays a step out as the step function does and hands the context to one part. Requests are fed in unequal portions
    side by side and a freed slot is used again."""

    def __init__(self, layers, width, dtype, folder, seed=0, page=4, pages=120, slots=2, edit=None, free=(4, 6, 8)):
        from tokenomos_b200 import models
        from tokenomos_b200.cache.manager import CacheManager
        from tokenomos_b200.engine.step import StepFunction

        self.config = model(16, width, layers)
        tensors = make_tensors(self.config, seed, free)
        if edit is not None:
            edit(tensors)
        write_folder(folder, self.config, tensors)
        self.w = {k: v.double() for k, v in tensors.items()}
        conf = models.configure(folder, work=dtype)
        self.dtype = conf.work
        self.model = models.load(folder, "cuda", conf)
        self.cache = CacheManager(self.model.state_specs(), page, pages, slots, conf.work, "cuda",
                                  max_len=(pages - 1) * page, poison=True)
        self.steps = StepFunction(self.model, self.cache)
        # hold and return a few pages so that the requests' pages are neither the first nor in order
        self.cache.admit("junk")
        self.cache.extend("junk", 3 * page)
        self.cache.admit("junk2")
        self.cache.extend("junk2", page)
        self.cache.release("junk")
        self.cache.release("junk2")

    def run(self, inputs: dict[str, torch.Tensor], plans: dict[str, list], fn, live=2) -> dict[str, torch.Tensor]:
        """``inputs``: request -> rows [n, width]; ``plans``: request -> list of (a, b) portions. ``fn(x, ctx)`` is called
        with the step's rows in the work dtype; its output rows are collected."""
        from tokenomos_b200.engine.step import StepEntry

        plans = {rid: list(p) for rid, p in plans.items()}
        waiting = list(inputs)
        active, got = [], {rid: [] for rid in inputs}
        while waiting or active:
            while waiting and len(active) < live:
                rid = waiting.pop(0)
                self.cache.admit(rid)
                active.append(rid)
            spans = [(rid, plans[rid].pop(0)) for rid in active]
            entries = [StepEntry(rid, [0] * (b - a), []) for rid, (a, b) in spans]
            ctx, _, _ = self.steps.layout(entries)
            x = torch.cat([inputs[rid][a:b] for rid, (a, b) in spans]).to(self.dtype).cuda().contiguous()
            out = fn(x, ctx)
            o = 0
            for rid, (a, b) in spans:
                self.cache.commit(rid, b - a)
                got[rid].append(out[o:o + b - a].double().cpu())
                o += b - a
            for rid in list(active):
                if not plans[rid]:
                    self.cache.release(rid)
                    active.remove(rid)
            self.cache.check()
        return {rid: torch.cat(parts) for rid, parts in got.items()}


def rows_for(lengths: dict[str, int], width: int, seed: int, scale: float = 1.0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    return {rid: (scale * torch.randn(n, width, generator=g)).to(torch.bfloat16).double() for rid, n in lengths.items()}


PLANS = {
    "whole": lambda n: [(0, n)],
    "decoded": lambda n: [(0, max(1, n - 20))] + [(i, i + 1) for i in range(max(1, n - 20), n)],
    "portions": lambda n: cuts_of(n, (5, 2, 17, 3, 2, 29, 1, 1, 4)),
    "tokens": lambda n: [(i, i + 1) for i in range(n)],
}


def close(got, want, tol, what):
    for rid, ref in want.items():
        assert torch.isfinite(got[rid]).all(), (what, rid)
        err = (got[rid] - ref).abs().amax(dim=-1)
        bad = (err > tol * ref.abs().max()).nonzero()
        assert bad.numel() == 0, (f"{what}: request {rid}: first wrong row {int(bad[0])} of {len(err)}: "
                                  f"{err[int(bad[0])].item():.3e} against {tol * ref.abs().max().item():.3e}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 30, 36, 512, 2048, 1027, 6144, 8200])
def test_norm_behind_a_sublayer_and_the_join_of_a_pair(width, dtype):
    """``stream + m n(x)`` in 32-bit and the norm that follows, alone and as the last add; and the mean of two normed rows:
    widths with and without whole 16-byte chunks, rows that stay in registers and rows that do not, strided rows."""
    from tokenomos_b200 import ops

    g = torch.Generator().manual_seed(width)
    T = 5
    stream = torch.randn(T, width, generator=g) * 3
    wide = torch.randn(T, 2 * width + 8, generator=g).to(dtype)
    dev = wide.cuda()
    wx, w = 0.5 * (1 + 0.3 * torch.randn(width, generator=g)), 1 + 0.3 * torch.randn(width, generator=g)
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    for lo in (0, width + 8):
        x = wide[:, lo:lo + width].double()
        for s in (stream, None):
            want_stream = (s.double() if s is not None else 0) + plain.rms(x, 1e-3) * wx.double()
            want = plain.rms(want_stream, 1e-5) * w.double()
            y, new = ops.stream32_post_norm(s.cuda() if s is not None else None, dev[:, lo:lo + width], wx.cuda(), 1e-3, w.cuda(), 1e-5)
            assert new.dtype == torch.float32 and (new.double().cpu() - want_stream).abs().max() <= 2e-6 * want_stream.abs().max()
            assert y.dtype == dtype and (y.double().cpu() - want).abs().max() <= tol * want.abs().max()
            y, again = ops.stream32_post_norm(s.cuda() if s is not None else None, dev[:, lo:lo + width], wx.cuda(), 1e-3, None, 0.0)
            assert y is None and torch.equal(again, new)
    a, b = wide[:, :width], wide[:, width + 8:]
    want = 0.5 * (plain.rms(a.double(), 1e-5) * wx.double() + plain.rms(b.double(), 1e-5) * w.double())
    got = ops.pair_norm_mean(dev[:, :width], dev[:, width + 8:], wx.cuda(), w.cuda(), 1e-5)
    assert (got.double().cpu() - want).abs().max() <= tol * want.abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups, width, kind", [(6, 192, "silu"), (1, 60, "sigmoid"), (3, 21, "silu"), (1, 2048, "sigmoid"),
                                                 (16, 2048, "silu"), (2, 1000, "sigmoid"), (1, 5000, "silu")])
def test_norm_then_gate(dtype, groups, width, kind):
    from tokenomos_b200 import ops

    g = torch.Generator().manual_seed(width)
    y = torch.randn(4, width, generator=g) * 2
    z = torch.randn(4, width + 5, generator=g).to(dtype)
    w = 1 + 0.3 * torch.randn(width, generator=g)
    zd = z[:, 5:].double()
    gate = torch.sigmoid(zd) * (zd if kind == "silu" else 1)
    want = plain.rms(y.double().view(4, groups, -1), 1e-4).reshape(4, width) * w.double() * gate
    got = ops.norm_gate(y.cuda(), z.cuda()[:, 5:], w.cuda(), 1e-4, groups, kind)
    assert (got.double().cpu() - want).abs().max() <= (2e-6 if dtype == torch.float32 else 6e-3) * want.abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff, T", [(24, 5), (24, 40), (21, 3), (256, 8), (256, 70), (40, 1)])
def test_gelu_gated_feed_forward_alone(ff, T, dtype, tmp_path):
    """Few rows (the activation in the product's epilogue) and many, feed-forward sizes with and without whole runs of 8."""
    rig = Rig([dict(delta(1, 1, 8, 8, 2), mlp=dense(ff))], 32, dtype, tmp_path, seed=ff)
    x = rows_for({"a": T}, 32, 29, 2.0)["a"]
    want = plain.feed_forward(x, rig.w, "l0.mlp.")
    got = rig.model.blocks[0].ffn.forward(x.to(rig.dtype).cuda()).double().cpu()
    assert (got - want).abs().max() <= (3e-6 if dtype == "float32" else 2e-2) * want.abs().max()


ATTENTION = [dict(heads=4, kv_heads=2, dim=12, vdim=20, window=11, softcap=12.0, bias_max=9),
             dict(heads=1, kv_heads=1, dim=6, vdim=40, window=1, softcap=5.0, bias_max=30),
             dict(heads=3, kv_heads=3, dim=24, vdim=8, window=500, softcap=70.0, bias_max=60),
             dict(heads=8, kv_heads=2, dim=64, vdim=64, window=70, softcap=20.0, bias_max=50),
             dict(heads=6, kv_heads=2, dim=128, vdim=64, window=33, softcap=20.0, bias_max=200),
             dict(heads=4, kv_heads=4, dim=48, vdim=96, window=65, softcap=55.0, bias_max=64),
             dict(heads=16, kv_heads=1, dim=104, vdim=128, window=64, softcap=15.0, bias_max=12)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "decoded", "portions"])
@pytest.mark.parametrize("case", ATTENTION)
def test_capped_and_biased_attention_alone(case, how, dtype, tmp_path):
    """Head layouts with values wider and narrower than the keys, one head, a window of one and one longer than any request,
    caps with and without a bounded softmax, tables that end inside and outside the window, sizes the tensor-core kernels
    take (padded tiles too) and sizes they do not; two requests side by side."""
    left = windowed(case["heads"], case["kv_heads"], case["dim"], case["vdim"], 3.0 / case["dim"], case["softcap"], case["bias_max"],
                    case["window"])
    rig = Rig([dict(parallel(left, memory(1, 4, 4, [0.5])), mlp=None)], 32, dtype, tmp_path, seed=3, page=4, pages=140, free=(1, 1, 10))
    pair = rig.model.blocks[0].mixer
    mixer = pair.branches[0]
    lengths = {"a": 97, "b": 38, "c": 140}
    x = rows_for(lengths, 32, 5)
    want = {rid: plain.windowed_attention(x[rid], rig.w, "l0.mix.left.", left, 1e-5) for rid in x}
    got = rig.run(x, {rid: PLANS[how](n) for rid, n in lengths.items()},
                  lambda rows, ctx: mixer.forward(rows, pair._contexts(ctx)[0], 0))
    close(got, want, 2e-5 if dtype == "float32" else 4e-2, f"attention {case} {how} {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "decoded", "portions"])
@pytest.mark.parametrize("window", [9, 64, 329])
def test_one_loud_key_at_page_borders_and_at_the_windows_edge(window, how, dtype, tmp_path):
    """One key that the last queries lean towards, everything else quiet: the query's own, around a page border, hundreds of
    positions back, just inside and just outside the window. A key that is dropped, read from a wrong page or let in one
    position too early or too late changes the output by its own size; the plain implementation with a window one longer
    or shorter is the control."""
    page, width, T = 8, 32, 330
    left = windowed(2, 1, 16, 16, 1.0, 25.0, 40, window)

    def edit(t):
        # keys read the first half of the input's channels alone, and both query heads read the second half as the key
        # head reads the first: a query row [0 | l] scores high against a key row [l | 0] and against no other query row
        k = t["l0.mix.left.k"].clone()
        k[:, width // 2:] = 0
        t["l0.mix.left.k"] = k
        t["l0.mix.left.q"] = torch.cat((k.roll(width // 2, dims=1), k.roll(width // 2, dims=1)))
        t["l0.mix.left.q.norm"].fill_(1.0)
        t["l0.mix.left.k.norm"].fill_(1.0)
        t["l0.mix.left.rel"] *= 0.3

    rig = Rig([dict(parallel(left, memory(1, 4, 4, [0.5])), mlp=None)], width, dtype, tmp_path, seed=9, page=page, pages=60, edit=edit)
    pair = rig.model.blocks[0].mixer
    mixer = pair.branches[0]
    tol = 2e-5 if dtype == "float32" else 4e-2
    last = T - 1
    places = [last, last - 1, last - window + 2, last - window + 1, last - window, last - window - 1]
    places += [p for p in (0, 1, page - 1, page, 2 * page, T - 257) if last - p < window]
    for loud in sorted({p for p in places if p >= 0}):
        g = torch.Generator().manual_seed(loud)
        # (the norm over the whole row brings every key to one size: quiet keys point away from the lean instead)
        lean = torch.randn(width // 2, generator=g).to(torch.bfloat16).double()
        x = torch.randn(T, width, generator=g).to(torch.bfloat16).double()
        x[:, :width // 2] = (x[:, :width // 2] - 1.5 * lean).to(torch.bfloat16).double()
        x[loud, :width // 2] = 3.0 * lean
        x[T - 3:, width // 2:] = 3.0 * lean
        want = plain.windowed_attention(x, rig.w, "l0.mix.left.", left, 1e-5)
        if loud in (last - window + 1, last - window):
            # the control: at the edge, a window one position off gives another last row
            off = dict(left, mask={"size": window + (1 if loud == last - window else -1)})
            other = plain.windowed_attention(x, rig.w, "l0.mix.left.", off, 1e-5)
            assert (want[-1] - other[-1]).abs().max() > 0.3 * want[-1].abs().max(), loud
        got = rig.run({"x": x}, {"x": PLANS[how](T)}, lambda rows, ctx: mixer.forward(rows, pair._contexts(ctx)[0], 0))
        close(got, {"x": want}, tol, f"loud key at {loud}, window {window}, {how}, {dtype}")


DELTA = [dict(heads=4, kv_heads=2, dim=12, vdim=8, conv=3), dict(heads=1, kv_heads=1, dim=5, vdim=3, conv=1),
         dict(heads=3, kv_heads=3, dim=48, vdim=72, conv=4), dict(heads=6, kv_heads=2, dim=64, vdim=33, conv=8),
         dict(heads=2, kv_heads=1, dim=130, vdim=40, conv=2)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "decoded", "portions", "tokens"])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("case", DELTA)
def test_delta_rule_alone(case, channel, how, dtype, tmp_path):
    """Head counts over shared and own q/k heads, key sizes of 5 to 130 (every register layout of the walk), one to eight taps,
    values that do not fill a block's columns, inner widths of one and more; three requests in unequal portions over two
    state rows."""
    rig = Rig([dict(delta(channel=channel, **case), mlp=None)], 40, dtype, tmp_path, seed=11, page=4, pages=90,
              free=(1 if case["conv"] == 1 else 7, 3, 4))
    mixer = rig.model.blocks[0].mixer
    m = rig.config["layers"][0]["mixer"]
    lengths = {"a": 75, "b": 41, "c": 9}
    x = rows_for(lengths, 40, 7)
    want = {rid: plain.delta(x[rid], rig.w, "l0.mix.", m, 1e-5, channel) for rid in x}
    got = rig.run(x, {rid: PLANS[how](n) for rid, n in lengths.items()}, lambda rows, ctx: mixer.forward(rows, ctx, 0))
    # (bfloat16: a norm over three values magnifies the rounding of each)
    tol = 2e-5 if dtype == "float32" else (4e-2 if case["vdim"] > 3 else 0.15)
    close(got, want, tol, f"delta rule {case} channel={channel} {how} {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "decoded", "portions", "tokens"])
@pytest.mark.parametrize("case", [dict(heads=3, dim=8, vdim=12, decay=[0.5, 0.9, 0.995]), dict(heads=1, dim=5, vdim=3, decay=[1.0]),
                                  dict(heads=2, dim=100, vdim=70, decay=[0.99, 0.0]), dict(heads=4, dim=32, vdim=32, decay=[0.6, 0.8, 0.9, 0.999]),
                                  dict(heads=2, dim=160, vdim=16, decay=[0.9, 0.7])])
def test_lightning_attention_alone(case, how, dtype, tmp_path):
    layer = dict(parallel(windowed(1, 1, 4, 4, 0.5, 10.0, 8, 4), memory(**case)), mlp=None)
    rig = Rig([layer], 40, dtype, tmp_path, seed=13, page=4, pages=90)
    pair = rig.model.blocks[0].mixer
    lengths = {"a": 75, "b": 41, "c": 9}
    x = rows_for(lengths, 40, 7)
    want = {rid: plain.lightning(x[rid], rig.w, "l0.mix.right.", case, 1e-5) for rid in x}
    got = rig.run(x, {rid: PLANS[how](n) for rid, n in lengths.items()},
                  lambda rows, ctx: pair.branches[1].forward(rows, pair._contexts(ctx)[1], 0))
    close(got, want, 2e-5 if dtype == "float32" else 4e-2, f"lightning attention {case} {how} {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "decoded", "portions"])
@pytest.mark.parametrize("width", [40, 36])
def test_pair_of_mixers(width, how, dtype, tmp_path):
    """Both branches from one product of the input, each with its own state, the mean of their normed outputs."""
    layer = dict(parallel(windowed(3, 1, 10, 6, 0.5, 10.0, 8, 7), memory(2, 12, 9, [0.8, 0.99])), mlp=None)
    rig = Rig([layer], width, dtype, tmp_path, seed=17, page=4, pages=90)
    mixer = rig.model.blocks[0].mixer
    assert mixer.in_proj is not None
    lengths = {"a": 75, "b": 41, "c": 9}
    x = rows_for(lengths, width, 7)
    want = {rid: plain.parallel(x[rid], rig.w, "l0.mix.", layer["mixer"], 1e-5) for rid in x}
    got = rig.run(x, {rid: PLANS[how](n) for rid, n in lengths.items()}, lambda rows, ctx: mixer.forward(rows, ctx, 0))
    close(got, want, 2e-5 if dtype == "float32" else 5e-2, f"pair {how} {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("channel", [False, True])
def test_delta_rule_keeps_and_overwrites_over_hundreds_of_tokens(channel, tmp_path):
    """Heads that all but never forget: what the first hundreds of tokens wrote is still there after 400 tokens decoded one by
    one, unless a later token with the same key has overwritten it (a step size near one)."""
    layer = dict(delta(2, 2, 16, 8, 2, channel=channel), mlp=None)

    def edit(t):
        t["l0.mix.A_log"] = torch.tensor([-7.0, -6.0]).to(torch.bfloat16)
        t["l0.mix.dt_bias"].fill_(-3.0)
        t["l0.mix.b"] *= 0.3

    rig = Rig([layer], 24, "float32", tmp_path, seed=13, page=8, pages=70, edit=edit)
    mixer = rig.model.blocks[0].mixer
    m = rig.config["layers"][0]["mixer"]
    x = rows_for({"a": 420}, 24, 17)
    x["a"][300:] *= 1e-3                       # after the first 300 tokens only what they left is read
    want = plain.delta(x["a"], rig.w, "l0.mix.", m, 1e-5, channel)
    # the control: what came more than a hundred tokens ago still carries the last row
    short = x["a"].clone()
    short[:300] *= 1e-3
    assert (plain.delta(short, rig.w, "l0.mix.", m, 1e-5, channel)[-1] - want[-1]).abs().max() > 0.1 * want[-1].abs().max()
    for plan in ([(0, 20)] + [(i, i + 1) for i in range(20, 420)], [(0, 420)], cuts_of(420, (64, 2, 31, 2, 2))):
        got = rig.run(x, {"a": plan}, lambda rows, ctx: mixer.forward(rows, ctx, 0))
        close(got, {"a": want}, 1e-4, "slow head")


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
        compare(got, want, (TOL_F32 if dtype == "float32" else TOL_BF16)[name], f"{name} {dtype} {mode}")
        results[mode] = got
    if dtype == "float32":
        for mode in ("tail", "portions", "mixed"):
            compare(results[mode], results["whole"], TOL_F32_SAME[name], f"{name} {dtype} {mode} vs whole")


def random_config(seed: int, wide: bool = False) -> tuple[dict, int, tuple]:
    """A configuration drawn from everything the design lets vary, a page size, and the sizes only the tensors give. ``wide``:
    among the sizes the tensor-core kernels take in bfloat16, mixed with sizes they do not."""
    import random

    rng = random.Random(seed + (1000 if wide else 0))
    pick = rng.choice
    width = pick([128, 192, 256]) if wide else pick([16, 24, 30, 40, 64])
    layers = []
    for i in range(rng.randint(3, 5) if wide else rng.randint(1, 6)):
        owners = [j for j, e in enumerate(layers) if "weights_of" not in e]
        if owners and rng.random() < 0.25:
            j = pick(owners)
            layers.append(dict(layers[j], weights_of=j))
            continue
        kind = pick(["delta", "channel_delta", "parallel"])
        kv = pick([1, 2, 3])
        if kind == "parallel":
            dims = [32, 48, 64, 96, 128] if wide else [4, 8, 10, 16, 24]
            left = windowed(kv * pick([1, 2, 4]), kv, pick(dims), pick(dims), pick([0.1, 0.2, 0.4]), pick([8.0, 20.0, 60.0]),
                            pick([20, 70, 300]), pick([16, 63, 64, 65, 130, 200]) if wide else pick([1, 2, 7, 33, 64, 1000]))
            heads = pick([1, 2, 4])
            layer = parallel(left, memory(heads, pick(dims), pick(dims), [pick([0.3, 0.9, 0.99, 0.999]) for _ in range(heads)]))
        else:
            dims = [32, 64, 128, 48] if wide else [4, 6, 8, 16, 40]
            layer = delta(kv * pick([1, 2]), kv, pick(dims), pick(dims), pick([1, 2, 3, 4, 7]), channel=kind == "channel_delta")
        layer["mlp"] = None if rng.random() < 0.2 else dense(pick([128, 384]) if wide else pick([8, 20, 64]))
        layers.append(layer)
    config = model(rng.randint(40, 300), width, layers, pick([1e-5, 1e-6]), pick([0.2, 0.5, 1.0]), pick([1.0, 3.0, 7.5]))
    return config, 16 if wide else pick([4, 8, 16]), (pick([1, 5, 16]), pick([2, 8, 11]), pick([2, 6, 16, 32]))


@pytest.mark.gpu
@pytest.mark.parametrize("wide", [False, True])
@pytest.mark.parametrize("seed", range(10))
def test_random_configurations(seed, wide, tmp_path):
    """Configurations nobody chose: whatever the draw gives, the 32-bit model meets the plain implementation however the requests
    are cut, and the 16-bit one stays close to it."""
    config, page, free = random_config(seed, wide)
    tensors = make_tensors(config, 300 + seed, free)
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
            compare(trace_util.collect(steps, per_step), want, tol, f"random configuration {seed} {dtype}: {config}")


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
    """One and two token prompts, and 300 tokens decoded one by one: across many pages, past the window, the recurrent states
    carried all the way."""
    for name in ("A", "D"):
        folder, w = folders[name]
        g = torch.Generator().manual_seed(99)
        vocab = CASES[name]["config"]["vocab"]
        reqs = {"one": torch.randint(0, vocab, (1,), generator=g).tolist(),
                "two": torch.randint(0, vocab, (2,), generator=g).tolist(),
                "long": torch.randint(0, vocab, (303,), generator=g).tolist()}
        want = {rid: plain.forward(CASES[name]["config"], w, ids)[0] for rid, ids in reqs.items()}
        steps = trace_util.tail_decoded(reqs, tail=300)
        page = CASES[name]["page"]
        per_step = trace_util.run_in_process(folder, dtype, steps, trace_util.max_live_tokens(steps, page), page,
                                             max_requests=4)
        compare(trace_util.collect(steps, per_step), want, (TOL_F32 if dtype == "float32" else TOL_BF16)[name],
                f"long decoding {name} {dtype}")


def test_a_changed_design_shows_in_the_plain_implementation(folders, monkeypatch):
    """Negative controls, planted in the plain implementation: a window one longer, the cap left out, the bias's last row
    reached too early, a read-out before the write, a decay of another head, unit lengths left out, the factor on the
    residual left out, and a layer that reads the state of the layer whose weights it uses all move the logits far
    beyond the bound that the engine meets."""
    name = "A"
    config, w = CASES[name]["config"], folders[name][1]
    ids = requests_for(name)["r4"]
    want = plain.forward(config, w, ids)[0]

    def moved(cfg=config, weights=w):
        got = plain.forward(cfg, weights, ids)[0]
        return ((got - want).abs().max() / want.abs().max()).item() / TOL_F32[name]

    def changed(edit):
        c = json.loads(json.dumps(config))
        edit(c)
        return c

    def both(key, value):
        def edit(c):
            for i in (1, 4):
                c["layers"][i]["mixer"]["left"][key] = value
        return edit

    assert moved() == 0
    assert moved(changed(both("mask", {"size": 12}))) > 100
    assert moved(changed(both("softcap", 1e6))) > 100
    assert moved(changed(both("bias_max", 5))) > 100
    assert moved(changed(lambda c: c.update(residual_mult=1.0))) > 100
    assert moved(changed(lambda c: [c["layers"][i]["mixer"]["right"].update(decay=[0.9, 0.5, 0.995]) for i in (1, 4)])) > 100
    monkeypatch.setattr(plain, "unit", lambda x: x)
    assert moved() > 100
    monkeypatch.undo()
    real = plain.delta_scan

    def early(q, k, v, g, beta):
        out = torch.zeros_like(v)
        for h in range(q.shape[1]):
            S = torch.zeros(q.shape[2], v.shape[2], dtype=torch.float64)
            for t in range(q.shape[0]):
                S = g[t, h][:, None] * S
                out[t, h] = S.T @ q[t, h]
                S = S + torch.outer(k[t, h], beta[t, h] * (v[t, h] - S.T @ k[t, h]))
        return out
    monkeypatch.setattr(plain, "delta_scan", early)
    assert moved() > 100
    monkeypatch.undo()
    monkeypatch.setattr(plain, "delta_scan", lambda q, k, v, g, beta: real(q, k, v, g.flip(1), beta))
    assert moved() > 100


@pytest.mark.gpu
def test_a_lost_state_shows(folders, monkeypatch):
    """The same replay without the convolution's state, or without the recurrent states, is far outside the bound that the real
    model meets (every index stays in bounds: the portions start from zeros)."""
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

    assert worst() <= TOL_F32[name]
    real_conv = ops.seq_conv
    monkeypatch.setattr(ops, "seq_conv", lambda u, taps, bias, state, cu, ctx, *rest, **kw: real_conv(
        u, taps, bias, state, cu, torch.zeros_like(ctx), *rest, **kw))
    assert worst() > 100 * TOL_F32[name]
    monkeypatch.undo()
    real_scan = ops.linmem_scan

    def forgetful(*args, **kw):
        args = list(args)
        args[7] = torch.zeros_like(args[7])              # seq_ctx: every portion starts from zero
        return real_scan(*args, **kw)
    monkeypatch.setattr(ops, "linmem_scan", forgetful)
    assert worst() > 100 * TOL_F32[name]


# ---------------------------------------------------------------------------------------------
# the entry points: LLM.generate through the scheduler, the command line, the trace program
# ---------------------------------------------------------------------------------------------

def teacher_forced_ok(config, w, prompt, reply, margin):
    """Every token of ``reply`` is the plain implementation's best, or within ``margin`` of it."""
    logits, _ = plain.forward(config, w, prompt + reply)
    for i, tok in enumerate(reply):
        row = logits[len(prompt) + i - 1]
        assert int(row.argmax()) == tok or row.max().item() - row[tok].item() <= margin, (i, tok)


@pytest.mark.gpu
@pytest.mark.parametrize("name, work, graphs", [("A", "fp32", False), ("B", "fp32", True), ("D", "bf16", True),
                                                ("C", "fp32", True), ("D", "fp32", False), ("A", "bf16", True)])
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
        teacher_forced_ok(config, w, prompt, out.token_ids, 1e-3 if work == "fp32" else 0.3)


@pytest.mark.gpu
def test_trace_program_and_command_line(folders, tmp_path):
    name = "A"
    folder, _ = folders[name]
    reqs = requests_for(name)
    want = oracle(name, folders, reqs)
    steps = trace_util.mixed(reqs, live=4, seed=3)
    per_step = trace_util.run_program(folder, "float32", steps, trace_util.max_live_tokens(steps, 64), tmp_path,
                                      CASES[name]["config"]["vocab"])
    compare(trace_util.collect(steps, per_step), want, TOL_F32[name], "trace program")
    cmd = [sys.executable, "-m", "tokenomos_b200.generate", "--model", str(folder), "--prompt-ids", "1,2,3,4",
           "--max-tokens", "5", "--arch-kw", '{"work": "fp32"}',
           "--engine-kw", '{"page": 4, "max_len": 64, "slots": 2, "pages": 40}']
    proc = subprocess.run(cmd, capture_output=True, text=True, cwd=ROOT, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [json.loads(ln) for ln in proc.stdout.splitlines() if ln.startswith("{")]
    assert len(lines) == 1 and len(lines[0]["token_ids"]) == 5
    teacher_forced_ok(CASES[name]["config"], folders[name][1], [1, 2, 3, 4], lines[0]["token_ids"], 1e-3)
