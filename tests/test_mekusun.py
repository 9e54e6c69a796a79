"""The Mekusun decoder in the engine against the plain implementation (``plain_mekusun``).

Every test that needs a kernel set takes the fixture ``kit``: the plain tensor-op set on the CPU
(``ref_kernels.RefKernels``, which checks the engine's bookkeeping: cache, state slots, batching, scheduling), and
under ``-m gpu`` the CUDA sets in float32 and bfloat16.  Configurations are made here, with random weights; they
differ from one another in every size.
"""

from __future__ import annotations

import copy
import math

import pytest
import torch

import helpers
import plain_mekusun as pm
from ref_kernels import RefKernels

from distie_b200.cache.manager import pages_needed
from distie_b200.config import ConfigError, EngineConfig, MekusunConfig, PartSpec, get_architecture
from distie_b200.engine.batch import BatchEntry, lay_out, views
from distie_b200.engine.engine import Engine, GenerateRequest
from distie_b200.engine.trace_replay import TraceSession
from distie_b200.kernels.interface import Averaged, KvSlot, Normed, RotaryTable, Terms
from distie_b200.models.decoder import model_tensor_specs
from distie_b200.parts import NORMS, BuildContext, ResidualStream
from distie_b200.weights import WeightsError, open_weights


def _mamba(inner, state, dt_rank, conv, mlp):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}, "mlp": mlp}


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, mlp, dims=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim if dims is None else dims}}}


def _delta(heads, dim, mlp):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def _config(vocab, width, eps, scale, cap, layers):
    return {"architecture": "Mekusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_softcap": cap, "layers": layers}


# Small: every branch once; pages of four; the delta layers' decay projections have different ranks.
SMALL = _config(96, 48, 1e-5, 5.0, 9.0, [
    _mamba(40, 6, 4, 4, _moe(5, 2, 16)),
    _latent(3, 8, 4, 6, 20, 0.4, 1000.0, _dense(40)),
    _delta(2, 12, _moe(4, 3, 24)),
    _latent(2, 12, 6, 10, 16, 0.3, 50.0, None),
])
# Awkward: sizes that are no multiples of four, single heads, a single state and more states than 16 and 32, one tap and
# five, a rotation of a part of the rotated dimensions, as many chosen experts as there are, one expert, layers without
# a feed-forward in the middle, a scale of one on the embedding, a cap that bends every logit.
AWKWARD = _config(101, 70, 1e-6, 1.0, 2.5, [
    _delta(3, 7, None),
    _mamba(50, 21, 7, 1, _dense(45)),
    _mamba(33, 1, 1, 5, _moe(3, 3, 10)),
    _latent(1, 10, 8, 5, 33, 0.25, 100.0, _moe(1, 1, 22), 6),
    _delta(1, 33, _moe(6, 1, 18)),
    _mamba(18, 40, 3, 2, None),
])
# Sizes of a real model's order: in bfloat16 the tensor-core products, latent attention and grouped experts run.
WIDE = _config(500, 256, 1e-5, 2.0, 20.0, [
    _mamba(512, 16, 16, 4, _moe(8, 2, 64)),
    _delta(2, 64, _dense(384)),
    _latent(4, 64, 32, 64, 128, 0.1, 10000.0, _moe(16, 4, 32)),
    _delta(1, 128, _moe(8, 2, 128)),
    _latent(16, 32, 16, 32, 64, 0.14, 500.0, _dense(200)),
])
RANKS = {"small": 8, "awkward": {0: 5, 4: 12}, "wide": 16}
CONFIGS = {"small": (SMALL, 4, 0), "awkward": (AWKWARD, 4, 1), "wide": (WIDE, 16, 2)}

FP32_TOL = 1e-4    # rms over the vocabulary of the logits' difference, mean taken off, over the logit scale
BF16_TOL = 6e-2

KITS = ["cpu", pytest.param("gpu32", marks=pytest.mark.gpu), pytest.param("gpu16", marks=pytest.mark.gpu)]
ORACLE = {"stored": None}  # the type whose roundings the plain implementation takes on for the kit in use


@pytest.fixture(params=KITS)
def kit(request):
    ORACLE["stored"] = torch.bfloat16 if request.param == "gpu16" else None
    if request.param == "cpu":
        return RefKernels(torch.float32, "cpu")
    from distie_b200.kernels import make_kernels

    return make_kernels(torch.float32 if request.param == "gpu32" else torch.bfloat16, "cuda:0")


def tolerance(kit) -> float:
    return FP32_TOL if kit.dtype == torch.float32 else BF16_TOL


def every_expert(cfg: dict) -> dict:
    """``cfg`` with every router choosing all of its experts: the weights still vary with the token, but no choice can
    be turned around by rounding."""
    out = copy.deepcopy(cfg)
    for layer in out["layers"]:
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out


def model(name: str, kit=None):
    """The configuration, its page size and random weights.  For the bfloat16 engine the routers choose every expert (a
    choice that hangs on less than 16-bit activations can tell apart changes every later token through the
    recurrences); the float32 engines run the choices everywhere, and ``test_clear_choices_in_sixteen_bits`` runs them
    in bfloat16 where they are clear."""
    cfg, page, seed = CONFIGS[name]
    cfg = every_expert(cfg) if kit is not None and kit.dtype != torch.float32 else copy.deepcopy(cfg)
    return cfg, page, pm.random_weights(cfg, seed, RANKS[name])


def engine_of(cfg, weights, page, kit, num_blocks: int, max_seqs: int = 4, **knobs):
    arch = get_architecture(cfg["architecture"])
    dtype = "float32" if kit.dtype == torch.float32 else "bfloat16"
    config = EngineConfig(num_blocks=num_blocks, page_size=page, max_seqs=max_seqs, dtype=dtype, device=str(kit.device),
                          decode_graphs=kit.device.type == "cuda", **{"token_budget": 4096, **knobs})
    stored = {k: v.to(torch.bfloat16) for k, v in weights.items()}
    return Engine.assemble(arch, arch.config_cls.from_dict(cfg), stored, kit, config)


def engine_for(name: str, kit, num_blocks: int, max_seqs: int = 4, **knobs):
    cfg, page, weights = model(name, kit)
    return engine_of(cfg, weights, page, kit, num_blocks, max_seqs, **knobs), cfg, weights


def plain_logits(cfg, weights, ids, margins=None, trace=None) -> torch.Tensor:
    """The oracle: the plain implementation in float64; for the bfloat16 engine with that type's roundings where an
    engine stores 16 bits between two products (and nowhere else)."""
    with pm.stored_as(ORACLE["stored"]):
        return pm.forward(cfg, weights, ids, torch.float64, trace=trace, margins=margins).float()


def row_errors(have: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    diff = have.double() - want.double()
    diff = diff - diff.mean(-1, keepdim=True)
    return diff.pow(2).mean(-1).sqrt() / float(want.double().std())


def assert_close(got: dict, expected: dict, tol: float, what: str) -> None:
    expected = helpers.expected_for(got, expected)
    for rid, want in expected.items():
        errors = row_errors(got[rid], want)
        at = int(errors.argmax())
        assert float(errors[at]) <= tol, f"{what}: request {rid}, position {at}: {float(errors[at]):.3e} of the logit scale"


def requests_of(cfg, lengths, seed=20):
    return {f"r{i}": helpers.random_ids(cfg["vocab"], n, seed + i) for i, n in enumerate(lengths)}


def step_for(kit, entries):
    layout = lay_out([BatchEntry(*e) for e in entries])
    return views(torch.from_numpy(layout.packed).to(kit.device), layout)[0], layout


def in_slices(x: torch.Tensor) -> torch.Tensor:
    """``x`` as three slices ``[3, T, n]`` whose sum it is exactly, as a split product leaves it."""
    return torch.stack([x * 0.5, x * 0.25, x * 0.25])


def _close(have, want, tol, what):
    scale = float(want.double().abs().max()) or 1.0
    err = float((have.double().cpu() - want.double()).abs().max()) / scale
    assert err <= tol, f"{what}: {err:.3e} of the largest value"


# -- configuration and weights -----------------------------------------------------------------------------
def test_config_reads_every_size_and_names_what_is_missing():
    cfg = MekusunConfig.from_dict(AWKWARD)
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.embedding_scale, cfg.logit_softcap, len(cfg.layers)) == (101, 70, 1e-6, 1.0, 2.5, 6)
    scan = cfg.layers[1].mixer
    assert (scan.inner, scan.state, scan.dt_rank, scan.conv) == (50, 21, 7, 1) and cfg.layers[1].mlp.ff == 45
    latent = cfg.layers[3].mixer
    assert (latent.heads, latent.dim, latent.rot_dim, latent.vdim, latent.kv_rank, latent.scale) == (1, 10, 8, 5, 33, 0.25)
    assert (latent.rot_base, latent.rot_dims) == (100.0, 6)
    assert (cfg.layers[4].mixer.heads, cfg.layers[4].mixer.dim) == (1, 33)
    assert (cfg.layers[4].mlp.experts, cfg.layers[4].mlp.top, cfg.layers[4].mlp.ff) == (6, 1, 18)
    assert cfg.layers[0].mlp is None and cfg.layers[5].mlp is None
    for path, match in (
        (("layers", 0, "mixer", "dt_rank"), r"layers\[0\]\.mixer\.dt_rank"),
        (("layers", 0, "mixer", "conv"), r"layers\[0\]\.mixer\.conv"),
        (("layers", 1, "mixer", "kv_rank"), r"layers\[1\]\.mixer\.kv_rank"),
        (("layers", 1, "mixer", "rot", "base"), r"layers\[1\]\.mixer\.rot\.base"),
        (("layers", 2, "mixer", "heads"), r"layers\[2\]\.mixer\.heads"),
        (("layers", 0, "mlp", "router", "top"), r"layers\[0\]\.mlp\.router\.top"),
        (("layers", 0, "mlp", "expert"), r"layers\[0\]\.mlp\.expert"),
        (("norm",), "norm"),
        (("embedding", "scale"), r"embedding\.scale"),
        (("logit_softcap",), "logit_softcap"),
        (("width",), "width"),
    ):
        broken = copy.deepcopy(SMALL)
        at = broken
        for key in path[:-1]:
            at = at[key]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=match):
            MekusunConfig.from_dict(broken)
    for change, match in (
        (lambda c: c["layers"][0].update(type="mamba2"), "mamba2"),
        (lambda c: c["layers"][1]["mlp"].update(kind="swiglu"), "swiglu"),
        (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), "dims"),
        (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
        (lambda c: c["layers"][2]["mixer"].update(dim=0), "dim"),
        (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    ):
        broken = copy.deepcopy(SMALL)
        change(broken)
        with pytest.raises(ConfigError, match=match):
            MekusunConfig.from_dict(broken)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    cfg = CONFIGS[name][0]
    arch = get_architecture("Mekusun")
    specs = model_tensor_specs(arch.recipe(arch.config_cls.from_dict(cfg)))
    ranks = {i: next(s.default_shape[0] for s in specs if s.name == f"l{i}.mix.w1")
             for i, layer in enumerate(cfg["layers"]) if layer["type"] == "general_delta"}
    assert {s.name: s.default_shape for s in specs} == {k: tuple(v) for k, v in pm.tensor_shapes(cfg, ranks).items()}


def test_a_size_that_only_the_checkpoint_gives():
    """The rank of the decay projection differs between the layers of one model and is in no configuration: any rank
    loads, as long as the two matrices of a layer agree on it."""
    cfg, page, weights = model("awkward")
    arch = get_architecture("Mekusun")
    spec = arch.recipe(arch.config_cls.from_dict(cfg))
    assert weights["l0.mix.w1"].shape == (5, 70) and weights["l4.mix.w2"].shape == (33, 12)
    open_weights(weights, model_tensor_specs(spec), spec.tolerated, torch.float32, "cpu")
    broken = dict(weights)
    broken["l4.mix.w2"] = torch.zeros(33, 11)
    with pytest.raises(WeightsError, match=r"l4\.mix\.w2: checkpoint \(33, 11\), model \(33, 12\)"):
        open_weights(broken, model_tensor_specs(spec), spec.tolerated, torch.float32, "cpu")
    # a layer without a feed-forward may carry the norms of one
    broken = dict(weights)
    broken["l0.norm2"] = broken["l0.ls2"] = torch.zeros(70)
    open_weights(broken, model_tensor_specs(spec), spec.tolerated, torch.float32, "cpu")


def test_random_model_folder_loads_by_its_config(tmp_path):
    from distie_b200.config import read_config
    from distie_b200.weights import write_random_model

    folder = write_random_model(str(tmp_path / "m"), SMALL, seed=3, std=0.1, norm_noise=0.05)
    arch, cfg = read_config(folder)
    assert arch.name == "Mekusun" and cfg.width == 48
    engine = Engine.assemble(arch, cfg, folder, RefKernels(torch.float32),
                             EngineConfig(num_blocks=8, page_size=16, max_seqs=2, dtype="float32", device="cpu", decode_graphs=False))
    out = engine.generate([[1, 2, 3]], max_new_tokens=3, ignore_eos=True)
    assert len(out[0].token_ids) == 3


# -- each mechanism alone: ops of the kernel set against the plain functions ------------------------------------
@pytest.mark.parametrize("width", [72, 201, 2304])
@pytest.mark.parametrize("count", [1, 4, 11])
def test_average_over_depth_between_two_norms(kit, width, count):
    """The layer's own result (residual + a normed sum of terms) joins the states, the residual becomes the weighted sum
    of them all, and its norm comes out; rows alone leave everything as it was; the last state of a model is not kept."""
    g = torch.Generator().manual_seed(width + count)
    tokens, dev = 9, kit.device
    residual = torch.randn(tokens, width, generator=g) * 2
    past = torch.randn(count, tokens, width, generator=g)
    mix = torch.randn(count + 1, generator=g)
    a, b = torch.randn(2, tokens, width, generator=g), torch.randn(tokens, width, generator=g) * 3
    w_delta, w_out = 1 + torch.randn(width, generator=g) * 0.2, 1 + torch.randn(width, generator=g) * 0.2
    own = residual.double() + pm.rms_unit(a.double().sum(0) + 0.5 * b.double(), 1e-5) * w_delta.double()
    average = pm.depth_average([*past.double(), own], mix.double())
    want = pm.rms_unit(average, 1e-6) * w_out.double()
    tol = 1e-5 if kit.dtype == torch.float32 else 2e-2
    for slots in (count + 2, count):
        history = torch.full((slots, tokens, width), float("nan"))
        history[:count] = past
        history = history.to(dev)
        value = Normed(Terms([(a.to(dev), 1.0), (b.to(dev), 0.5)]), w_delta.to(dev), 1e-5)
        ahead = Averaged(value, history, count, mix.to(dev))
        res, rows = residual.clone().to(dev), torch.tensor([4, 1], dtype=torch.int32, device=dev)
        picked = torch.empty(2, width, dtype=kit.dtype, device=dev)
        kit.average_add_rmsnorm(ahead, res, w_out.to(dev), 1e-6, picked, rows)
        _close(picked, want[[4, 1]], tol, "picked rows")
        assert torch.equal(res.cpu(), residual) and torch.equal(history[:count].cpu(), past)
        out = torch.empty(tokens, width, dtype=kit.dtype, device=dev)
        kit.average_add_rmsnorm(ahead, res, w_out.to(dev), 1e-6, out)
        _close(res, average, 3e-6, "average")
        _close(out, want, tol, "norm")
        assert torch.equal(history[:count].cpu(), past)
        if slots > count:
            _close(history[count], own, 3e-6, "the layer's own result")
    # a plain sum pending, nothing pending, and no norm behind it
    for value, result in ((b.to(dev), residual.double() + b.double()), (None, residual.double())):
        history = torch.zeros(count + 1, tokens, width)
        history[:count] = past
        res = residual.clone().to(dev)
        ahead = Averaged(value, history.to(dev), count, mix.to(dev))
        kit.average_add_rmsnorm(ahead, res, None, 0.0, None)
        _close(res, pm.depth_average([*past.double(), result], mix.double()), 3e-6, "average alone")
        stream = ResidualStream(residual.clone().to(dev), ahead)
        _close(stream.settle(), pm.depth_average([*past.double(), result], mix.double()), 3e-6, "settled")


def test_a_layer_scale_rides_the_norm_of_a_sublayers_output(kit):
    g = torch.Generator().manual_seed(2)
    weights = {"n.w": torch.randn(40, generator=g) * 0.3, "n.scale": torch.randn(40, generator=g)}
    spec = PartSpec("rmsnorm", {"eps": 1e-5, "name": "w", "offset": 1.0, "times": "scale"}, "n.")
    cls = NORMS.get("rmsnorm")
    specs = cls.tensor_specs(spec, 40)
    assert [s.name for s in specs] == ["n.w", "n.scale"]
    norm = cls.build(spec, BuildContext(kit, 40, open_weights(weights, specs, (), kit.dtype, kit.device)))
    delta, residual = torch.randn(6, 40, generator=g) * 2, torch.randn(6, 40, generator=g)
    stream = ResidualStream(residual.clone().to(kit.device), norm.pending(delta.to(kit.device)))
    want = residual.double() + pm.zero_centred_norm(delta.double(), weights["n.w"].double(), 1e-5) * weights["n.scale"].double()
    _close(stream.settle(), want, 2e-6, "scaled norm")


@pytest.mark.parametrize("channels,taps", [(36, 4), (50, 1), (33, 5), (256, 3), (512, 4)])
def test_convolution_also_in_the_engines_type(kit, channels, taps):
    g = torch.Generator().manual_seed(channels)
    n = 21
    x, bias, weight = torch.randn(n, channels + 8, generator=g), torch.randn(channels, generator=g), torch.randn(channels, taps, generator=g)
    want = pm.silu(pm.causal_conv(x[:, :channels].double(), weight.double(), bias.double()))
    dev = kit.device
    for cuts in ([n], [1, 2, 9, 1, 1, 7]):
        state = torch.zeros(2, taps - 1, channels, device=dev) if taps > 1 else None
        got, at = [], 0
        for count in cuts:
            step, _ = step_for(kit, [(1, [0] * count, at, ())])
            wide, narrow = kit.short_conv(in_slices(x[at : at + count]).to(dev)[..., :channels], weight.to(dev), bias.to(dev), state,
                                          step, "silu", typed=True)
            assert narrow.dtype == kit.dtype and torch.equal(narrow, wide.to(kit.dtype))
            got.append(wide.cpu())
            at += count
        _close(torch.cat(got), want, 2e-5, "convolution")


def _walk(kit, lengths, portions, run):
    """``run(seat -> (first, count) list in step order, step)`` over portions of several requests side by side; returns
    the rows each seat got."""
    done = {seat: 0 for seat in lengths}
    got = {seat: [] for seat in lengths}
    portions = {seat: list(p) for seat, p in portions.items()}
    while any(portions.values()):
        entries, order = [], []
        for seat in sorted(portions, key=lambda s: (portions[s][0] if portions[s] else 0) != 1):  # single tokens first
            if portions[seat]:
                count = portions[seat].pop(0)
                entries.append((seat, [0] * count, done[seat], ()))
                order.append((seat, done[seat], count))
                done[seat] += count
        step, _ = step_for(kit, entries)
        out = run(order, step).float().cpu()
        at = 0
        for seat, _, count in order:
            got[seat].append(out[at : at + count])
            at += count
    assert done == lengths
    return {seat: torch.cat(rows) for seat, rows in got.items()}


@pytest.mark.parametrize("channels,states,length", [(36, 5, 40), (9, 1, 25), (64, 16, 60), (130, 16, 700), (50, 24, 45), (40, 24, 530),
                                                    (40, 33, 30), (18, 64, 420), (16, 100, 20), (257, 200, 12)])
def test_selective_scan_in_portions(kit, channels, states, length):
    """Two requests side by side, whole and in portions down to single tokens; rates of decay from a memory of thousands
    of tokens to none; the first token of each request is large, so that it still shows at the end."""
    if kit.device.type == "cpu" and length > 100:
        pytest.skip("long walks run on the GPU only")
    g = torch.Generator().manual_seed(channels + states)
    lengths = {2: length, 1: 9}
    rank = 6
    data = {}
    for seat, n in lengths.items():
        data[seat] = {"x": torch.randn(n, channels, generator=g), "dt": torch.randn(n, channels, generator=g),
                      "bc": torch.randn(n, rank + 2 * states, generator=g), "z": torch.randn(n, channels, generator=g)}
        data[seat]["x"][0] *= 30.0
    rates = -torch.exp(torch.rand(states, channels, generator=g) * 9 - 7)
    skip, bias = torch.randn(channels, generator=g), torch.randn(channels, generator=g) - 1
    want = {}
    for seat, d in data.items():
        e = {k: v.double() for k, v in d.items()}
        y = pm.selective_scan(e["x"], pm.softplus(e["dt"] + bias.double()), e["bc"][:, rank : rank + states], e["bc"][:, rank + states :],
                              rates.double().T, skip.double())
        want[seat] = y * pm.silu(e["z"])
    dev = kit.device
    cuts = [1, 2, 1, 1, 5]
    portioned = {2: cuts + [length - 10 - 3, 1, 2] if length <= 60 else [1, 2, length - 140, 130, 1, 1, 5], 1: [2, 1, 1, 4, 1]}
    for portions in ({2: [length], 1: [9]}, {2: [p for p in portioned[2] if p > 0], 1: portioned[1]}):
        portions[2][-1] += length - sum(portions[2])
        state = torch.zeros(4, states, channels, device=dev)
        untouched = torch.randn(states, channels, generator=g)
        state[3] = untouched.to(dev)

        def run(order, step):
            rows = {k: torch.cat([data[s][k][a : a + c] for s, a, c in order]) for k in ("x", "dt", "bc", "z")}
            bc, dt, z = (in_slices(rows[k]).to(dev) for k in ("bc", "dt", "z"))
            out = torch.empty(rows["x"].shape, dtype=kit.dtype, device=dev)
            kit.selective_scan(rows["x"].to(dev), dt, bc[:, :, rank : rank + states], bc[:, :, rank + states :], z, rates.to(dev),
                               skip.to(dev), bias.to(dev), state, step, out)
            return out

        got = _walk(kit, lengths, portions, run)
        for seat in lengths:
            _close(got[seat], want[seat], 1e-5 if kit.dtype == torch.float32 else 1e-2, f"seat {seat}, portions {portions[seat]}")
            tail = slice(lengths[seat] // 2, None)  # the first tokens are large: the rest on a scale of its own
            _close(got[seat][tail], want[seat][tail], 2e-5 if kit.dtype == torch.float32 else 1e-2, f"seat {seat}, second half")
        assert torch.equal(state[3].cpu(), untouched) and float(state[0].abs().max()) == 0
    if kit.device.type == "cuda" and length > 400:
        assert kit.kernel_counts.get("selective_scan_tiled"), "a long portion of few channels is cut into tiles"


@pytest.mark.parametrize("heads,dim,length", [(2, 12, 30), (3, 7, 26), (1, 32, 40), (1, 33, 24), (5, 16, 20), (2, 64, 150), (1, 128, 70),
                                              (1, 100, 24), (2, 200, 14), (1, 256, 20)])
def test_channel_delta_in_portions(kit, heads, dim, length):
    """Two requests side by side, whole and in portions down to single tokens.  A key that is zero (whose unit key is
    zero, not undefined), a strong early key read back late by a query along it, removal and decay between their
    extremes per channel."""
    g = torch.Generator().manual_seed(heads + dim)
    n = heads * dim
    lengths = {2: length, 1: 7}
    data = {}
    for seat, t in lengths.items():
        proj = torch.randn(t, 4 * n + 3, generator=g)
        proj[:, n : 2 * n] /= math.sqrt(dim)
        proj[:, 3 * n : 4 * n] *= 2
        proj[2, n : 2 * n] = 0.0
        proj[1, n : 2 * n] *= 8.0
        proj[t - 2, :n] = proj[1, n : 2 * n]
        data[seat] = {"proj": proj, "decay": torch.randn(t, n, generator=g) * 3}
    w0, a_bias = torch.randn(n, generator=g) * 2 - 4, torch.randn(n, generator=g) - 1
    want = {}
    for seat, d in data.items():
        t = lengths[seat]
        p = d["proj"].double()
        r, k, v = (p[:, i * n : (i + 1) * n].reshape(t, heads, dim) for i in range(3))
        decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(d["decay"].double() + w0.double())).reshape(t, heads, dim)
        rate = torch.sigmoid(p[:, 3 * n : 4 * n] + a_bias.double()).reshape(t, heads, dim)
        want[seat] = pm.delta_rule(r, k, v, decay, rate).reshape(t, n)
    dev = kit.device
    portioned = [1, 2, 1, 1, 5]
    for portions in ({2: [length], 1: [7]}, {2: portioned + [length - 13, 1, 2], 1: [2, 1, 1, 3]}):
        state = torch.zeros(4, heads, dim, dim, device=dev)
        state[3] = 1.0

        def run(order, step):
            proj, decay = (torch.cat([data[s][k][a : a + c] for s, a, c in order]) for k in ("proj", "decay"))
            return kit.channel_delta(in_slices(proj).to(dev)[..., : 4 * n], in_slices(decay).to(dev), w0.to(dev), a_bias.to(dev), state, step,
                                     heads, dim)

        got = _walk(kit, lengths, portions, run)
        for seat in lengths:
            _close(got[seat], want[seat], 2e-5, f"seat {seat}, portions {portions[seat]}")
        assert bool((state[3] == 1.0).all()) and float(state[0].abs().max()) == 0


def _latent_slot(kit, row, rank, pages, page_size, table):
    dev = kit.device
    k = torch.zeros(pages, 1, page_size, row, dtype=kit.dtype, device=dev)
    return KvSlot(k, k[..., :rank], torch.tensor(table, dtype=torch.int32, device=dev), page_size, pages)


@pytest.mark.parametrize("heads,dim,rot,dims,vdim,rank,page,n", [(3, 8, 4, 4, 6, 20, 4, 61), (1, 10, 8, 6, 5, 33, 4, 50),
                                                                (4, 64, 32, 32, 64, 128, 16, 200), (16, 32, 16, 16, 32, 64, 8, 150)])
def test_attention_through_a_latent_with_keys_that_stand_out(kit, heads, dim, rot, dims, vdim, rank, page, n):
    """From the stacked projection (queries straight from it, no query latent) through pages handed out in reverse, in
    portions and token by token.  The very first row, rows on either side of page borders and every seventh carry a
    direction that every query looks for, with strengths of their own: one far key among hundreds decides most of an
    output."""
    g = torch.Generator().manual_seed(rank + n)
    eps, base, scale = 1e-5, 100.0, 0.6
    columns = heads * (dim + rot)
    up_k, up_v = torch.randn(heads, dim, rank, generator=g) / math.sqrt(rank), torch.randn(heads, rank, vdim, generator=g) / math.sqrt(rank)
    a = torch.randn(rank, generator=g)
    a = a / a.norm() * math.sqrt(rank)
    proj = torch.randn(n, columns + rank + rot, generator=g)
    marked = {0: 5.0}
    for border in range(2 * page, n, 2 * page):
        marked[border - 1], marked[border] = 3.0 + border % 3, 4.5 - border % 2
    for j in range(3, n, 7):
        marked.setdefault(j, 1.0 + (j * 5 % 9) * 0.3)
    for j, strength in marked.items():
        proj[j, columns : columns + rank] = strength * a + torch.randn(rank, generator=g)
    q = proj[:, :columns].view(n, heads, dim + rot)
    q[..., :dim] += 2.0 * torch.einsum("hdr,r->hd", up_k, a) / math.sqrt(dim)
    weight = 1 + 0.2 * torch.randn(rank, generator=g)
    if kit.dtype != torch.float32:
        up_k, up_v = up_k.to(torch.bfloat16).float(), up_v.to(torch.bfloat16).float()
    rounded = torch.bfloat16 if kit.dtype != torch.float32 else None
    positions = torch.arange(n)
    with pm.stored_as(rounded):
        d = proj.double()
        down = d[:, columns:]
        c = pm.stored(pm.rms_unit(down[:, :rank], eps) * weight.double())
        part = pm.stored(pm.rotate_half(down[:, None, rank:], positions, base, dims))
        qd = d[:, :columns].view(n, heads, dim + rot)
        q_all = torch.cat([pm.stored(qd[..., :dim]), pm.stored(pm.rotate_half(qd[..., dim:], positions, base, dims))], -1)
        keys = torch.cat([torch.einsum("hdr,tr->thd", up_k.double(), c), part.expand(n, heads, rot)], -1)
        values = torch.einsum("hrv,tr->thv", up_v.double(), c)
        want = pm.causal_softmax_attention(q_all, keys, values, scale).reshape(n, heads * vdim)
    dev = kit.device
    table = RotaryTable((base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)).float().to(dev), dims)
    width = pages_needed(n, page)
    for cuts in ([1, 1, 2, page - 1, 1, 2, 3 * page, 1, 1, 4 * page + 1], [n]):
        kv = _latent_slot(kit, rank + rot, rank, width + 1, page, [[-1] * width, list(range(width - 1, -1, -1))])
        got, at, cuts = [], 0, list(cuts)
        while at < n:
            count = min(cuts.pop(0) if cuts else 1, n - at)
            step, _ = step_for(kit, [(1, [0] * count, at, ())])
            rows = in_slices(proj[at : at + count]).to(dev)
            kit.latent_kv_write(rows[..., columns:], step, kv, table, 0, None, rank, weight.to(dev), rot, eps, None)
            folded, rotated = kit.latent_queries(rows[..., :columns], up_k.to(dev, kit.dtype), step, table, heads, dim, rot)
            mixed = torch.empty(heads, count, rank, dtype=kit.dtype, device=dev)
            kit.latent_attention(folded, rotated, step, kv, heads, rank, rot, scale, None, mixed)
            got.append(kit.latent_values(mixed, up_v.to(dev, kit.dtype), None, heads, vdim).float().cpu())
            at += count
        kit.check_errors()
        _close(torch.cat(got), want, 2e-5 if kit.dtype == torch.float32 else 3e-2, "latent attention")


@pytest.mark.parametrize("kind,numbers", [("xielu", (0.7, 1.3)), ("xielu", (2.1, 0.55)), ("gelu", None), ("relu2", None)])
@pytest.mark.parametrize("tokens,width,ff", [(5, 48, 40), (40, 70, 45), (70, 64, 200), (300, 256, 384), (130, 128, 96)])
def test_activations_on_a_products_accumulators(kit, kind, numbers, tokens, width, ff):
    g = torch.Generator().manual_seed(tokens + ff)
    x, w = torch.randn(tokens, width, generator=g) * 2, torch.randn(ff, width, generator=g) / math.sqrt(width)
    if kit.dtype != torch.float32:
        x, w = x.to(torch.bfloat16).float(), w.to(torch.bfloat16).float()
    z = x.double() @ w.double().T
    if kind == "xielu":  # the factors as the plain function makes them from the two learned numbers
        p, q = (torch.log(torch.expm1(torch.tensor(v, dtype=torch.float64))) for v in (numbers[0], numbers[1] - 0.5))
        want = pm.xielu(z, p, q)
    else:
        want = pm.erf_gelu(z) if kind == "gelu" else torch.relu(z) ** 2
    have = kit.linear_act(x.to(kit.device, kit.dtype), w.to(kit.device, kit.dtype), kind, numbers)
    assert have.dtype == kit.dtype
    _close(have.float(), want, 1e-5 if kit.dtype == torch.float32 else 1e-2, kind)
    small = z.abs() < 0.05  # close to zero both branches are half the input
    assert int(small.sum()) > 5 or tokens * ff < 400
    if kind == "xielu":
        assert float((have.float().cpu().double() - want)[small].abs().max()) <= (1e-5 if kit.dtype == torch.float32 else 5e-4)


@pytest.mark.parametrize("experts,top,width", [(5, 2, 48), (3, 3, 70), (1, 1, 40), (8, 2, 256), (16, 4, 128), (40, 7, 64)])
def test_softmax_over_the_chosen_logits_alone(kit, experts, top, width):
    g = torch.Generator().manual_seed(experts * 7 + top)
    dev = kit.device
    for tokens in (9, 150):
        x = torch.randn(tokens, width, generator=g)
        router = torch.randn(experts, width, generator=g) * 4.0 / math.sqrt(width)
        bias = torch.randn(experts, generator=g) * 2
        if kit.dtype != torch.float32:
            x, router = x.to(torch.bfloat16).float(), router.to(torch.bfloat16).float()
        logits = x.double() @ router.double().T + bias.double()
        chosen, weights = pm.route(logits, top)
        ids, have = kit.route_top(x.to(dev, kit.dtype), router.to(dev, kit.dtype), top, "softmax_chosen", logit_bias=bias.to(dev))
        ranked = torch.sort(logits, -1, descending=True).values
        gaps = (ranked[:, :-1] - ranked[:, 1:])[:, : top].min(-1).values if experts > 1 else torch.full((tokens,), 9.0)
        clear = gaps > 1e-4
        assert int(clear.sum()) >= 0.9 * tokens
        assert torch.equal(ids.cpu().long()[clear], chosen[clear])
        _close(have.cpu()[clear], weights[clear], 1e-5, "weights")
        # the bias is part of the logits: a large one chooses and outweighs, and the weights still sum to one
        push = torch.zeros(experts)
        push[-1] = 60.0
        ids2, have2 = kit.route_top(x.to(dev, kit.dtype), router.to(dev, kit.dtype), top, "softmax_chosen", logit_bias=push.to(dev))
        assert bool((ids2[:, 0] == experts - 1).all()) and float((have2[:, 0] - 1).abs().max()) < 1e-6
        # without a bias
        ids3, have3 = kit.route_top(x.to(dev, kit.dtype), router.to(dev, kit.dtype), top, "softmax_chosen")
        assert float((have3.sum(-1) - 1).abs().max()) < 1e-5


@pytest.mark.parametrize("experts,top,width,ff,tokens", [(5, 2, 48, 16, 9), (3, 3, 70, 10, 40), (1, 1, 64, 22, 7), (8, 2, 256, 64, 300),
                                                         (4, 2, 128, 32, 70), (16, 4, 128, 104, 200), (6, 1, 40, 18, 130)])
def test_experts_of_two_matrices(kit, experts, top, width, ff, tokens):
    g = torch.Generator().manual_seed(experts + tokens)
    x = torch.randn(tokens, width, generator=g)
    w = {}
    for e in range(experts):
        w[f"e{e}.up"], w[f"e{e}.down"] = torch.randn(ff, width, generator=g) / math.sqrt(width), torch.randn(width, ff, generator=g) / math.sqrt(ff)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).to(torch.int32)
    ids[: tokens // 2, 0] = ids[0, 0]  # one expert takes most of the rows, another may take none
    weights = torch.rand(tokens, top, generator=g)
    if kit.dtype != torch.float32:
        x = x.to(torch.bfloat16).float()
        w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    wd = {k: v.double() for k, v in w.items()}
    want = torch.zeros(tokens, width, dtype=torch.float64)
    with pm.stored_as(None if kit.dtype == torch.float32 else torch.bfloat16):
        for t in range(tokens):
            for e, s in zip(ids[t].tolist(), weights[t].double()):
                want[t] += s * pm.expert(x[t : t + 1].double(), wd, f"e{e}.")[0]
    dev = kit.device
    up, down = (torch.stack([w[f"e{e}.{n}"] for e in range(experts)]).to(dev, kit.dtype) for n in ("up", "down"))
    out = kit.routed_act(x.to(dev, kit.dtype), ids.to(dev), weights.to(dev), up, down, "gelu")
    assert out.shape == (top, tokens, width) and out.dtype == torch.float32
    _close(out.sum(0), want, 2e-5 if kit.dtype == torch.float32 else 2e-2, "experts")
    kit.check_errors()


# -- each kind of layer alone in a model, then all of them ---------------------------------------------------
ALONE = {
    "scan": [_mamba(36, 5, 3, 4, None)],
    "scan_of_one_tap": [_mamba(24, 16, 8, 1, None)],
    "scan_of_many_states": [_mamba(20, 70, 2, 2, None)],
    "latent": [_latent(3, 6, 4, 5, 12, 0.5, 30.0, None)],
    "delta": [_delta(2, 9, None)],
    "one_head": [_delta(1, 20, None)],
    "dense": [_latent(1, 8, 2, 8, 8, 0.3, 10.0, _dense(44))],
    "routed": [_delta(1, 8, _moe(6, 2, 20))],
    "twice": [_mamba(16, 4, 2, 3, _dense(24)), _mamba(24, 3, 5, 2, None)],
}


@pytest.mark.parametrize("kind", list(ALONE))
def test_layers_of_a_kind_prefill_against_single_tokens(kit, kind):
    cfg = _config(60, 56, 1e-5, 3.0, 6.0, copy.deepcopy(ALONE[kind]))
    if kit.dtype != torch.float32:
        cfg = every_expert(cfg)
    weights = pm.random_weights(cfg, 40, 6)
    requests = requests_of(cfg, [41, 6], seed=70)
    expected = {rid: plain_logits(cfg, weights, ids) for rid, ids in requests.items()}
    for schedule in (helpers.schedule_whole, lambda r: helpers.schedule_tail(r, tail=25)):
        steps = schedule(requests)
        engine = engine_of(cfg, weights, 4, kit, num_blocks=pages_needed(41, 4) + 2, max_seqs=2)
        got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
        assert_close(got, expected, tolerance(kit), kind)


def test_every_layers_average_leans_on_all_states(kit):
    """With layer scales of zero every layer's result is what it was given, and the residual after layer i follows from
    the weights of the averages alone, by hand."""
    cfg, page, weights = model("small")
    weights = {k: torch.zeros_like(v) if k.endswith((".ls1", ".ls2")) else v for k, v in weights.items()}
    ids = helpers.random_ids(cfg["vocab"], 13, 3)
    trace = []
    plain_logits(cfg, weights, ids, trace=trace)
    factor, states = 1.0, [1.0]  # every state is a multiple of the embedding output
    for i in range(len(cfg["layers"])):
        states.append(factor)
        mix = weights[f"l{i}.dwa"]
        factor = float(sum(float(mix[j]) * states[j] for j in range(i + 2)))
        x0 = weights["embed"][torch.tensor(ids)].double() * cfg["embedding"]["scale"]
        _close(trace[i], factor * x0, 1e-12, f"layer {i}")
    steps = helpers.schedule_tail({"a": ids}, tail=5)
    engine = engine_of(cfg, weights, page, kit, num_blocks=8, max_seqs=1)
    got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
    assert_close(got, {"a": plain_logits(cfg, weights, ids)}, tolerance(kit), "averages alone")


@pytest.mark.gpu
def test_clear_choices_in_sixteen_bits():
    """The bfloat16 engine with routers that choose a few of their experts, on prompts whose every choice is clear
    (found by trying seeds against the plain implementation): whole prompts, prefill against single tokens, portions."""
    from distie_b200.kernels import make_kernels

    kit = make_kernels(torch.bfloat16, "cuda:0")
    ORACLE["stored"] = torch.bfloat16
    cfg, page, weights = copy.deepcopy(SMALL), 4, pm.random_weights(SMALL, 0, RANKS["small"], router_gain=12.0)
    requests = {}
    for seed in range(400, 2400):
        ids = helpers.random_ids(cfg["vocab"], 6, seed)
        margins = []
        plain_logits(cfg, weights, ids, margins)
        if float(torch.stack(margins).min()) >= 0.5:
            requests[f"c{len(requests)}"] = ids
            if len(requests) == 3:
                break
    assert len(requests) == 3, "no prompts with clear choices among the seeds tried"
    expected = {rid: plain_logits(cfg, weights, ids) for rid, ids in requests.items()}
    for schedule in (helpers.schedule_whole, lambda r: helpers.schedule_tail(r, tail=4), helpers.schedule_portions):
        steps = schedule(requests)
        engine = engine_of(cfg, weights, page, kit, num_blocks=16, max_seqs=2)
        got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
        assert_close(got, expected, BF16_TOL, "clear choices")
    assert kit.kernel_counts.get("routed_act") and kit.kernel_counts.get("route_top")


LENGTHS = {"small": [70, 1, 29, 51], "awkward": [45, 3, 23, 38], "wide": [230, 97, 2, 140]}
SCHEDULES = {
    "whole": helpers.schedule_whole,
    "tail": lambda r: helpers.schedule_tail(r, tail=30),
    "portions": helpers.schedule_portions,
    "mixed": lambda r: helpers.schedule_mixed(r, seed=5, live_max=3, refeed=1),
}


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("mode", list(SCHEDULES))
def test_replay_against_plain(kit, name, mode):
    """Whole prompts, prefill against token-by-token decoding, portions down to two tokens, and batches of unequal
    requests (portions beside single tokens, a request given up and fed again) in a pool made for the schedule's
    peak and three seats, so that pages, seats and state slots are used again."""
    if name == "wide" and kit.device.type == "cpu" and mode != "mixed":
        pytest.skip("the wide configuration runs on the CPU in one mode only: it is slow there")
    cfg, page, weights = model(name, kit)
    requests = requests_of(cfg, LENGTHS[name])
    steps = SCHEDULES[mode](requests)
    peak = helpers.peak_tokens(steps, granule=page)
    engine, _, _ = engine_for(name, kit, num_blocks=pages_needed(peak, page), max_seqs=3)
    got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
    expected = {rid: plain_logits(cfg, weights, ids) for rid, ids in requests.items()}
    assert_close(got, expected, tolerance(kit), f"{name}/{mode}")
    assert engine.cache.free_seats == 3 and all(g.pool.num_free == g.num_pages for g in engine.cache.groups)
    if kit.device.type == "cuda":
        ran = kit.kernel_counts
        assert all(ran.get(n) for n in ("selective_scan", "channel_delta", "average_add_rmsnorm", "routed_act", "latent_kv_write"))
        if name == "wide" and kit.dtype == torch.bfloat16:
            assert ran.get("latent_attention_mma")
            if mode in ("whole", "tail"):  # portions long enough for full tiles
                assert ran.get("gemm_tcgen05") and ran.get("gemm_tcgen05_grouped") is not None


@pytest.mark.parametrize("name", ["small", "awkward"])
def test_cuts_at_around_and_across_page_borders(kit, name):
    """The first tokens one by one; portions that end just before, at and just after page borders; two tokens at a
    time across one; then single tokens across the next ones."""
    cfg, page, weights = model(name, kit)
    ids = helpers.random_ids(cfg["vocab"], 6 * page + 5, 77)
    cuts = [1, 1, 1, page - 3, 2, page - 1, 1, 1, page, 2, 2, page + 1, 1, 1, 2]
    steps, at = [], 0
    while at < len(ids):
        size = min(max(1, cuts.pop(0)) if cuts else 1, len(ids) - at)
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": ids[at : at + size], "want": list(range(size))}],
                      "end": ["a"] if at + size == len(ids) else []})
        at += size
    engine, _, _ = engine_for(name, kit, num_blocks=pages_needed(len(ids), page))
    got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
    assert_close(got, {"a": plain_logits(cfg, weights, ids)}, tolerance(kit), name)


def _unit(n, g):
    v = torch.randn(n, generator=g)
    return v / v.norm()


@pytest.mark.parametrize("through", ["latent", "scan", "delta"])
def test_a_far_token_decides_through_the_whole_model(kit, through):
    """One layer and 160 tokens, the second of which is one of two: the logits late in the sequence change by much when
    it changes, in a prompt and in tokens decoded alone, and the engine must follow the plain implementation in both.
    Through the latent attention that token's key stands out among all others; through the recurrences the state is
    made to forget slowly and the token to write strongly."""
    g = torch.Generator().manual_seed(4)
    width = 32
    layer = {"latent": _latent(2, 8, 4, 8, 16, 4.0, 100.0, None), "scan": _mamba(24, 4, 4, 2, None), "delta": _delta(2, 8, None)}[through]
    cfg = _config(50, width, 1e-5, 1.0, 30.0, [layer])
    weights = pm.random_weights(cfg, 9, 4)
    common, direction = _unit(width, g), _unit(width, g)
    direction = direction - (direction @ common) * common
    direction = direction / direction.norm()
    embed = 0.5 * torch.randn(50, width, generator=g) + 2.0 * common
    embed = embed - torch.outer(embed @ direction, direction)  # no other token lies along the direction
    embed[7], embed[8] = embed[7] + 9.0 * direction, embed[8] - 9.0 * direction
    weights["embed"] = embed
    m = "l0.mix."
    if through == "latent":  # every query looks along the first unrotated dimension, where token 7's key lies
        weights[m + "q"] *= 0.05
        weights[m + "dkv"][0] = 4.0 * direction
        for head in range(2):
            weights[m + "q"][head * 12] = 2.0 * common
            weights[m + "uk"][head * 8] = 0.0
            weights[m + "uk"][head * 8, 0] = 2.0
    elif through == "scan":  # half the states forget nothing over the sequence
        weights[m + "A_log"][:, :2] = -9.0
        weights[m + "in"][:24] = 0.2 * weights[m + "in"][:24] + 3.0 * direction
        weights[m + "conv"][:, -1] = 1.0
        weights[m + "x"][8:] *= 4.0  # what late tokens read the state with
        weights[m + "D"] *= 0.1
        weights[m + "conv.b"] *= 0.1
    else:
        weights[m + "w0"] = torch.full_like(weights[m + "w0"], -9.0)
        weights[m + "a.b"] = torch.full_like(weights[m + "a.b"], -6.0)
        weights[m + "a"] *= 0.1
        weights[m + "k"] = 0.03 * weights[m + "k"] + torch.outer(_unit(16, g), 1.0 * common)
        weights[m + "v"] = 0.05 * weights[m + "v"] + torch.outer(_unit(16, g), 8.0 * direction)
    weights["l0.norm1"] = torch.zeros_like(weights["l0.norm1"])  # the directions stay at right angles
    weights["l0.ls1"] = torch.full_like(weights["l0.ls1"], 3.0)
    weights = {k: v.to(torch.bfloat16).float() for k, v in weights.items()}
    others = [t for t in helpers.random_ids(48, 190, 5) if t not in (7, 8)][:160]
    expected, got = {}, {}
    for far in (7, 8):
        ids = [others[0], far] + others[1:]
        expected[far] = plain_logits(cfg, weights, ids)
        steps = helpers.schedule_tail({"a": ids}, tail=40)
        engine = engine_of(cfg, weights, 8, kit, num_blocks=pages_needed(len(ids), 8), max_seqs=1)
        got[far] = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
        assert_close(got[far], {"a": expected[far]}, tolerance(kit), f"far token {far}")
    moved = row_errors(expected[7][-60:], expected[8][-60:])
    assert float(moved.min()) > 2 * tolerance(kit) and float(moved.median()) > 0.15, \
        f"the far token does not show in the late logits ({float(moved.min()):.3f}, {float(moved.median()):.3f}): the test's weights are too weak"


def test_long_decoding_beside_requests_that_come_and_go(kit):
    """Two tokens of prompt, then 150 tokens one by one beside another request that comes and goes twice over (its
    seat, pages and states are used again)."""
    cfg, page, weights = model("small", kit)
    long_ids = helpers.random_ids(cfg["vocab"], 152, 5)
    other = helpers.random_ids(cfg["vocab"], 40, 6)
    steps = [{"step": 0, "entries": [{"id": "long", "tokens": long_ids[:2], "want": [0, 1]}], "end": []}]
    for at in range(2, len(long_ids)):
        entries = [{"id": "long", "tokens": [long_ids[at]], "want": [0]}]
        end = ["long"] if at == len(long_ids) - 1 else []
        if 40 <= at < 60:
            part = (at - 40) % 10
            entries.append({"id": f"o{(at - 40) // 10}", "tokens": other[4 * part : 4 * part + 4], "want": [3]})
            if part == 9:
                end.append(f"o{(at - 40) // 10}")
        steps.append({"step": at - 1, "entries": entries, "end": end})
    engine, _, _ = engine_for("small", kit, num_blocks=pages_needed(152, page) + pages_needed(40, page), max_seqs=2, max_model_len=160)
    got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
    want_other = plain_logits(cfg, weights, other)[3::4]
    assert_close(got, {"long": plain_logits(cfg, weights, long_ids), "o0": want_other, "o1": want_other}, tolerance(kit), "long")
    if kit.device.type == "cuda":  # steps of single tokens replayed the captured decode step
        assert engine.runner.use_graphs and engine.runner.graph_replays >= 100


@pytest.mark.parametrize("name", ["small", "awkward"])
def test_greedy_generation_through_the_scheduler(kit, name):
    """``Engine.run``: prompts cut into portions of five beside decoding requests, two seats for three requests, and
    one request sent back and recomputed; every token must be the plain implementation's arg-max (or a near tie)."""
    cfg, page, weights = model(name, kit)
    prompts = [helpers.random_ids(cfg["vocab"], n, 300 + n) for n in (17, 4, 26)]
    new_tokens = 12
    pool = pages_needed(max(len(p) for p in prompts) + new_tokens, page) * 2 + 1
    engine, _, _ = engine_for(name, kit, num_blocks=pool, max_seqs=2, prefill_chunk=5)
    sent_back, seen = [], []

    def on_token(request_id, token, finished):
        if request_id == "g0":
            seen.append(token)
            if len(seen) == 4:
                sent_back.append(engine.scheduler.force_preempt("g0"))

    results = engine.run([GenerateRequest(f"g{i}", p, new_tokens) for i, p in enumerate(prompts)], ignore_eos=True, on_token=on_token)
    assert sent_back == [True] and results[0].preemptions == 1
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == new_tokens
        whole = prompt + result.token_ids[:-1]
        logits = plain_logits(cfg, weights, whole)[len(prompt) - 1 :]
        for index, token in enumerate(result.token_ids):
            slack = (2e-4 if kit.dtype == torch.float32 else 8e-2) * float(logits[index].std())
            assert float(logits[index, token]) >= float(logits[index].max()) - slack, f"{result.request_id}: output {index} is no arg-max"


# -- the command line and the trace runner, as a user runs them ---------------------------------------------
@pytest.mark.gpu
def test_command_line_and_trace_runner(tmp_path):
    """``init-random`` writes a Mekusun folder from its configuration file, ``generate`` decodes greedily from it and
    ``bin/trace_run`` replays steps against it (a portion, then portions beside single tokens, then an ended request's
    seat used again): tokens and logits are the plain implementation's."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    from distie_b200.weights import ModelTensors

    ORACLE["stored"] = None  # both child processes run the float32 engine
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    env = dict(os.environ, PYTHONPATH=root + os.pathsep + os.environ.get("PYTHONPATH", ""))
    config_file = tmp_path / "cfg.json"
    config_file.write_text(json.dumps(SMALL))
    folder = tmp_path / "model"
    subprocess.run([sys.executable, "-m", "distie_b200", "init-random", "--config", str(config_file), "--out", str(folder),
                    "--seed", "9", "--std", "0.3", "--dtype", "bfloat16"], check=True, env=env, cwd=root, timeout=600)
    stored = ModelTensors(str(folder))
    weights = {name: stored.tensor(name).float() for name in stored.keys()}
    prompt = helpers.random_ids(SMALL["vocab"], 9, 11)
    done = subprocess.run([sys.executable, "-m", "distie_b200", "generate", "--model", str(folder), "--dtype", "fp32",
                           "--prompt", " ".join(map(str, prompt)), "--max-new-tokens", "6", "--num-blocks", "8",
                           "--ignore-eos"], capture_output=True, text=True, env=env, cwd=root, timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    tokens = json.loads(done.stdout)[0]["token_ids"]
    assert len(tokens) == 6
    logits = plain_logits(SMALL, weights, prompt + tokens[:-1])[len(prompt) - 1 :]
    for index, token in enumerate(tokens):
        assert float(logits[index, token]) >= float(logits[index].max()) - 2e-4 * float(logits[index].std())
    a, b, c = (helpers.random_ids(SMALL["vocab"], n, 50 + n) for n in (21, 13, 7))
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[17:18], "want": [0]}, {"id": "b", "tokens": b[:6], "want": [5]}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": a[18:19], "want": [0]}, {"id": "b", "tokens": b[6:], "want": [6]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "a", "tokens": a[19:20], "want": []}, {"id": "c", "tokens": c, "want": [6]}], "end": ["c"]},
        {"step": 4, "entries": [{"id": "a", "tokens": a[20:], "want": [0]}], "end": ["a"]},
    ]
    out_dir = tmp_path / "out"
    done = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out_dir),
                           "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps), env=env,
                          cwd=root, timeout=900, capture_output=True, text=True)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(5)]
    la, lb, lc = (plain_logits(SMALL, weights, ids) for ids in (a, b, c))
    wanted = {0: torch.stack([la[0], la[16]]), 1: torch.stack([la[17], lb[5]]), 2: torch.stack([la[18], lb[12]]),
              3: lc[6:7], 4: la[20:21]}
    for step, want in wanted.items():
        have = torch.from_numpy(np.fromfile(out_dir / f"{step}.f32", dtype="<f4").reshape(want.shape[0], -1).copy())
        assert float(row_errors(have, want).max()) <= FP32_TOL, f"step {step}"
