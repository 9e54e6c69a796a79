"""The Labolix decoder in the engine against the plain implementation (``plain_labolix``).

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
import plain_labolix as pl
from ref_kernels import RefKernels

from distie_b200.cache.manager import pages_needed
from distie_b200.config import ConfigError, EngineConfig, LabolixConfig, PartSpec, get_architecture
from distie_b200.engine.batch import BatchEntry, lay_out, views
from distie_b200.engine.engine import Engine, GenerateRequest
from distie_b200.engine.trace_replay import TraceSession
from distie_b200.kernels.interface import Averaged, KvSlot, Normed, RotaryTable, Terms
from distie_b200.models.decoder import model_tensor_specs
from distie_b200.parts import FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, BuildContext, build_part
from distie_b200.weights import WeightsError, open_weights

BY_WAVE = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40}
BY_RAMP = {"factor": 3.0, "fast": 8.0, "slow": 0.5, "original": 64}


def _rot(base, dims, scaling=None):
    return {"base": base, "dims": dims, **({"scaling": scaling} if scaling else {})}


def _attention(heads, kv_heads, dim, vdim, scale, rot, mlp):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                                       "scale": scale, "rot": rot}}


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, window, rot, mlp):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "mask": {"size": window}, "rot": rot}}


def _retention(heads, dim, vdim, decay, rot, mlp):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": rot}}


def _dense(ff, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _again(layers, index):
    return {**copy.deepcopy(layers[index]), "weights_of": index}


def _config(vocab, width, eps, cap, layers):
    return {"architecture": "Labolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


# Small: every branch once, two layers run again; pages of four.
_S = [
    _attention(3, 1, 12, 8, 0.3, _rot(100.0, 8, BY_WAVE), _dense(40)),
    _retention(3, 8, 10, [0.9, 0.97, 0.995], _rot(50.0, 6), _dense(36, 0.8)),
    _latent(2, 8, 4, 6, 20, 0.4, 9, _rot(1000.0, 4, BY_RAMP), _dense(40)),
]
SMALL = _config(96, 48, 1e-5, 9.0, _S + [_again(_S, 2), _again(_S, 1), _again(_S, 0)])
# Awkward: sizes that are no multiples of four, single heads, odd values, a window of one token and one of a page and a
# bit, a decay of one and one that forgets at once, layers without a feed-forward, no scaling, a factor below one, rotations
# of two dimensions and of all, a layer whose weights come from a later one, one that names another that names a third.
_A = [
    _retention(1, 33, 7, [1.0], _rot(100.0, 2), None),
    _latent(1, 10, 6, 5, 33, 0.25, 1, _rot(10.0, 6), _dense(45, 0.5)),
    _attention(5, 5, 7, 13, 0.5, _rot(30.0, 6), None),
    _latent(3, 5, 2, 9, 14, 0.7, 6, _rot(200.0, 2, {"factor": 0.5, "fast": 4.0, "slow": 1.0, "original": 30}), None),
    _retention(2, 6, 19, [0.3, -0.8], _rot(500.0, 6), _dense(18, 3.0)),
    _attention(4, 2, 18, 3, 0.2, _rot(1000.0, 18, {"factor": 2.0, "low": 2.0, "high": 2.5, "original": 25}), _dense(21)),
]
_A = _A + [{**copy.deepcopy(_A[4]), "weights_of": 7}, None, {**copy.deepcopy(_A[2]), "weights_of": 2}]
_A[7] = {**copy.deepcopy(_A[4]), "weights_of": 4}
AWKWARD = _config(101, 70, 1e-6, 2.5, _A)
# Sizes of a real model's order: in bfloat16 the tensor-core products, attentions and the chunks of the retention run.
_W = [
    _attention(4, 2, 128, 128, 0.09, _rot(10000.0, 64, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 100}), _dense(384, 2.0)),
    _retention(2, 64, 128, [0.97, 0.999], _rot(10000.0, 64), _dense(200)),
    _latent(4, 64, 32, 64, 128, 0.1, 70, _rot(10000.0, 32, BY_RAMP), _dense(384)),
    _attention(4, 1, 64, 32, 0.12, _rot(500.0, 48), None),
    _retention(4, 128, 40, [0.95, 0.99, 0.9995, 1.0], _rot(1000.0, 96), None),
    _latent(16, 32, 16, 32, 64, 0.14, 200, _rot(500.0, 16), _dense(256)),
    _attention(6, 3, 80, 48, 0.11, _rot(700.0, 80), _dense(128)),
]
WIDE = _config(500, 256, 1e-5, 20.0, _W + [_again(_W, 1), _again(_W, 2)])
CONFIGS = {"small": (SMALL, 4, 0), "awkward": (AWKWARD, 4, 1), "wide": (WIDE, 16, 2)}

FP32_TOL = 1e-4    # rms over the vocabulary of the logits' difference, mean taken off, over the logit scale
BF16_TOL = 5e-2

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


def model(name: str):
    cfg, page, seed = CONFIGS[name]
    return copy.deepcopy(cfg), page, pl.random_weights(cfg, seed)


def engine_of(cfg, weights, page, kit, num_blocks: int, max_seqs: int = 4, **knobs):
    arch = get_architecture(cfg["architecture"])
    dtype = "float32" if kit.dtype == torch.float32 else "bfloat16"
    config = EngineConfig(num_blocks=num_blocks, page_size=page, max_seqs=max_seqs, dtype=dtype, device=str(kit.device),
                          decode_graphs=kit.device.type == "cuda", **{"token_budget": 4096, **knobs})
    stored = {k: v.to(torch.bfloat16) for k, v in weights.items()}
    return Engine.assemble(arch, arch.config_cls.from_dict(cfg), stored, kit, config)


def engine_for(name: str, kit, num_blocks: int, max_seqs: int = 4, **knobs):
    cfg, page, weights = model(name)
    return engine_of(cfg, weights, page, kit, num_blocks, max_seqs, **knobs), cfg, weights


def plain_logits(cfg, weights, ids, trace=None) -> torch.Tensor:
    """The oracle: the plain implementation in float64; for the bfloat16 engine with that type's roundings where an
    engine stores 16 bits between two products (and nowhere else)."""
    with pl.stored_as(ORACLE["stored"]):
        return pl.forward(cfg, weights, ids, torch.float64, trace=trace).float()


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
    cfg = LabolixConfig.from_dict(AWKWARD)
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.logit_softcap, len(cfg.layers)) == (101, 70, 1e-6, 2.5, 9)
    assert cfg.weights_of == (0, 1, 2, 3, 4, 5, 4, 4, 2)
    first, latent, plain = cfg.layers[0].mixer, cfg.layers[3].mixer, cfg.layers[5].mixer
    assert (first.heads, first.dim, first.vdim, first.decay, first.rot.base, first.rot.dims) == (1, 33, 7, (1.0,), 100.0, 2)
    assert (latent.heads, latent.dim, latent.rot_dim, latent.vdim, latent.kv_rank, latent.scale, latent.window) == (3, 5, 2, 9, 14, 0.7, 6)
    assert latent.rot.scaling == {"factor": 0.5, "fast": 4.0, "slow": 1.0, "original": 30.0}
    assert (plain.heads, plain.kv_heads, plain.dim, plain.vdim, plain.scale, plain.rot.dims) == (4, 2, 18, 3, 0.2, 18)
    assert plain.rot.scaling == {"factor": 2.0, "low": 2.0, "high": 2.5, "original": 25.0}
    assert cfg.layers[0].mlp is None and (cfg.layers[4].mlp.ff, cfg.layers[4].mlp.limit) == (18, 3.0)
    for path, match in (
        (("layers", 0, "mixer", "kv_heads"), r"layers\[0\]\.mixer\.kv_heads"),
        (("layers", 0, "mixer", "rot", "dims"), r"layers\[0\]\.mixer\.rot\.dims"),
        (("layers", 0, "mixer", "rot", "scaling", "high"), r"layers\[0\]\.mixer\.rot\.scaling\.high"),
        (("layers", 1, "mixer", "decay"), r"layers\[1\]\.mixer\.decay"),
        (("layers", 1, "mixer", "rot"), r"layers\[1\]\.mixer\.rot"),
        (("layers", 2, "mixer", "mask"), r"layers\[2\]\.mixer\.mask"),
        (("layers", 2, "mixer", "rot", "scaling", "slow"), r"layers\[2\]\.mixer\.rot\.scaling\.slow"),
        (("layers", 0, "mlp", "limit"), r"layers\[0\]\.mlp\.limit"),
        (("layers", 0, "mlp", "kind"), r"layers\[0\]\.mlp\.kind"),
        (("norm",), "norm"),
        (("vocab",), "vocab"),
    ):
        broken = copy.deepcopy(SMALL)
        at = broken
        for key in path[:-1]:
            at = at[key]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=match):
            LabolixConfig.from_dict(broken)
    for change, match in (
        (lambda c: c["layers"][0].update(type="mamba2"), "mamba2"),
        (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe"),
        (lambda c: c["layers"][0]["mlp"].update(limit=0), "limit"),
        (lambda c: c["layers"][0]["mixer"].update(kv_heads=2), "kv_heads"),
        (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "dims"),
        (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5]), "decay"),
        (lambda c: c["layers"][1]["mixer"]["rot"].update(scaling=BY_WAVE), "scaling"),
        (lambda c: c["layers"][3].update(weights_of=9), "weights_of"),
        (lambda c: c["layers"][3].update(weights_of=3), "itself"),
        (lambda c: c["layers"][2].update(weights_of=3), "itself"),
        (lambda c: c["layers"][3]["mixer"].update(scale=0.1), r"layers\[3\] runs the weights of layer 2"),
        (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    ):
        broken = copy.deepcopy(SMALL)
        change(broken)
        with pytest.raises(ConfigError, match=match):
            LabolixConfig.from_dict(broken)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    cfg = CONFIGS[name][0]
    arch = get_architecture("Labolix")
    spec = arch.recipe(arch.config_cls.from_dict(cfg))
    specs = model_tensor_specs(spec)
    assert {s.name: s.default_shape for s in specs} == {k: tuple(v) for k, v in pl.tensor_shapes(cfg).items()}
    assert len(spec.order) == len(cfg["layers"]) and spec.num_cache_slots == len(cfg["layers"])
    weights = pl.random_weights(cfg, 1)
    open_weights(weights, specs, spec.tolerated, torch.float32, "cpu")
    for i, layer in enumerate(cfg["layers"]):  # a layer without a feed-forward may carry the norm of one, others no more
        broken = {**weights, f"l{i}.norm2.alpha": torch.ones(())}
        if layer["mlp"] is None and "weights_of" not in layer:
            open_weights(broken, specs, spec.tolerated, torch.float32, "cpu")
        elif "weights_of" in layer:
            with pytest.raises(WeightsError, match=f"l{i}.norm2.alpha"):
                open_weights(broken, specs, spec.tolerated, torch.float32, "cpu")


def test_random_model_folder_loads_by_its_config(tmp_path):
    from distie_b200.config import read_config
    from distie_b200.weights import write_random_model

    folder = write_random_model(str(tmp_path / "m"), SMALL, seed=3, std=0.1, norm_noise=0.05)
    arch, cfg = read_config(folder)
    assert arch.name == "Labolix" and cfg.width == 48
    engine = Engine.assemble(arch, cfg, folder, RefKernels(torch.float32),
                             EngineConfig(num_blocks=8, page_size=16, max_seqs=2, dtype="float32", device="cpu", decode_graphs=False))
    out = engine.generate([[1, 2, 3]], max_new_tokens=3, ignore_eos=True)
    assert len(out[0].token_ids) == 3


def test_parts_refuse_what_they_do_not_serve():
    base = {"heads": 2, "key_dim": 4, "value_dim": 4, "decay": [0.5, 0.9], "eps": 1e-5}
    position = PartSpec("rotary", {"head_dim": 4, "theta": 10.0})
    specs = MIXERS.get("decay_attention").tensor_specs
    assert [t.name for t in specs(PartSpec("decay_attention", base), 8)] == ["q", "k", "v", "g", "o", "norm"]
    turned = {**base, "activation": "none", "position": position, "norm": "head", "gate": "silu"}
    assert [t.name for t in specs(PartSpec("decay_attention", turned), 8)] == ["q", "k", "v", "g", "o"]
    for change in ({"decay": [0.5]}, {"gate": "tanh"}, {"norm": "none"}, {"position": position}, {"activation": "none"}, {"key_scale": 0.5}):
        with pytest.raises(ValueError):
            specs(PartSpec("decay_attention", {**base, **change}), 8)
    attention = {"num_heads": 2, "num_kv_heads": 1, "head_dim": 4, "sink": True, "sink_score": 0.0}
    with pytest.raises(ValueError, match="one of the two"):
        MIXERS.get("gqa_attention").tensor_specs(PartSpec("gqa_attention", attention), 8)
    latent = {"num_heads": 1, "head_dim": 4, "rot_dim": 2, "value_dim": 4, "kv_rank": 4, "q_rank": None, "window": 0}
    with pytest.raises(ValueError, match="window"):
        MIXERS.get("latent_attention").tensor_specs(PartSpec("latent_attention", latent), 8)
    with pytest.raises(ValueError, match="limit"):
        FEED_FORWARDS.get("swiglu")._limit(PartSpec("swiglu", {"limit": -1.0}))


# -- each mechanism alone: ops of the kernel set against the plain functions ------------------------------------
@pytest.mark.parametrize("width", [48, 201, 2304])
def test_dynamic_tanh_behind_a_residual_sum(kit, width):
    """Small and large elements (the norm is linear around zero and flat far out), a sum of terms, rows alone, and the
    pending forms other arrangements leave."""
    g = torch.Generator().manual_seed(width)
    tokens, dev = 9, kit.device
    residual = torch.randn(tokens, width, generator=g) * torch.tensor([0.01, 1.0, 30.0]).repeat(3)[:, None]
    a, b = torch.randn(3, tokens, width, generator=g), torch.randn(tokens, width, generator=g)
    weights = {"n": 1 + torch.randn(width, generator=g) * 0.3, "n.b": torch.randn(width, generator=g), "n.alpha": torch.tensor(0.7)}
    spec = PartSpec("dynamic_tanh", {"weight": "n", "bias": "n.b", "alpha": "n.alpha"}, "")
    cls = NORMS.get("dynamic_tanh")
    norm = cls.build(spec, BuildContext(kit, width, open_weights(weights, cls.tensor_specs(spec, width), (), kit.dtype, dev)))
    tol = 1e-6 if kit.dtype == torch.float32 else 5e-3

    def wanted(x):
        return pl.squash(x, 0.7, weights["n"].double(), weights["n.b"].double())

    summed = residual.double() + a.double().sum(0) + 0.5 * b.double()
    for delta, result in ((None, residual.double()), (a.to(dev), residual.double() + a.double().sum(0)),
                          (Terms([(a.to(dev), 1.0), (b.to(dev), 0.5)]), summed)):
        res, out = residual.clone().to(dev), torch.empty(tokens, width, dtype=kit.dtype, device=dev)
        rows, picked = torch.tensor([4, 0, 4], dtype=torch.int32, device=dev), torch.empty(3, width, dtype=kit.dtype, device=dev)
        norm.apply(delta, res, picked, rows)
        assert torch.equal(res.cpu(), residual)
        _close(picked, wanted(result)[[4, 0, 4]], tol, "picked rows")
        norm.apply(delta, res, out)
        _close(res, result, 1e-6, "residual")
        _close(out, wanted(result), tol, "norm")
    # many terms; what a normed sublayer or an average over depth leaves pending
    many = Terms([(b.to(dev), 0.1 * i) for i in range(30)])
    res, out = residual.clone().to(dev), torch.empty(tokens, width, dtype=kit.dtype, device=dev)
    norm.apply(many, res, out)
    _close(out, wanted(residual.double() + 43.5 * b.double()), max(tol, 1e-5), "thirty terms")
    w_delta = 1 + torch.randn(width, generator=g) * 0.2
    own = residual.double() + pl.rms_unit(b.double(), 1e-5) * w_delta.double()
    res = residual.clone().to(dev)
    norm.apply(Normed(b.to(dev), w_delta.to(dev), 1e-5), res, out)
    _close(out, wanted(own), max(tol, 1e-5), "behind a normed output")
    history, mix = torch.zeros(2, tokens, width), torch.tensor([0.4, 0.8])
    history[0] = a[0]
    res = residual.clone().to(dev)
    norm.apply(Averaged(b.to(dev), history.to(dev), 1, mix.to(dev)), res, out)
    _close(out, wanted(0.4 * a[0].double() + 0.8 * (residual.double() + b.double())), max(tol, 1e-5), "behind an average")


@pytest.mark.parametrize("limit", [0.5, 2.0, 7.0])
@pytest.mark.parametrize("tokens,width,ff", [(5, 48, 40), (40, 70, 45), (64, 64, 200), (70, 64, 36), (130, 128, 96), (300, 256, 384)])
def test_capped_gated_layer(kit, limit, tokens, width, ff):
    """Gates and ups on both sides of their limits (the gate has no lower one)."""
    g = torch.Generator().manual_seed(tokens + ff)
    x, w = torch.randn(tokens, width, generator=g), torch.randn(2 * ff, width, generator=g) * 1.5 * limit / math.sqrt(width)
    if kit.dtype != torch.float32:
        x, w = x.to(torch.bfloat16).float(), w.to(torch.bfloat16).float()
    gate, up = x.double() @ w[:ff].double().T, x.double() @ w[ff:].double().T
    for z, low in ((gate, -limit), (up, -limit)):
        assert int((z > limit).sum()) and int((z < low).sum())
    have = kit.linear_glu(x.to(kit.device, kit.dtype), w.to(kit.device, kit.dtype), limit)
    assert have.dtype == kit.dtype
    _close(have.float(), pl.capped_glu(gate, up, limit), 1e-5 if kit.dtype == torch.float32 else 1e-2, "capped layer")


def test_rotations_and_their_slowed_waves(kit):
    """Tables of both scalings and of none, and the rotation of neighbouring pairs and of halves, against the plain ones."""
    positions = torch.tensor([0, 1, 7, 63, 500, 4001])
    g = torch.Generator().manual_seed(1)
    ctx = BuildContext(kit, 8, None)
    cases = [
        ({"head_dim": 16, "rotary_dim": 12, "theta": 100.0, "scaling": BY_WAVE}, pl.frequencies_by_wavelength(100.0, 12, **BY_WAVE), 1.0),
        ({"head_dim": 20, "theta": 5e5, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}},
         pl.frequencies_by_wavelength(5e5, 20, 8.0, 1.0, 4.0, 2048), 1.0),
        ({"head_dim": 16, "theta": 1e4, "scaling": BY_RAMP}, *pl.frequencies_by_ramp(1e4, 16, BY_RAMP["factor"], BY_RAMP["original"],
                                                                                   BY_RAMP["fast"], BY_RAMP["slow"])),
        ({"head_dim": 2, "theta": 50.0, "scaling": {"factor": 2.0, "fast": 2.0, "slow": 1.0, "original": 20}},
         *pl.frequencies_by_ramp(50.0, 2, 2.0, 20, 2.0, 1.0)),
        ({"head_dim": 64, "rotary_dim": 48, "theta": 1e6}, pl.plain_frequencies(1e6, 48), 1.0),
    ]
    for params, freqs, strength in cases:
        for interleaved in (False, True):
            table = build_part(POSITION_ENCODINGS, PartSpec("rotary", {**params, "interleaved": interleaved, "factor": strength}), ctx).rotary_table()
            _close(table.inv_freq, torch.tensor(freqs, dtype=torch.float64), 1e-6, "frequencies")
            heads, dim, dims = 3, params["head_dim"], 2 * len(freqs)
            x = torch.randn(len(positions), 2 * heads * dim + 5, generator=g)
            step, _ = step_for(kit, [(0, [0] * 2, 0, ()), (1, [0], 7, ()), (2, [0], 63, ()), (0, [0], 500, ()), (1, [0], 4001, ())])
            order = step.positions.cpu().long()
            got = kit.rotate_heads(in_slices(x).to(kit.device), step, table, heads, dim, 0.3)
            pairs = pl.neighbours if interleaved else pl.halves(dims)
            parts = x[:, : 2 * heads * dim].double().reshape(len(positions), 2 * heads, dim)
            want = pl.turn(parts, order, freqs, pairs, strength)
            want[:, heads:] *= 0.3
            _close(got[:, : 2 * heads * dim], want.reshape(len(positions), -1), 3e-4, "rotation")  # angles of thousands in float32
            near = order < 100
            _close(got[near.to(got.device)][:, : 2 * heads * dim], want[near].reshape(int(near.sum()), -1), 1e-5, "rotation")
            assert torch.equal(got[:, 2 * heads * dim :].cpu(), x[:, 2 * heads * dim :])


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


@pytest.mark.parametrize("heads,dim,vdim,dims,interleaved,length", [
    (3, 8, 10, 6, False, 30), (1, 33, 7, 2, True, 70), (2, 6, 19, 6, False, 66), (2, 64, 64, 64, False, 150), (2, 128, 128, 128, False, 400),
    (5, 32, 48, 16, True, 129), (1, 128, 40, 96, False, 300), (2, 40, 128, 40, False, 200), (1, 200, 60, 20, False, 40), (1, 64, 200, 64, True, 90)])
def test_retention_in_portions(kit, heads, dim, vdim, dims, interleaved, length):
    """Two requests side by side, whole and in portions down to single tokens, with cuts inside, at and just past the
    edges of chunks; decays of one (nothing is ever forgotten), close to one, and of almost nothing; an early key that is
    large and a query late in the sequence that looks along it; a state slot that must stay as it is."""
    g = torch.Generator().manual_seed(heads + dim)
    if kit.device.type == "cpu" and length > 100:
        pytest.skip("long walks run on the GPU only")
    base, eps, scale = 60.0, 1e-5, dim ** -0.5
    qk, vv = heads * dim, heads * vdim
    lengths = {2: length, 1: 9}
    data = {}
    for seat, n in lengths.items():
        proj = torch.randn(n, 2 * qk + 2 * vv + 3, generator=g)
        proj[1, qk : 2 * qk] *= 6.0
        proj[n - 2, :qk] = proj[1, qk : 2 * qk]
        data[seat] = proj
    decay = torch.tensor([1.0, 0.02, 0.995, 0.9, -0.7][:heads]) if heads > 1 else torch.tensor([0.999])
    freqs, pairs = pl.plain_frequencies(base, dims), pl.neighbours if interleaved else pl.halves(dims)
    table = RotaryTable(torch.tensor(freqs, dtype=torch.float32, device=kit.device), dims, interleaved)
    want = {}
    for seat, proj in data.items():
        n, p = lengths[seat], data[seat].double()
        q, k = (pl.turn(p[:, i * qk : (i + 1) * qk].reshape(n, heads, dim), torch.arange(n), freqs, pairs) for i in range(2))
        o = pl.rms_unit(pl.retain(q, k * scale, p[:, 2 * qk : 2 * qk + vv].reshape(n, heads, vdim), decay.double()), eps).reshape(n, vv)
        z = p[:, 2 * qk + vv : 2 * qk + 2 * vv]
        want[seat] = {"silu": o * z * torch.sigmoid(z), "sigmoid": o * torch.sigmoid(z)}
    dev = kit.device
    ways = [({2: [length], 1: [9]}, "silu"), ({2: [1, 2, 1, 1, 5, length - 13, 1, 2], 1: [2, 1, 1, 4, 1]}, "sigmoid")]
    if length > 140:
        ways.append(({2: [63, 1, 65, length - 131, 2], 1: [1, 2, 6]}, "silu"))
    for portions, gate in ways:
        state = torch.zeros(4, heads, vdim, dim, device=dev)
        untouched = torch.randn(heads, vdim, dim, generator=g)
        state[3] = untouched.to(dev)

        def run(order, step):
            proj = torch.cat([data[s][a : a + c] for s, a, c in order])
            rows = (in_slices(proj) if len(order) > 1 else proj.unsqueeze(0)).to(dev)
            out = torch.empty(proj.shape[0], vv, dtype=kit.dtype, device=dev)
            kit.retention(rows[..., : 2 * qk + vv], rows[..., 2 * qk + vv : 2 * qk + 2 * vv], table, scale, decay.to(dev), state, step,
                          heads, dim, vdim, None, eps, gate, out)
            return out

        got = _walk(kit, lengths, portions, run)
        for seat in lengths:
            _close(got[seat], want[seat][gate], 3e-5 if kit.dtype == torch.float32 else 1e-2, f"seat {seat}, portions {portions[seat]}")
        assert torch.equal(state[3].cpu(), untouched) and float(state[0].abs().max()) == 0
    if kit.device.type == "cuda":
        assert kit.kernel_counts.get("retention_single")
        chunked = kit.dtype == torch.bfloat16 and max(dim, vdim) <= 128
        assert bool(kit.kernel_counts.get("retention_chunks")) == chunked and bool(kit.kernel_counts.get("rotate_heads")) != chunked


@pytest.mark.gpu
def test_the_state_behind_a_portion_is_float32():
    """In the 16-bit engine too: a portion's chunks leave the state a token-by-token float64 walk leaves, but for the
    rounding of each token's own key and value; what was in the state before passes through in full."""
    from distie_b200.kernels import make_kernels

    kit = make_kernels(torch.bfloat16, "cuda:0")
    g = torch.Generator().manual_seed(3)
    heads, dim, vdim, n = 2, 64, 96, 200
    qk, vv = heads * dim, heads * vdim
    proj, decay = torch.randn(n, 2 * qk + 2 * vv, generator=g), torch.tensor([1.0, 0.99])
    state = torch.zeros(2, heads, vdim, dim, device="cuda:0")
    start = torch.randn(heads, vdim, dim, generator=g) * 1e4
    state[1] = start.cuda()
    step, _ = step_for(kit, [(1, [0] * n, 50, ())])
    rows = proj.unsqueeze(0).cuda()
    out = torch.empty(n, vv, dtype=torch.bfloat16, device="cuda:0")
    kit.retention(rows[..., : 2 * qk + vv], rows[..., 2 * qk + vv :], None, 1.0, decay.cuda(), state, step, heads, dim, vdim, None, 1e-5,
                  "silu", out)
    k, v = proj[:, qk : 2 * qk].double().reshape(n, heads, dim), proj[:, 2 * qk : 2 * qk + vv].double().reshape(n, heads, vdim)
    want = start.double().clone()
    for head in range(heads):
        for t in range(n):
            want[head] = float(decay[head]) * want[head] + torch.outer(v[t, head], k[t, head])
    assert float((state[1].cpu().double() - want).abs().max()) < 0.1, "the state is kept in fewer bits than 32"
    # and what the portion reads of it: the state's share of every read-out is exact to 22 bits of it
    q = proj[:, :qk].double().reshape(n, heads, dim)
    o = torch.zeros(n, heads, vdim, dtype=torch.float64)
    for head in range(heads):
        S = start[head].double()
        for t in range(n):
            S = float(decay[head]) * S + torch.outer(v[t, head], k[t, head])
            o[t, head] = S @ q[t, head]
    z = proj[:, 2 * qk + vv :].double()
    _close(out.float(), pl.rms_unit(o, 1e-5).reshape(n, vv) * z * torch.sigmoid(z), 6e-3, "read-out")


def _kv_slot(kit, kv_heads, dim, vdim, pages, page, table):
    dev = kit.device
    return KvSlot(torch.zeros(pages, kv_heads, page, dim, dtype=kit.dtype, device=dev),
                  torch.zeros(pages, kv_heads, page, vdim, dtype=kit.dtype, device=dev),
                  torch.tensor(table, dtype=torch.int32, device=dev), page, pages)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,page,n", [
    (3, 1, 12, 8, 8, 4, 50), (5, 5, 7, 13, 6, 4, 40), (4, 2, 128, 128, 64, 16, 300), (4, 1, 64, 32, 48, 16, 200), (6, 3, 80, 48, 80, 8, 170),
    (8, 2, 128, 64, 32, 16, 150), (2, 2, 32, 96, 32, 16, 140), (10, 1, 64, 64, 64, 16, 130), (2, 1, 160, 128, 80, 16, 70)])
def test_attention_with_one_in_the_denominator(kit, heads, kv_heads, dim, vdim, dims, page, n):
    """From the stacked projection through pages handed out in reverse, in portions and token by token.  Keys at page
    borders, the very first one and every eleventh stand out for every query, each with a strength of its own; a stretch of
    queries points away from every key, so that the one in the denominator takes nearly all the weight."""
    g = torch.Generator().manual_seed(dim + n)
    base, scale = 80.0, 0.7 / math.sqrt(dim)
    freqs = pl.plain_frequencies(base, dims)
    q_end, k_end = heads * dim, (heads + kv_heads) * dim
    proj = torch.randn(n, k_end + kv_heads * vdim, generator=g)
    q, k = proj[:, :q_end].view(n, heads, dim), proj[:, q_end:k_end].view(n, kv_heads, dim)
    a = torch.randn(dim, generator=g)
    a[:dims] = 0  # along dimensions that are not rotated, where there are any
    a = a / a.norm() if dims < dim else torch.zeros(dim)
    q += 4.0 * a * math.sqrt(dim)
    for j, strength in {0: 2.0, **{b - 1: 1.5 for b in range(page, n, 3 * page)}, **{b: 1.2 for b in range(page, n, 2 * page)},
                        **{j: 0.8 + (j % 5) * 0.2 for j in range(5, n, 11)}}.items():
        k[j] += strength * a
    q[n // 2 : n // 2 + 9] *= -1.0
    rounded = torch.bfloat16 if kit.dtype != torch.float32 else None
    with pl.stored_as(rounded):
        positions, of = torch.arange(n), [h // (heads // kv_heads) for h in range(heads)]
        qd = pl.stored(pl.turn(q.double(), positions, freqs, pl.neighbours))
        kd = pl.stored(pl.turn(k.double(), positions, freqs, pl.neighbours))
        vd = pl.stored(proj[:, k_end:].double().reshape(n, kv_heads, vdim))
        want = pl.attend(qd, kd[:, of], vd[:, of], scale, torch.zeros(heads, dtype=torch.float64)).reshape(n, heads * vdim)
    dev = kit.device
    table = RotaryTable(torch.tensor(freqs, dtype=torch.float32, device=dev), dims, True)
    sink, width = torch.zeros(heads, device=dev), pages_needed(n, page)
    for cuts in ([1, 1, 2, page - 1, 1, 2, 3 * page, 1, 1, 4 * page + 1], [n]):
        kv = _kv_slot(kit, kv_heads, dim, vdim, width + 1, page, [[-1] * width, list(range(width - 1, -1, -1))])
        got, at, cuts = [], 0, list(cuts)
        while at < n:
            count = min(cuts.pop(0) if cuts else 1, n - at)
            step, _ = step_for(kit, [(1, [0] * count, at, ())])
            q_out = torch.empty(count, q_end, dtype=kit.dtype, device=dev)
            kit.qkv_norm_write(in_slices(proj[at : at + count]).to(dev), None, step, kv, table, heads, kv_heads, dim, vdim, None, None,
                               None, None, q_out)
            out = torch.empty(count, heads * vdim, dtype=kit.dtype, device=dev)
            kit.attention(q_out, out, step, kv, heads, kv_heads, dim, None, scale, None, 0, 0.0, sink)
            got.append(out.float().cpu())
            at += count
        kit.check_errors()
        _close(torch.cat(got), want, 2e-5 if kit.dtype == torch.float32 else 3e-2, "attention")


def test_one_key_and_one_in_the_denominator(kit):
    """A first token: its value times e^s / (1 + e^s), for a score that is zero, large and strongly negative."""
    dim, vdim = 12, 5
    for s, share in ((0.0, 0.5), (30.0, 1.0), (-30.0, 0.0), (1.0, math.e / (1 + math.e))):
        kv = _kv_slot(kit, 1, dim, vdim, 2, 4, [[0]])
        kv.k[0, 0, 0, 0] = 1.0
        kv.v[0, 0, 0] = torch.arange(1.0, vdim + 1, device=kit.device).to(kit.dtype)
        step, _ = step_for(kit, [(0, [0], 0, ())])
        q = torch.zeros(1, dim, dtype=kit.dtype, device=kit.device)
        q[0, 0] = s
        out = torch.empty(1, vdim, dtype=kit.dtype, device=kit.device)
        kit.attention(q, out, step, kv, 1, 1, dim, None, 1.0, None, 0, 0.0, torch.zeros(1, device=kit.device))
        _close(out.float(), share * torch.arange(1.0, vdim + 1)[None], 1e-5 if kit.dtype == torch.float32 else 6e-3, f"score {s}") if share else \
            _close(out.float() + 1, torch.ones(1, vdim), 1e-5, "nothing")


@pytest.mark.parametrize("heads,dim,rot,dims,vdim,rank,page,n,window", [
    (3, 8, 4, 4, 6, 20, 4, 61, 9), (1, 10, 6, 6, 5, 33, 4, 30, 1), (2, 6, 4, 2, 5, 24, 4, 40, 4), (2, 6, 4, 2, 5, 24, 4, 40, 39),
    (4, 64, 32, 32, 64, 128, 16, 260, 70), (16, 32, 16, 16, 32, 64, 8, 200, 64), (4, 32, 16, 16, 32, 64, 16, 330, 129),
    (20, 32, 32, 32, 32, 256, 16, 210, 100), (2, 16, 64, 64, 16, 512, 16, 200, 33), (3, 16, 8, 8, 16, 64, 16, 150, 1000)])
def test_latent_attention_over_a_window_with_sinks(kit, heads, dim, rot, dims, vdim, rank, page, n, window):
    """From the stacked projection through pages handed out in reverse, in portions and token by token, with the pages
    that a window has passed taken out of the block table (looking one up is an error).  Rows at page borders and every
    seventh carry a direction that every query looks for, the older the stronger: a key one position outside the
    window would outweigh everything inside.  Sinks from weak to strong."""
    g = torch.Generator().manual_seed(rank + n)
    eps, base, scale, strength = 1e-5, 100.0, 0.5, 1.3
    columns = heads * (dim + rot)
    up_k, up_v = torch.randn(heads, dim, rank, generator=g) / math.sqrt(rank), torch.randn(heads, rank, vdim, generator=g) / math.sqrt(rank)
    a = torch.randn(rank, generator=g)
    a = a / a.norm() * math.sqrt(rank)
    proj = torch.randn(n, columns + rank + rot, generator=g)
    marked = {j: 1.0 + (j * 5 % 9) * 0.3 for j in range(3, n, 7)}
    marked.update({j: 3.0 - 1.5 * j / n for b in range(2 * page, n, 2 * page) for j in (b - 1, b)})
    marked[0] = 5.0
    for j, s in marked.items():
        proj[j, columns : columns + rank] = s * a + torch.randn(rank, generator=g)
    q = proj[:, :columns].view(n, heads, dim + rot)
    q[..., :dim] += 2.0 * torch.einsum("hdr,r->hd", up_k, a) / math.sqrt(dim)
    weight, sink = 1 + 0.2 * torch.randn(rank, generator=g), torch.linspace(-2.0, 4.0, heads)
    if kit.dtype != torch.float32:
        up_k, up_v = up_k.to(torch.bfloat16).float(), up_v.to(torch.bfloat16).float()
    freqs, positions = pl.plain_frequencies(base, dims), torch.arange(n)
    with pl.stored_as(torch.bfloat16 if kit.dtype != torch.float32 else None):
        d = proj.double()
        c = pl.stored(pl.rms_unit(d[:, columns : columns + rank], eps) * weight.double())
        part = pl.stored(pl.turn(d[:, None, columns + rank :], positions, freqs, pl.neighbours, strength))
        qd = d[:, :columns].reshape(n, heads, dim + rot)
        q_all = torch.cat([pl.stored(qd[..., :dim]), pl.stored(pl.turn(qd[..., dim:], positions, freqs, pl.neighbours, strength))], -1)
        keys = torch.cat([torch.einsum("hdr,tr->thd", up_k.double(), c), part.expand(n, heads, rot)], -1)
        values = torch.einsum("hrv,tr->thv", up_v.double(), c)
        want = pl.attend(q_all, keys, values, scale, sink.double(), window).reshape(n, heads * vdim)
    dev = kit.device
    table = RotaryTable(torch.tensor(freqs, dtype=torch.float32, device=dev), dims, True, strength)
    width = pages_needed(n, page)
    for cuts in ([1, 1, 2, page - 1, 1, 2, 3 * page, 1, 1, 4 * page + 1, 2], [n]):
        k = torch.zeros(width + 1, 1, page, rank + rot, dtype=kit.dtype, device=dev)
        host = torch.tensor([[-1] * width, list(range(width - 1, -1, -1))], dtype=torch.int32)
        got, at, cuts = [], 0, list(cuts)
        while at < n:
            count = min(cuts.pop(0) if cuts else 1, n - at)
            host[1, : max(0, at - window + 1) // page] = -1
            kv = KvSlot(k, k[..., :rank], host.to(dev), page, width + 1)
            step, _ = step_for(kit, [(1, [0] * count, at, ())])
            rows = in_slices(proj[at : at + count]).to(dev)
            kit.latent_kv_write(rows[..., columns:], step, kv, table, 0, None, rank, weight.to(dev), rot, eps, None)
            folded, rotated = kit.latent_queries(rows[..., :columns], up_k.to(dev, kit.dtype), step, table, heads, dim, rot)
            mixed = torch.empty(heads, count, rank, dtype=kit.dtype, device=dev)
            kit.latent_attention(folded, rotated, step, kv, heads, rank, rot, scale, sink.to(dev), mixed, window)
            got.append(kit.latent_values(mixed, up_v.to(dev, kit.dtype), None, heads, vdim).float().cpu())
            at += count
        kit.check_errors()
        _close(torch.cat(got), want, 3e-5 if kit.dtype == torch.float32 else 3e-2, "latent attention")


@pytest.mark.parametrize("heads,dim,rot,dims,vdim,rank,page,window,gated", [
    (4, 64, 32, 32, 64, 128, 16, 70, False), (3, 128, 64, 64, 128, 256, 16, 200, False), (2, 64, 64, 48, 40, 64, 4, None, True),
    (5, 128, 8, 8, 96, 72, 32, 129, False), (1, 64, 16, 16, 128, 512, 16, 1, False), (6, 128, 48, 32, 64, 128, 24, 1000, True),
    (2, 32, 16, 16, 32, 64, 16, 60, False)])
def test_latents_of_long_portions_expanded_to_keys_and_values(kit, heads, dim, rot, dims, vdim, rank, page, window, gated):
    """The whole way from the query projection to the heads' outputs, three requests in a step: a single token behind a
    long past, a long portion behind a past that is no multiple of a block, and one from position 0.  The rows before each
    window are taken out of the block tables; marked rows sit at page, block and window borders, old ones the strongest."""
    g = torch.Generator().manual_seed(rank + dim)
    eps, base, scale = 1e-5, 100.0, 0.5
    dev, on_gpu = kit.device, kit.device.type == "cuda"
    pasts, counts = ([300, 261, 0], [1, 150, 140]) if on_gpu else ([40, 21, 0], [1, 30, 17])
    lengths = [p + c for p, c in zip(pasts, counts)]
    reach = window or 10 ** 6
    up_k, up_v = torch.randn(heads, dim, rank, generator=g) / math.sqrt(rank), torch.randn(heads, vdim, rank, generator=g) / math.sqrt(rank)
    sink = torch.linspace(-2.0, 3.0, heads)
    if kit.dtype != torch.float32:
        up_k, up_v = up_k.to(torch.bfloat16).float(), up_v.to(torch.bfloat16).float()
    a = torch.randn(rank, generator=g)
    a = a / a.norm()
    columns = heads * (dim + rot)
    freqs = pl.plain_frequencies(base, dims)
    table = RotaryTable(torch.tensor(freqs, dtype=torch.float32, device=dev), dims, True)
    width = pages_needed(max(lengths), page)
    pages = 3 * width + 1
    slab = torch.full((pages, 1, page, rank + rot), 7.0, dtype=kit.dtype, device=dev)
    host = torch.full((3, width), -1, dtype=torch.int32)
    order = torch.randperm(3 * width, generator=g).to(torch.int32).reshape(3, width)
    qs, gates, wanted = [], [], []
    for r, n in enumerate(lengths):
        q = torch.randn(n, heads, dim + rot, generator=g)
        q[..., :dim] += 2.0 * torch.einsum("hdr,r->hd", up_k, a) * math.sqrt(rank / dim)
        c = torch.randn(n, rank, generator=g)
        marks = {0: 5.0, **{j: 1.0 + (j * 5 % 7) * 0.3 for j in range(3, n, 9)}, **{b: 3.0 - b / n for b in range(page, n, 3 * page)},
                 **{j: 2.5 for j in (127, 128, pasts[r] - 1, pasts[r], n - reach, n - reach - 1) if 0 <= j < n}}
        for j, s in marks.items():
            c[j] += s * a * math.sqrt(rank) / 3
        part, gate = torch.randn(n, 1, rot, generator=g), torch.randn(n, heads, generator=g)
        positions = torch.arange(n)
        with pl.stored_as(torch.bfloat16 if kit.dtype != torch.float32 else None):
            cd, rd = pl.stored(c.double()), pl.stored(part.double())
            qd = torch.cat([pl.stored(q[..., :dim].double()), pl.stored(pl.turn(q[..., dim:].double(), positions, freqs, pl.neighbours))], -1)
            keys = torch.cat([torch.einsum("hdr,tr->thd", up_k.double(), cd), rd.expand(n, heads, rot)], -1)
            o = pl.attend(qd, keys, torch.einsum("hvr,tr->thv", up_v.double(), cd), scale, sink.double(), window)
        if gated:
            o = o * torch.sigmoid(gate.double())[..., None]
        wanted.append(o.reshape(n, heads * vdim)[pasts[r] :])
        qs.append(q.reshape(n, columns)[pasts[r] :])
        gates.append(gate[pasts[r] :])
        first = max(0, pasts[r] - reach + 1) // page
        held = pages_needed(n, page)
        host[r, first:held] = order[r, first:held]
        for j in range(first * page, n):
            slab[int(order[r, j // page]), 0, j % page] = torch.cat([cd[j], rd[j, 0]]).to(dev, kit.dtype)
    kv = KvSlot(slab, slab[..., :rank], host.to(dev), page, pages)
    step, layout = step_for(kit, [(r, [0] * counts[r], pasts[r], ()) for r in range(3)])
    rows = torch.cat([in_slices(q) for q in qs], 1).to(dev)
    up_rows = torch.cat([up_k.reshape(-1, rank), up_v.reshape(-1, rank)]).to(dev, kit.dtype)
    keys_first = up_rows[: heads * dim].view(heads, dim, rank)
    values_turned = up_rows[heads * dim :].view(heads, vdim, rank).transpose(1, 2).contiguous()
    got = kit.latent_heads(rows, keys_first, values_turned, up_rows, in_slices(torch.cat(gates)).to(dev) if gated else None, step,
                           layout.seqs, kv, table, heads, dim, rot, vdim, rank, scale, sink.to(dev), window)
    kit.check_errors()
    _close(got.float(), torch.cat(wanted), 3e-5 if kit.dtype == torch.float32 else 3e-2, "heads")
    if on_gpu:
        assert bool(kit.kernel_counts.get("attention_flat_tcgen05")) == (kit.dtype == torch.bfloat16 and dim >= 64)


# -- each kind of layer alone in a model, then all of them ---------------------------------------------------
ALONE = {
    "attention": [_attention(2, 1, 10, 6, 0.4, _rot(40.0, 6, BY_WAVE), None)],
    "attention_of_one_head": [_attention(1, 1, 6, 20, 0.4, _rot(10.0, 6), None)],
    "latent": [_latent(3, 6, 4, 5, 12, 0.5, 7, _rot(30.0, 4, BY_RAMP), None)],
    "latent_that_sees_itself": [_latent(2, 6, 4, 5, 12, 0.5, 1, _rot(30.0, 4), None)],
    "retention": [_retention(2, 9, 5, [0.99, 0.6], _rot(30.0, 8), None)],
    "dense": [_retention(1, 8, 8, [0.9], _rot(10.0, 8), _dense(44))],
    "again": [_retention(1, 8, 8, [0.95], _rot(10.0, 4), _dense(20)), {**_retention(1, 8, 8, [0.95], _rot(10.0, 4), _dense(20)), "weights_of": 0}],
}


@pytest.mark.parametrize("kind", list(ALONE))
def test_layers_of_a_kind_prefill_against_single_tokens(kit, kind):
    cfg = _config(60, 56, 1e-5, 6.0, copy.deepcopy(ALONE[kind]))
    weights = pl.random_weights(cfg, 40)
    requests = requests_of(cfg, [41, 6], seed=70)
    expected = {rid: plain_logits(cfg, weights, ids) for rid, ids in requests.items()}
    for schedule in (helpers.schedule_whole, lambda r: helpers.schedule_tail(r, tail=25)):
        steps = schedule(requests)
        engine = engine_of(cfg, weights, 4, kit, num_blocks=pages_needed(41, 4) + 2, max_seqs=2)
        got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
        assert_close(got, expected, tolerance(kit), kind)


def test_no_cap_on_the_logits(kit):
    cfg, page, weights = model("small")
    del cfg["logit_softcap"]
    ids = helpers.random_ids(cfg["vocab"], 13, 3)
    steps = helpers.schedule_tail({"a": ids}, tail=5)
    engine = engine_of(cfg, weights, page, kit, num_blocks=8, max_seqs=1)
    got = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))
    want = plain_logits(cfg, weights, ids)
    assert float(want.abs().max()) > 9.0
    assert_close(got, {"a": want}, tolerance(kit), "plain logits")


def test_a_layer_that_runs_again_has_a_cache_and_a_state_of_its_own(kit):
    """A model whose layers run twice equals one with two copies of the weights."""
    cfg, page, weights = model("small")
    twice = copy.deepcopy(cfg)
    copies = dict(weights)
    for index, layer in enumerate(twice["layers"]):
        source = layer.pop("weights_of", None)
        if source is not None:
            copies.update({f"l{index}.{name.split('.', 1)[1]}": w for name, w in weights.items() if name.startswith(f"l{source}.")})
    requests = requests_of(cfg, [37, 20])
    steps = helpers.schedule_mixed(requests, seed=3, live_max=2)
    got = []
    for c, w in ((cfg, weights), (twice, copies)):
        engine = engine_of(c, w, page, kit, num_blocks=pages_needed(64, page), max_seqs=2)
        got.append(helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps)))
    for rid in requests:
        assert torch.equal(torch.as_tensor(got[0][rid]), torch.as_tensor(got[1][rid]))
    assert_close(got[0], {rid: plain_logits(cfg, weights, ids) for rid, ids in requests.items()}, tolerance(kit), "twice")


LENGTHS = {"small": [70, 1, 29, 51], "awkward": [45, 3, 23, 38], "wide": [330, 97, 2, 140]}
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
    if name == "wide" and kit.device.type == "cpu":
        pytest.skip("the wide configuration runs on the GPU only: it is slow on the CPU")
    cfg, page, weights = model(name)
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
        assert all(ran.get(n) for n in ("add_dynamic_tanh", "qkv_norm_write", "latent_kv_write"))
        if name == "wide" and kit.dtype == torch.bfloat16:
            assert ran.get("latent_attention_mma") and ran.get("retention_chunks")
            assert not ran.get("linear_recurrence") and not ran.get("rotate_heads")
            if mode in ("whole", "tail"):  # portions long enough for full tiles
                assert ran.get("gemm_tcgen05") and ran.get("attention_prefill_tcgen05")


@pytest.mark.parametrize("name", ["small", "awkward"])
def test_cuts_at_around_and_across_page_borders(kit, name):
    """The first tokens one by one; portions that end just before, at and just after page borders; two tokens at a
    time across one; then single tokens across the next ones."""
    cfg, page, weights = model(name)
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


@pytest.mark.parametrize("window,page", [(1, 4), (4, 4), (7, 4), (16, 16), (33, 16), (70, 8)])
def test_just_inside_and_just_outside_the_window(kit, window, page):
    """One layer whose attention looks for one token: where it lies ``window - 1`` tokens back the logits are those that
    see it, one further back they are exactly those of a sequence without it, in a prompt and in tokens decoded alone."""
    width, n = 40, window + 30
    cfg = _config(50, width, 1e-5, 30.0, [_latent(2, 8, 4, 8, 16, 2.0, window, _rot(100.0, 4), None)])
    weights = pl.random_weights(cfg, 9)
    m = "l0.mix."
    weights[m + "sink"] = torch.tensor([-1.0, 0.5])
    embed = torch.randn(50, width, generator=torch.Generator().manual_seed(2)) * 0.3
    embed[:, :4] = 0.0
    embed[:, 0], embed[7, 1], embed[8, 1] = 2.0, 6.0, -6.0  # what all tokens share; what marks 7 and 8 apart
    weights["embed"] = embed
    weights[m + "q"] *= 0.1
    weights[m + "dkv"] *= 0.3
    weights[m + "dkv"][:16, 1] = 0.0
    weights[m + "dkv"][0, 1] = 4.0
    for head in range(2):  # every query looks along the first plain dimension, where the marked keys lie
        weights[m + "q"][head * 12, 0] = 2.5
        weights[m + "uk"][head * 8] = 0.0
        weights[m + "uk"][head * 8, 0] = 2.0
    weights["l0.norm1.b"] = torch.zeros(width)
    weights = {k: v.to(torch.bfloat16).float() for k, v in weights.items()}
    others = [t for t in helpers.random_ids(48, 3 * n, 5) if t not in (7, 8)][: n - 1]
    at, got = 6, {}
    for marked in (7, 8):
        ids = others[:at] + [marked] + others[at:]
        for mode, steps in (("whole", helpers.schedule_whole({"a": ids})), ("tail", helpers.schedule_tail({"a": ids}, tail=n - 4)),
                            ("portions", helpers.schedule_portions({"a": ids}))):
            engine = engine_of(cfg, weights, page, kit, num_blocks=pages_needed(n, page), max_seqs=1)
            got[marked, mode] = helpers.collect(steps, helpers.run_schedule(TraceSession(engine), steps))["a"]
            assert_close({"a": got[marked, mode]}, {"a": plain_logits(cfg, weights, ids)}, tolerance(kit), f"token {marked}, {mode}")
    for mode in ("whole", "tail", "portions"):
        one, two = torch.as_tensor(got[7, mode]), torch.as_tensor(got[8, mode])
        assert torch.equal(one[at + window :], two[at + window :]), "a token outside the window still counts"
        assert float(row_errors(one, two)[at : at + window].min()) > 0.02, "a token inside the window does not count"


def _unit(n, g):
    v = torch.randn(n, generator=g)
    return v / v.norm()


@pytest.mark.parametrize("through", ["attention", "retention"])
def test_a_far_token_decides_through_the_whole_model(kit, through):
    """One layer and 160 tokens, the second of which is one of two: the logits late in the sequence change by much when
    it changes, in a prompt and in tokens decoded alone, and the engine must follow the plain implementation in both."""
    g = torch.Generator().manual_seed(4)
    width = 32
    layer = {"attention": _attention(2, 1, 12, 8, 3.0, _rot(100.0, 4), None),
             "retention": _retention(2, 12, 8, [0.999, 1.0], _rot(100.0, 4), None)}[through]
    cfg = _config(50, width, 1e-5, 30.0, [layer])
    weights = pl.random_weights(cfg, 9)
    m = "l0.mix."
    embed = 0.3 * torch.randn(50, width, generator=g)
    embed[:, :3] = 0.0
    embed[:, 0], embed[7:9, 1], embed[7, 2], embed[8, 2] = 2.0, 6.0, 6.0, -6.0  # shared; what marks two tokens; what tells them apart
    weights["embed"] = embed
    weights["l0.norm1.b"] = torch.zeros(width)
    weights[m + "q"] *= 0.1
    weights[m + "k"] *= 0.05
    for head in range(2):  # queries look along a dimension behind the rotated ones, where the marked token's key lies
        weights[m + "q"][head * 12 + 8, 0] = 3.0
    rows = [8] if through == "attention" else [8, 20]
    for row in rows:
        weights[m + "k"][row, 1] = 4.0
    weights[m + "k"][:, 2] = 0.0
    weights[m + "v"][:, 2] *= 4.0
    if through == "retention":  # what other tokens write is small
        weights[m + "v"][:, 3:] *= 0.1
        weights[m + "v"][:, :2] *= 0.1
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
    assert float(moved.min()) > 2 * tolerance(kit) and float(moved.median()) > 0.13, \
        f"the far token does not show in the late logits ({float(moved.min()):.3f}, {float(moved.median()):.3f}): the test's weights are too weak"


def test_long_decoding_beside_requests_that_come_and_go(kit):
    """Two tokens of prompt, then 150 tokens one by one beside another request that comes and goes twice over (its
    seat, pages and states are used again); the windowed layers have long given the first pages back."""
    cfg, page, weights = model("small")
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
    session = TraceSession(engine)
    outputs = helpers.run_schedule(session, steps[:-1])
    windowed = [g for g in engine.cache.groups if g.need.window is not None]
    assert windowed and all(len(g.pages_of(session.live["long"][0])) <= pages_needed(g.need.window, page) + 1 for g in windowed)
    outputs.update(helpers.run_schedule(session, steps[-1:]))
    got = helpers.collect(steps, outputs)
    want_other = plain_logits(cfg, weights, other)[3::4]
    assert_close(got, {"long": plain_logits(cfg, weights, long_ids), "o0": want_other, "o1": want_other}, tolerance(kit), "long")
    if kit.device.type == "cuda":  # steps of single tokens replayed the captured decode step
        assert engine.runner.use_graphs and engine.runner.graph_replays >= 100


@pytest.mark.parametrize("name", ["small", "awkward"])
def test_greedy_generation_through_the_scheduler(kit, name):
    """``Engine.run``: prompts cut into portions of five beside decoding requests, two seats for three requests, and
    one request sent back and recomputed; every token must be the plain implementation's arg-max (or a near tie)."""
    cfg, page, weights = model(name)
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
    """``init-random`` writes a Labolix folder from its configuration file, ``generate`` decodes greedily from it and
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
