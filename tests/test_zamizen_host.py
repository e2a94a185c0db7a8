"""What of the Zamizen design needs no GPU: config.json key by key, what the
cache and the state slots must hold (a layer that reads another's keys has no
pages of its own, but state for its queries' convolution), the tensors a model
declares, and the plain implementation's own pieces against each other."""
import copy
import math

import pytest
import torch

import plain_zamizen as pz
from lyapunov_engine_b200.config.base import ConfigError
from lyapunov_engine_b200.config.zamizen import ZamizenConfig
from lyapunov_engine_b200.models.model import Model
from lyapunov_engine_b200.parts.base import ModelSpec, PartSpec, RunSpec
from lyapunov_engine_b200.parts.rope import ramped_rates
from lyapunov_engine_b200.registry import spec_for

SCALING = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}
CFG = {"architecture": "Zamizen", "vocab": 50, "width": 40, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
       "layers": [{"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.3, "conv": 4,
                                                  "rot": {"dims": 8, "base": 5000.0}}, "mlp": {"kind": "dense", "ff": 24}},
                  {"type": "latent_attention", "mixer": {"heads": 3, "dim": 6, "rot_dim": 10, "vdim": 9, "kv_rank": 14,
                                                         "scale": 0.25, "rot": {"dims": 10, "base": 300.0, "scaling": SCALING}},
                   "mlp": None},
                  {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.5, "conv": 2,
                                                  "kv_from": 0, "rot": {"dims": 8, "base": 5000.0}}, "mlp": None},
                  {"type": "latent_attention", "mixer": {"heads": 2, "dim": 8, "rot_dim": 4, "vdim": 16, "kv_rank": 20,
                                                         "scale": 0.4, "rot": {"dims": 4, "base": 10000.0}},
                   "mlp": {"kind": "dense", "ff": 56}}]}


def edit(cfg, path, value=None, delete=False):
    broken = copy.deepcopy(cfg)
    at = broken
    for key in path[:-1]:
        at = at[key]
    if delete:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return broken


def test_config_is_read_key_by_key():
    c = ZamizenConfig.from_dict(CFG)
    assert (c.vocab, c.width, c.norm_eps, c.residual_mult) == (50, 40, 1e-5, 0.6)
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.taps, a.rot_dims, a.rot_base, a.kv_from) == \
        (4, 2, 12, 20, 0.3, 4, 8, 5000.0, None)
    b = c.layers[1].mixer
    assert (b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.scale, b.rot_base) == (3, 6, 10, 9, 14, 0.25, 300.0)
    assert b.scaling.as_dict() == SCALING and c.layers[3].mixer.scaling is None
    assert [layer.ff for layer in c.layers] == [24, 0, 0, 56] and c.layers[2].mixer.kv_from == 0
    required = [("vocab",), ("width",), ("norm",), ("norm", "eps"), ("residual_mult",), ("layers",), ("layers", 0, "type"),
                ("layers", 0, "mixer"), ("layers", 0, "mlp", "kind"), ("layers", 0, "mlp", "ff")]
    required += [("layers", 0, "mixer", k) for k in ("heads", "kv_heads", "dim", "vdim", "scale", "conv", "rot")]
    required += [("layers", 1, "mixer", k) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot")]
    required += [("layers", i, "mixer", "rot", k) for i in (0, 1) for k in ("dims", "base")]
    required += [("layers", 1, "mixer", "rot", "scaling", k) for k in SCALING]
    for path in required:
        with pytest.raises(ConfigError) as e:
            ZamizenConfig.from_dict(edit(CFG, path, delete=True))
        assert str(path[-1]) in str(e.value), (path, str(e.value))
    for path, value in [(("layers", 0, "type"), "window"), (("layers", 0, "mlp", "kind"), "moe"),
                        (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "rot", "dims"), 7),
                        (("layers", 0, "mixer", "rot", "dims"), 14), (("layers", 0, "mixer", "conv"), 0),
                        (("layers", 0, "mixer", "rot", "scaling"), SCALING), (("layers", 1, "mixer", "rot", "dims"), 8),
                        (("layers", 2, "mixer", "kv_from"), 1), (("layers", 2, "mixer", "kv_from"), 2),
                        (("layers", 2, "mixer", "kv_from"), 7), (("layers", 2, "mixer", "vdim"), 12),
                        (("layers", 2, "mixer", "dim"), 16)]:
        with pytest.raises(ConfigError):
            ZamizenConfig.from_dict(edit(CFG, path, value))
    # a layer that reads keys of a layer which has none of its own
    chained = copy.deepcopy(CFG)
    chained["layers"].append(edit(CFG["layers"][2], ("mixer", "kv_from"), 2))
    with pytest.raises(ConfigError):
        ZamizenConfig.from_dict(chained)


def test_declared_tensors_are_the_designs():
    model = Model(spec_for(CFG))
    assert {d.name: tuple(d.shape) for d in model.tensors()} == pz.tensor_shapes(CFG)
    roles = {d.name: d.role for d in model.tensors()}
    for name in ("l0.norm1", "l0.norm1b.b", "l0.mix.q.b", "l0.mix.v.conv", "l0.mix.o.b", "l1.mix.dkv.norm", "final.norm.b"):
        assert roles[name] == "vector"         # kept in 32 bits
    for name in ("l0.mix.q", "l1.mix.g", "l1.mix.uk", "l3.mlp.up", "head"):
        assert roles[name] == "matrix"


def test_pages_and_state():
    model = Model(spec_for(CFG))
    # heads of 12 and 20 are held as 32; a latent of 14 with 10 turned entries as 32, one of 20 with 4 as 32 too
    assert [(g.num_kv_heads, g.head_dim, g.values) for g in model.groups] == [(2, 32, True), (1, 32, False)]
    assert model.streams_per_group == [1, 2]
    assert [(r.group, r.stream, r.writes) for r in model.runs] == [(0, 0, True), (1, 0, True), (0, 0, False), (1, 1, True)]
    # q | k | v of the first layer (4 + 2 + 2 heads), the queries alone of the one that reads its keys
    assert [tuple(s.shape) for s in model.states] == [(3, 8 * 32), (1, 6 * 32)]
    one = edit(CFG, ("layers", 0, "mixer", "conv"), 1)
    assert [tuple(s.shape) for s in Model(spec_for(one)).states] == [(1, 6 * 32)]


def test_what_does_not_fit_together_is_refused():
    spec = spec_for(CFG)
    with pytest.raises(ValueError, match="no keys of its own"):
        Model(ModelSpec(**{**spec.__dict__, "run_order": tuple(RunSpec(i) for i in range(4))}))
    # a bias on a mixer's output in an arrangement that adds none
    block = spec.layers[0].block
    params = {k: v for k, v in block.params.items() if k not in ("mixer_output_norm", "feed_forward_output_norm", "output_scale")}
    from lyapunov_engine_b200.parts.base import BLOCKS
    with pytest.raises(ValueError, match="bias"):
        BLOCKS.build(PartSpec("prenorm", params))
    with pytest.raises(ValueError):
        BLOCKS.build(PartSpec("prenorm", {**block.params, "feed_forward_output_norm": None}))


# ------------------------------------------------------------------ rates, layouts, the plain implementation's pieces
@pytest.mark.parametrize("rot,base,scaling", [(32, 10000.0, SCALING), (10, 300.0, SCALING), (64, 1e6, {"factor": 8.0, "original": 4096, "fast": 32, "slow": 1}),
                                              (2, 50.0, SCALING), (16, 1e4, None), (8, 7.0, {"factor": 2.0, "original": 7, "fast": 1.2, "slow": 1.1})])
def test_ramped_rates(rot, base, scaling):
    got, magnitude = ramped_rates(rot, base, scaling)
    want, m = pz.yarn_rates(rot, base, scaling)
    torch.testing.assert_close(got, want, rtol=1e-12, atol=0)
    assert abs(magnitude - m) < 1e-12
    if scaling:
        plain = pz.plain_rates(rot, base)
        assert bool((got <= plain * (1 + 1e-12)).all()) and bool((got >= plain / scaling["factor"] * (1 - 1e-12)).all())
        assert m == 0.1 * math.log(scaling["factor"]) + 1.0


def test_halves_and_pairs_are_one_turn_in_another_order():
    g = torch.Generator().manual_seed(0)
    x = torch.randn(5, 2, 12, generator=g, dtype=torch.float64)
    pos = torch.tensor([0, 1, 7, 300, 5])
    order = torch.arange(12).view(2, 6).t().reshape(-1)
    torch.testing.assert_close(pz.turn_pairs(x[..., order], pos, 12, 100.0), pz.turn_halves(x, pos, 12, 100.0)[..., order])
    # entries behind the turned ones pass unchanged
    assert torch.equal(pz.turn_pairs(x, pos, 8, 100.0)[..., 8:], x[..., 8:])


def test_the_convolution_starts_from_zeros_and_ends_at_the_current_token():
    u = torch.arange(1.0, 7.0, dtype=torch.float64)[:, None]
    taps = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64)
    assert pz.causal_conv(u, taps)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0, 456.0]


def test_the_last_norm_before_the_stream_has_the_layers_factor():
    """Doubling the factor doubles what one layer adds to the stream."""
    cfg = {**CFG, "layers": [edit(CFG["layers"][0], ("mlp",), None)]}
    w = pz.random_weights(cfg, seed=1)
    out = {}
    for m in (0.5, 1.0):
        layers = []
        pz.forward({**cfg, "residual_mult": m}, w, [3, 4, 5], layers_out=layers)
        out[m] = layers[0] - w["embed"][[3, 4, 5]]
    torch.testing.assert_close(out[1.0], 2 * out[0.5])
