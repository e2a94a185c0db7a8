"""What of the Zuzenex design needs no GPU: config.json key by key, what the
cache and the state slots must hold (every pass over a layer with its own), the
tensors a model declares, and the plain implementation's own pieces against
each other."""
import copy
import math

import pytest
import torch

import plain_zuzenex as pz
from lyapunov_engine_b200.config.base import ConfigError
from lyapunov_engine_b200.config.zuzenex import ZuzenexConfig
from lyapunov_engine_b200.models.model import Model
from lyapunov_engine_b200.registry import spec_for

CFG = {"architecture": "Zuzenex", "vocab": 50, "width": 32, "norm": {"eps": 1e-5}, "loop": {"start": 0, "stop": 2, "times": 2},
       "layers": [{"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.3,
                                                  "q_temp": {"coef": 0.2, "every": 9}},
                   "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 4, "identity": 2, "top": 3},
                           "shared": {"ff": 16}}},
                  {"type": "lightning", "mixer": {"heads": 3, "dim": 8, "vdim": 20, "decay": [0.5, 0.9, 0.99]},
                   "mlp": {"kind": "dense", "ff": 40}},
                  {"type": "lightning", "mixer": {"heads": 1, "dim": 6, "vdim": 4, "decay": [0.7]}, "mlp": None},
                  {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.25},
                   "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 3, "top": 1}}}]}


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
    c = ZuzenexConfig.from_dict(CFG)
    assert (c.vocab, c.width, c.norm_eps, c.loop) == (50, 32, 1e-5, (0, 2, 2))
    assert c.run_order() == [0, 1, 0, 1, 2, 3] == pz.run_order(CFG)
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.q_temp.coef, a.q_temp.every) == (4, 2, 8, 12, 0.3, 0.2, 9)
    assert c.layers[1].mixer.decay == (0.5, 0.9, 0.99) and c.layers[1].feed_forward.kind == "dense"
    f = c.layers[0].feed_forward
    assert (f.ff, f.experts, f.identity, f.top, f.shared_ff) == (24, 4, 2, 3, 16)
    assert c.layers[2].feed_forward is None and c.layers[3].mixer.q_temp is None
    assert (c.layers[3].feed_forward.identity, c.layers[3].feed_forward.shared_ff) == (0, 0)
    required = [("vocab",), ("width",), ("norm",), ("norm", "eps"), ("layers",), ("loop", "times"), ("layers", 0, "type"),
                ("layers", 0, "mixer"), ("layers", 0, "mixer", "heads"), ("layers", 0, "mixer", "kv_heads"),
                ("layers", 0, "mixer", "dim"), ("layers", 0, "mixer", "vdim"), ("layers", 0, "mixer", "scale"),
                ("layers", 0, "mixer", "q_temp", "coef"), ("layers", 0, "mixer", "q_temp", "every"),
                ("layers", 0, "mlp", "kind"), ("layers", 0, "mlp", "expert"), ("layers", 0, "mlp", "router"),
                ("layers", 0, "mlp", "router", "experts"), ("layers", 0, "mlp", "router", "top"),
                ("layers", 0, "mlp", "shared", "ff"), ("layers", 1, "mixer", "heads"), ("layers", 1, "mixer", "dim"),
                ("layers", 1, "mixer", "vdim"), ("layers", 1, "mixer", "decay"), ("layers", 1, "mlp", "ff")]
    for path in required:
        with pytest.raises(ConfigError) as e:
            ZuzenexConfig.from_dict(edit(CFG, path, delete=True))
        assert str(path[-1]) in str(e.value), (path, str(e.value))
    for path, value in [(("layers", 0, "type"), "window"), (("layers", 0, "mlp", "kind"), "sparse"),
                        (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 1, "mixer", "decay"), [0.5, 0.9]),
                        (("layers", 1, "mixer", "decay"), [0.5, 0.9, 1.5]), (("layers", 1, "mixer", "decay"), 0.5),
                        (("layers", 0, "mlp", "router", "top"), 7), (("layers", 0, "mixer", "q_temp", "every"), 0),
                        (("layers", 0, "mlp", "router", "identity"), -1), (("loop", "stop"), 9), (("loop", "start"), 3)]:
        with pytest.raises(ConfigError):
            ZuzenexConfig.from_dict(edit(CFG, path, value))


def test_optional_keys():
    plain = edit(edit(CFG, ("loop",), delete=True), ("layers", 0, "mixer", "q_temp"), delete=True)
    c = ZuzenexConfig.from_dict(plain)
    assert c.run_order() == [0, 1, 2, 3] and c.layers[0].mixer.q_temp is None
    # all of the router's choices may be identity experts plus one
    ZuzenexConfig.from_dict(edit(CFG, ("layers", 0, "mlp", "router"), {"experts": 1, "identity": 4, "top": 5}))
    # a stretch that runs no time at all
    assert ZuzenexConfig.from_dict(edit(CFG, ("loop", "times"), 0)).run_order() == [2, 3]


def test_declared_tensors_are_the_designs():
    model = Model(spec_for(CFG))
    declared = {d.name: tuple(d.shape) for d in model.tensors()}
    assert declared == {k: tuple(v) for k, v in pz.tensor_shapes(CFG).items()}
    roles = {d.name: d.role for d in model.tensors()}
    for name in ("l0.norm1", "l0.mix.q.norm", "l0.mix.sink", "l0.mlp.router", "l0.mlp.correction", "l1.mix.norm", "final.norm"):
        assert roles[name] == "vector"         # kept in 32 bits
    for name in ("l0.mix.q", "l1.mix.g", "l0.mlp.e0.up", "head"):
        assert roles[name] == "matrix"


def test_every_pass_has_a_cache_and_a_state_of_its_own():
    model = Model(spec_for(CFG))
    runs = model.runs
    assert [r.layer for r in runs] == [0, 1, 0, 1, 2, 3]
    pools = [(r.group, r.stream) for r in runs if r.group is not None]
    assert len(pools) == 3 and len(set(pools)) == 3 and all(r.writes for r in runs)
    # heads of 8 and 12 are held as 16; two kv heads each: one geometry for all three
    assert [(g.num_kv_heads, g.head_dim, g.window) for g in model.groups] == [(2, 16, None)]
    states = [r.state for r in runs if r.state is not None]
    assert states == [0, 1, 2]
    assert [tuple(s.shape) for s in model.states] == [(3, 20, 8), (3, 20, 8), (1, 4, 6)]


# ------------------------------------------------------------------ the plain implementation's pieces
def test_a_sink_is_a_key_with_no_value():
    """exp(sink) in the denominator = one more key of that score whose value is zero."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(7, h, 5, generator=g, dtype=torch.float64) for h in (4, 2, 2))
    sink = torch.tensor([-2.0, 0.0, 1.5, 40.0], dtype=torch.float64)
    got = pz.attend_with_sink(q, k, v, 0.4, sink)
    for h in range(4):
        for t in range(7):
            s = torch.cat([(q[t, h] @ k[:t + 1, h // 2].T) * 0.4, sink[h:h + 1]])
            want = torch.softmax(s, 0)[:-1] @ v[:t + 1, h // 2]
            torch.testing.assert_close(got[t, h], want)


def test_the_query_temperature_steps_where_it_should():
    f = pz.query_temperature(torch.arange(40), 0.5, 10)
    assert torch.equal(f[:9], torch.ones(9, dtype=torch.float64))            # floor((p + 1) / 10) = 0 up to p = 8
    torch.testing.assert_close(f[9:19], torch.full((10,), 1 + 0.5 * math.log(2.0), dtype=torch.float64))
    torch.testing.assert_close(f[39], torch.tensor(1 + 0.5 * math.log(5.0), dtype=torch.float64))


def test_the_recurrence_is_a_weighted_sum_over_the_past():
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(9, 2, n, generator=g, dtype=torch.float64) for n in (4, 4, 6))
    decay = [0.8, 0.99]
    got = pz.decayed_memory(q, k, v, decay)
    for h in range(2):
        for t in range(9):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            torch.testing.assert_close(got[t, h], want)


def test_the_correction_moves_the_choice_and_not_the_weights():
    w = {"m.router": torch.tensor([[2.0], [1.0], [0.0]], dtype=torch.float64),
         "m.correction": torch.tensor([0.0, 0.0, 5.0], dtype=torch.float64)}
    h = torch.ones(1, 1, dtype=torch.float64)
    ids, share, _ = pz.route(h, w, "m.", {"router": {"experts": 2, "identity": 1, "top": 2}})
    assert ids.tolist() == [[2, 0]]
    s = torch.softmax(torch.tensor([2.0, 1.0, 0.0], dtype=torch.float64), 0)
    torch.testing.assert_close(share[0], torch.stack([s[2], s[0]]) / (s[0] + s[2]))
