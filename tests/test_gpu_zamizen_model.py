"""Zamizen models through the framework (its loader, cache and state manager,
step function and kernels, driven by the trace replay program and by the
generation entry point) against the plain implementation of
tests/plain_zamizen.py: whole prompts, token-by-token decoding, portions down to
two tokens, mixed batches on a pool whose pages and state slots are used again,
long decoding over page borders from the first token on, far tokens, greedy
generation.  The configurations differ from one another in every size and in
the order of their layers; one takes the values that make mechanisms vanish or
equal 1, one has sizes the tensor-core kernels take whole, one has sizes no
kernel takes in 16-byte pieces, one a latent beyond the tensor-core head sizes.
Scores are sharp, so that a key that is missed, a convolution that starts over,
or keys of the wrong layer move the logits far beyond the tolerance (asserted)."""
import copy
import json
import os
import random

import numpy as np
import pytest
import torch

import plain_zamizen as pz
import replay_util as ru

pytestmark = pytest.mark.gpu


def ff(n):
    return {"kind": "dense", "ff": n} if n else None


def attention(heads, kv_heads, dim, vdim, scale, conv, rot, base, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv,
         "rot": {"dims": rot, "base": base}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": ff(mlp)}


def latent(heads, dim, rot, vdim, rank, scale, base, mlp, scaling=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"dims": rot, "base": base}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": m, "mlp": ff(mlp)}


def config(vocab, width, mult, layers, eps=1e-5):
    return {"architecture": "Zamizen", "vocab": vocab, "width": width, "residual_mult": mult, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # every size its own; two layers that read keys of two others, one of them with other query heads and another scale
    "a": (config(211, 96, 0.6, [
        attention(4, 2, 16, 24, 0.5, 4, 8, 900.0, 72), latent(3, 16, 8, 24, 40, 0.4, 700.0, 40, (4.0, 32, 4.0, 0.5)),
        attention(2, 1, 24, 8, 0.3, 2, 24, 5e4, None), attention(6, 2, 16, 24, 0.7, 3, 8, 900.0, None, kv_from=0),
        latent(2, 24, 16, 40, 24, 0.3, 1e4, None, (2.0, 100, 16.0, 1.0)), attention(2, 1, 24, 8, 0.4, 5, 24, 5e4, 56, kv_from=2)]), 8),
    # the values that make a mechanism vanish or equal to 1
    "b": (config(97, 64, 1.0, [
        attention(1, 1, 16, 16, 1.0, 1, 0, 10.0, 16), latent(1, 16, 2, 16, 16, 1.0, 50.0, None),
        attention(1, 1, 16, 16, 1.0, 1, 0, 10.0, None, kv_from=0), latent(2, 8, 16, 8, 8, 0.5, 1e4, 24, (1.0, 64, 8.0, 1.0)),
        attention(2, 2, 16, 16, 0.25, 2, 16, 1e4, 32)], eps=1e-6), 4),
    # sizes the tensor-core kernels take whole (heads of 64 and 128)
    "c": (config(300, 128, 0.8, [
        latent(4, 64, 64, 64, 64, 0.1, 1e5, 192, (8.0, 128, 8.0, 1.0)), attention(4, 2, 64, 64, 0.2, 3, 32, 5e5, 128),
        attention(4, 2, 64, 64, 0.1, 3, 32, 5e5, 256, kv_from=1), latent(8, 16, 16, 32, 48, 0.3, 1e4, None)]), 16),
    # sizes no kernel takes in 16-byte pieces; an odd latent; a negative scale and factor
    "d": (config(130, 100, -0.5, [
        latent(3, 7, 6, 5, 21, 0.5, 300.0, 36, (3.0, 50, 3.0, 0.4)), attention(3, 1, 21, 10, 0.4, 7, 12, 2e3, 42),
        attention(3, 1, 21, 10, -0.3, 6, 12, 2e3, None, kv_from=1)]), 8),
    # a latent beyond the tensor-core head sizes, several hundred tokens, heads larger than a lane's piece
    "e": (config(256, 160, 0.7, [
        latent(4, 32, 32, 48, 144, 0.2, 2e4, 224, (2.0, 256, 16.0, 1.0)), attention(2, 1, 144, 80, 0.1, 4, 64, 1e6, 96),
        latent(6, 24, 8, 16, 72, 0.3, 1e4, None), attention(2, 1, 144, 80, 0.12, 4, 64, 1e6, None, kv_from=1)]), 16),
}
LENGTHS = {"a": (23, 47, 75, 141), "b": (9, 70, 35, 101), "c": (40, 130, 601, 215), "d": (12, 66, 31, 90), "e": (70, 150, 480, 310)}
PROMPTS = {"a": (3, 30, 41, 100), "b": (1, 64, 2, 67), "c": (8, 128, 560, 101), "d": (2, 40, 30, 51), "e": (50, 129, 440, 290)}


def write_folder(folder, cfg, weights, dtype):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    save_file({k: v.to(dtype).contiguous() for k, v in weights.items()}, os.path.join(folder, "model.safetensors"))


def references(cfg, weights, requests):
    exact = {r: pz.forward(cfg, weights, ids) for r, ids in requests.items()}
    rounded = {r: pz.forward(cfg, weights, ids, round_to=torch.bfloat16) for r, ids in requests.items()}
    noise = float(np.sqrt(np.mean([float((rounded[r] - exact[r]).pow(2).mean()) for r in requests])))
    return dict(requests=requests, exact=exact, rounded=rounded, noise=noise)


def make_model(tmp_path_factory, name, cfg, page, weights, lengths=(), prompts=(), seed=7, requests=None):
    folders = {}
    for dtype, tag in ((torch.float32, "float32"), (torch.bfloat16, "bfloat16")):
        folders[tag] = str(tmp_path_factory.mktemp(f"zamizen_{name}_{tag}"))
        write_folder(folders[tag], cfg, weights, dtype)
    g = torch.Generator().manual_seed(seed)
    if requests is None:
        requests = {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}
    return dict(references(cfg, weights, requests), cfg=cfg, page=page, w=weights, folders=folders,
                prompt_lens={f"r{i}": n for i, n in enumerate(prompts)})


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return {name: make_model(tmp_path_factory, name, cfg, page, pz.random_weights(cfg, seed=len(name) + cfg["width"]),
                             LENGTHS[name], PROMPTS[name]) for name, (cfg, page) in CONFIGS.items()}


def check(m, trace, dtype, out_dir, pool=None, what="", extra=()):
    """Runs the trace and compares every wanted place.  float32: tight.
    bfloat16: in units of what rounding activations to bfloat16 moves the plain
    implementation's own logits by (root mean square over all places): the
    median place within 1.5 units, no place beyond 3 times the worst place of the plain
    implementation's own rounded run, and no more loud places than twice what that run has."""
    pool = pool or sum((len(v) + 63) // 64 * 64 for v in m["requests"].values())
    got = ru.run_trace(trace, m["folders"][dtype], dtype, str(out_dir), pool, m["page"], extra=extra)
    assert len(got) == sum(len(w) for w in trace.wanted)
    if dtype == "float32":
        return ru.compare(got, {r: v.float() for r, v in m["exact"].items()}, atol=3e-4, rtol=3e-4, what=what)
    units, own = [], []
    for (rid, p), row in sorted(got.items()):
        assert np.all(np.isfinite(row))
        d = row.astype(np.float64) - m["exact"][rid][p].numpy()
        units.append(float(np.sqrt(np.mean(d * d))) / m["noise"])
        own.append(float((m["rounded"][rid][p] - m["exact"][rid][p]).pow(2).mean().sqrt()) / m["noise"])
    worst = int(np.argmax(units))
    print(f"{what}: median {np.median(units):.2f} worst {units[worst]:.2f} (own {max(own):.2f})")
    limit = 3.0 * max(2.0, max(own))
    assert units[worst] <= limit, f"{what}: place {sorted(got)[worst]}: {units[worst]:.1f} units of rounding noise (limit {limit:.1f})"
    assert float(np.median(units)) <= 1.5, f"{what}: the median place lies {np.median(units):.2f} units of rounding noise off"
    loud, loud_own = sum(u > 2.5 for u in units), sum(u > 2.5 for u in own)
    assert loud <= 2 * loud_own + max(2, len(units) // 50), f"{what}: {loud} of {len(units)} loud places ({loud_own} of its own)"


def test_what_is_left_out_or_one_off_would_show(models):
    """The plain implementation with a mechanism left out or one off moves the
    logits by far more than the comparisons allow."""
    m = models["a"]
    ids, exact = m["requests"]["r3"], m["exact"]["r3"]

    def moved(cfg=m["cfg"], w=m["w"]):
        return float((pz.forward(cfg, w, ids) - exact).abs().amax(dim=-1)[10:].median())

    def with_layer(i, **keys):
        cfg = copy.deepcopy(m["cfg"])
        cfg["layers"][i]["mixer"].update(keys)
        return cfg

    def with_weights(f):
        return {k: f(k, v) for k, v in m["w"].items()}

    limit = 10 * 3e-4
    assert moved(dict(m["cfg"], residual_mult=0.62)) > limit
    cfg = copy.deepcopy(m["cfg"])
    del cfg["layers"][1]["mixer"]["rot"]["scaling"]
    assert moved(cfg) > limit
    assert moved(with_layer(0, rot={"dims": 16, "base": 900.0})) > limit
    assert moved(with_layer(3, scale=0.72)) > limit
    for end in ("mix.q.b", "mix.v.b", "mix.o.b", "norm1b.b", "norm2b.b"):
        assert moved(w=with_weights(lambda k, v: torch.zeros_like(v) if k.endswith(end) else v)) > limit, end
    # the convolution one token late; a gate that is open
    assert moved(w=with_weights(lambda k, v: torch.roll(v, -1, 1) if k.endswith(".k.conv") else v)) > limit
    assert moved(w=with_weights(lambda k, v: torch.zeros_like(v) if k == "l1.mix.g" else v)) > limit


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(models, name, dtype, tmp_path):
    check(models[name], ru.whole_trace(models[name]["requests"]), dtype, tmp_path, what=f"{name} {dtype} whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_then_token_by_token(models, name, dtype, tmp_path):
    check(models[name], ru.tail_trace(models[name]["requests"], tail=44), dtype, tmp_path, what=f"{name} {dtype} decode")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_down_to_two_tokens(models, name, dtype, tmp_path):
    m = models[name]
    check(m, ru.portions_trace(m["requests"]), dtype, tmp_path / "1", what=f"{name} {dtype} portions")
    check(m, ru.portions_trace(m["requests"], sizes=(2, 2, 3, 2, 129, 2, 258)), dtype, tmp_path / "2",
          what=f"{name} {dtype} small portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_mixed_batches_on_a_pool_that_is_used_again(models, name, dtype, tmp_path):
    """Twice the requests, up to four live on four state slots, on a pool that
    just holds the peak: late requests get pages and state rows that others
    gave back with their keys and projected values still in them."""
    m = models[name]
    requests, prompts = dict(m["requests"]), dict(m["prompt_lens"])
    g = torch.Generator().manual_seed(11)
    for rid, ids in list(m["requests"].items()):
        requests[rid + "x"] = torch.randint(0, m["cfg"]["vocab"], (min(len(ids), 150),), generator=g).tolist()
        prompts[rid + "x"] = min(m["prompt_lens"][rid], 120)
    trace = ru.mixed_trace(requests, prompts, chunk=16, max_live=4, seed=5)
    assert any(len(s["entries"]) >= 3 for s in trace.steps)
    both = m.get("both") or references(m["cfg"], m["w"], requests)
    m["both"] = both
    check(dict(m, **both), trace, dtype, tmp_path, pool=ru.peak_pool_tokens(trace, m["page"]), what=f"{name} {dtype} mixed",
          extra=("--max-num-seqs", "4"))
    pages = ru.read_pages(str(tmp_path))
    assert pages["allocations"] > pages["pool_pages"] and pages["reuses"] > 0, pages


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["c", "e"])
def test_a_batch_of_unequal_requests_against_each_alone(models, name, dtype, tmp_path):
    """Four requests whose portions have 1 to 300 tokens in one step: the logits of each alone."""
    m = models[name]
    requests = m["requests"]
    trace, at = ru.Trace(), {r: 0 for r in requests}
    for sizes in ((300, 2, 40, 1), (1, 128, 1, 257), (258, 1, 100, 5), (42, 84, 3, 3)):
        entries = []
        for r, n in zip(("r2", "r1", "r3", "r0"), sizes):
            n = min(n, len(requests[r]) - at[r])
            if n:
                entries.append((r, requests[r][at[r]:at[r] + n], "all"))
                at[r] += n
        trace.step(entries)
    check(m, trace, dtype, tmp_path, what=f"{name} unequal {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "d"])
def test_first_tokens_and_long_decoding(models, name, dtype, tmp_path):
    """One request token by token from its first token on, past many pages
    (the captured decode step serves it), beside a second request that joins
    late: the convolutions' first tokens see zeros before them."""
    m = models[name]
    g = torch.Generator().manual_seed(3)
    ids = torch.randint(0, m["cfg"]["vocab"], (170,), generator=g).tolist()
    other = m["requests"]["r1"]
    t = ru.Trace()
    for i, tok in enumerate(ids):
        entries = [("long", [tok], [0])]
        j = i - 100
        if 0 <= j < len(other):
            entries.append(("r1", [other[j]], [0]))
        t.step(entries, end=(["long"] if i == len(ids) - 1 else []) + (["r1"] if j == len(other) - 1 else []))
    check(dict(m, **references(m["cfg"], m["w"], {"long": ids, "r1": other})), t, dtype, tmp_path, pool=256,
          what=f"{name} {dtype} long decoding")
    assert ru.read_pages(str(tmp_path))["graph_steps"] > 100


FAR = {"key": config(40, 32, 0.9, [attention(2, 1, 16, 16, 3.0, 3, 8, 1e4, None)], eps=1e-6),
       "shared key": config(40, 48, 0.9, [attention(1, 1, 16, 16, 0.01, 2, 4, 1e4, None),
                                          attention(2, 1, 16, 16, 3.0, 3, 4, 1e4, None, kv_from=0)], eps=1e-6),
       "latent": config(40, 32, 0.9, [latent(2, 16, 8, 16, 24, 1.5, 1e4, None, (2.0, 64, 4.0, 1.0))], eps=1e-6)}


@pytest.mark.parametrize("what", sorted(FAR))
def test_a_far_token_decides(what, tmp_path_factory, tmp_path):
    """Hundreds of positions on, what one early token was still moves the last
    logits by many times what the comparison allows (through a key that a
    sharp score singles out: the early place is the one that moves them most).
    The engine must agree with the plain implementation in a whole prompt, in
    portions and token by token."""
    cfg = FAR[what]
    w = pz.random_weights(cfg, seed=9, sharp=6.0)
    ids = torch.randint(0, 40, (402,), generator=torch.Generator().manual_seed(2)).tolist()
    base = pz.forward(cfg, w, ids)

    def moved(place):
        lost = list(ids)
        lost[place] = (ids[place] + 3) % 40
        return float((pz.forward(cfg, w, lost)[-1] - base[-1]).abs().max())

    assert max(moved(p) for p in range(2, 60)) > 20 * 3e-4
    m = make_model(tmp_path_factory, "far", cfg, 8, w, requests={"far": ids})
    for dtype in ("float32", "bfloat16"):
        for k, trace in enumerate((ru.whole_trace(m["requests"]), ru.tail_trace(m["requests"], tail=12),
                                   ru.portions_trace(m["requests"], sizes=(3, 130, 2, 64, 200, 2)))):
            check(m, trace, dtype, tmp_path / f"{dtype}{k}", what=f"far {what} {dtype} {k}")


def test_state_rows_and_pages_are_given_back_and_zeroed(models):
    """Two state slots for five requests: every late request starts in a row
    that still holds an earlier request's projected values, and must start from zero."""
    from lyapunov_engine_b200 import LLMEngine, SamplingParams
    m = models["a"]
    engine = LLMEngine.from_pretrained(m["folders"]["float32"], dtype="float32", num_blocks=40, block_size=m["page"],
                                       max_num_seqs=2, max_num_batched_tokens=24, max_model_len=160)
    g = torch.Generator().manual_seed(2)
    prompts = [torch.randint(0, m["cfg"]["vocab"], (n,), generator=g).tolist() for n in (3, 37, 1, 26, 12)]
    outs = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.output_tokens == pz.greedy(m["cfg"], m["w"], p, 9), (p, o.output_tokens)
        assert o.finish_reason == "length"
    assert engine.block_manager.audit() == ""


@pytest.mark.parametrize("name", ["b", "c", "d", "e"])
def test_greedy_generation_through_the_entry_point(models, name):
    from lyapunov_engine_b200 import LLMEngine, SamplingParams
    m = models[name]
    engine = LLMEngine.from_pretrained(m["folders"]["float32"], dtype="float32", num_blocks=64, block_size=m["page"],
                                       max_num_seqs=3, max_num_batched_tokens=32, max_model_len=192)
    g = torch.Generator().manual_seed(4)
    prompts = [torch.randint(0, m["cfg"]["vocab"], (n,), generator=g).tolist() for n in (5, 41, 2, 19)]
    outs = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=7, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.output_tokens == pz.greedy(m["cfg"], m["w"], p, 7), (p, o.output_tokens)


@pytest.mark.parametrize("name", ["a", "d"])
def test_the_stream_after_every_layer(models, name):
    """The residual stream after every layer (what is still pending entered,
    through its norm) against the plain implementation."""
    from lyapunov_engine_b200 import build
    from lyapunov_engine_b200.cache import DeviceCache
    from lyapunov_engine_b200.engine.llm_engine import load_model
    from lyapunov_engine_b200.engine.step import ModelRunner
    from lyapunov_engine_b200.parts.base import NormedAddend
    m = models[name]
    host = build.load_host()
    loaded = load_model(m["folders"]["float32"], "float32", "cuda:0", max_model_len=128)
    cache = DeviceCache(loaded.model, loaded.runtime, 32, m["page"], 1)
    runner = ModelRunner(loaded.model, cache, loaded.runtime, 128, 1, 128, use_cuda_graphs=False, check_status=True)
    ids = m["requests"]["r1"]
    seen = []

    def observe(index, stream):
        u = stream.update
        assert isinstance(u, NormedAddend) and u.centered
        y = stream.pending
        y = (y.sum(0) if y.dim() == 3 else y).double()
        if u.input_bias is not None:
            y = y + u.input_bias.double()
        seen.append((stream.resid.double() + pz.layer_norm(y, u.weight.double(), u.bias.double(), u.eps)).cpu())

    forward = loaded.model.forward
    loaded.model.forward = lambda ctx, c: forward(ctx, c, observe=observe)
    seq = host.Sequence(0, ids, host.SamplingParams())
    assert cache.manager.grow(seq, len(ids))
    runner.step([host.StepEntry(seq, 0, len(ids), [0])])
    want = []
    pz.forward(m["cfg"], m["w"], ids, layers_out=want)
    assert len(seen) == len(want) == len(m["cfg"]["layers"])
    for got, ref in zip(seen, want):
        torch.testing.assert_close(got, ref, atol=2e-4, rtol=2e-4)


def draw_config(rng):
    """A configuration with every size and the order of the layers drawn at random."""
    layers = []
    mlp = lambda: rng.choice([0, 64, 96, 200, 256])

    def a_latent():
        rot = rng.choice([4, 8, 16, 32, 48])
        scaling = rng.choice([None, (rng.choice([1.5, 2.0, 8.0]), rng.choice([64, 200, 1000]), rng.choice([4.0, 16.0, 32.0]),
                                     rng.choice([0.5, 1.0, 2.0]))])
        return latent(rng.choice([1, 2, 3, 6, 8]), rng.choice([8, 16, 24, 48, 64]), rot, rng.choice([16, 24, 40, 64]),
                      rng.choice([16, 40, 64, 80, 112, 160]), rng.uniform(0.1, 0.3), rng.choice([1e3, 1e4, 5e5]), mlp(), scaling)

    def an_attention():
        heads, dim = rng.choice([2, 4, 6, 8]), rng.choice([24, 32, 48, 64, 80, 128])
        own = [i for i, layer in enumerate(layers) if layer["type"] == "attention" and "kv_from" not in layer["mixer"]]
        if own and rng.random() < 0.6:
            j = rng.choice(own)
            m = layers[j]["mixer"]
            return attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], rng.uniform(0.08, 0.3), rng.choice([2, 3, 4]),
                             m["rot"]["dims"], m["rot"]["base"], mlp(), kv_from=j)
        return attention(heads, rng.choice([g for g in (1, 2, 3, 4, 8) if heads % g == 0]), dim,
                         rng.choice([dim, dim // 2, 40, 16, 96]), rng.uniform(0.08, 0.3), rng.choice([1, 2, 3, 4, 5]),
                         rng.choice([r for r in (0, 8, 16, 24, 64) if r <= dim]), rng.choice([1e3, 1e4, 1e6]), mlp())

    for kind in [a_latent, an_attention] + [rng.choice([a_latent, an_attention]) for _ in range(rng.choice([2, 3, 4]))]:
        layers.append(kind())
    return config(rng.choice([300, 512, 777, 1000]), rng.choice([128, 192, 288, 384]), rng.uniform(0.3, 1.2), layers,
                  eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", [41, 42, 43, 44])
def test_configurations_drawn_at_random(seed, tmp_path_factory, tmp_path):
    """Sizes, layer order, readers of other layers' keys and page size drawn at
    random: whole prompts, portions and a mixed batch on a pool that just holds
    the peak, both types."""
    rng = random.Random(seed)
    cfg, page = draw_config(rng), rng.choice([16, 32, 64])
    m = make_model(tmp_path_factory, f"drawn{seed}", cfg, page, pz.random_weights(cfg, seed=seed), (150, 70, 300, 33),
                   (120, 64, 270, 2))
    for dtype in ("float32", "bfloat16"):
        check(m, ru.whole_trace(m["requests"]), dtype, tmp_path / f"w{dtype}", what=f"drawn {seed} {dtype} whole")
        check(m, ru.portions_trace(m["requests"]), dtype, tmp_path / f"p{dtype}", what=f"drawn {seed} {dtype} portions")
        trace = ru.mixed_trace(m["requests"], m["prompt_lens"], chunk=16, max_live=4, seed=5)
        check(m, trace, dtype, tmp_path / f"m{dtype}", pool=ru.peak_pool_tokens(trace, page), what=f"drawn {seed} {dtype} mixed",
              extra=("--max-num-seqs", "4"))


def test_command_line_generates_from_random_weights(tmp_path):
    """`generate --random-weights` builds a Zamizen model from a config.json alone."""
    import subprocess
    import sys
    folder = tmp_path / "cfg"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(CONFIGS["b"][0]))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "lyapunov"), "generate", "--model", str(folder),
                           "--random-weights", "--prompt-ids", "1,2,3", "--max-tokens", "4", "--temperature", "0"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
