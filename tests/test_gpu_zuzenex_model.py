"""Zuzenex models through the framework (its loader, cache and state manager,
step function and kernels, driven by the trace replay program and by the
generation entry point) against the plain implementation of
tests/plain_zuzenex.py: whole prompts, token-by-token decoding, portions down to
two tokens, mixed batches on a pool whose pages and state slots are used again,
long decoding over page borders and the steps of the query temperature from the
first token on, greedy generation.  The configurations differ from one another
in every size and in the order of their layers; one takes the values that make
mechanisms vanish or equal 1 (one head, one expert, no identity expert, a decay
of 1, a temperature that never moves), one leaves out every key that may be
absent and has sizes the tensor-core kernels take whole, one has sizes no kernel
takes in 16-byte pieces.  Scores are sharp, sinks large and some heads remember
hundreds of tokens, so that a key that is missed, a sink that is left out, a
temperature that steps one position late or a state that is dropped moves the
logits far beyond the tolerance (asserted)."""
import copy
import json
import os

import numpy as np
import pytest
import torch

import plain_zuzenex as pz
import replay_util as ru

pytestmark = pytest.mark.gpu


def moe(ff, experts, identity, top, shared):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if identity is not None:
        m["router"]["identity"] = identity
    if shared:
        m["shared"] = {"ff": shared}
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def attention(heads, kv_heads, dim, vdim, scale, temp, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def lightning(dim, vdim, decay, mlp):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def config(vocab, width, layers, loop=None, eps=1e-5):
    c = {"architecture": "Zuzenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # every size its own; a stretch of layers run three times; a layer without feed-forward
    "a": (config(211, 96, [attention(4, 2, 16, 24, 0.5, (0.4, 11), moe(40, 5, 2, 2, 56)),
                           lightning(20, 12, (0.4, 0.93, 0.997), dense(72)),
                           lightning(24, 40, (0.98, 0.7), moe(32, 3, 4, 3, 16)),
                           attention(6, 3, 24, 8, 0.3, (0.7, 30), None)], loop=(1, 3, 3)), 8),
    # the values that make a mechanism vanish or equal to 1
    "b": (config(97, 64, [lightning(16, 16, (1.0,), moe(32, 1, 0, 1, 32)),
                          attention(1, 1, 16, 16, 1.0, (0.0, 1), dense(16)),
                          lightning(8, 16, (0.0, 0.5), None),
                          attention(2, 2, 8, 8, 0.8, (0.5, 1), moe(16, 1, 3, 4, 0))], loop=(2, 3, 1), eps=1e-6), 4),
    # every key that may be absent is absent; sizes the tensor-core kernels take whole (heads of 64 and 128, segments of
    # 256 tokens and more)
    "c": (config(300, 128, [attention(4, 2, 64, 64, 0.2, None, moe(128, 8, None, 2, 0)),
                            lightning(64, 64, (0.9, 0.999), dense(256)),
                            attention(2, 1, 128, 64, 0.1, None, None),
                            lightning(128, 128, (0.995,), moe(64, 4, None, 1, 0))]), 16),
    # sizes no kernel takes in 16-byte pieces; heads that are padded in the cache; a loop over everything
    "d": (config(130, 100, [attention(3, 1, 21, 10, 0.4, (0.3, 5), moe(36, 3, 1, 2, 20)),
                            lightning(11, 7, (0.9, 0.99, 0.6), moe(42, 2, 2, 1, 0))], loop=(0, 2, 2)), 8),
}
CONFIGS["e"] = (
    # no router, so that no rounding can flip a choice and every place is held to the tight bounds in bfloat16 too;
    # sizes that are padded (lightning heads of 80 and 48, attention heads of 56 beside values of 64), several segments
    config(256, 160, [lightning(80, 96, (0.97, 0.9993), dense(224)),
                      attention(4, 2, 56, 64, 0.15, (0.3, 100), dense(320)),
                      lightning(48, 64, (0.6, 0.99, 0.998), None),
                      attention(3, 3, 32, 48, 0.25, None, dense(96))], loop=(1, 3, 2)), 16)
LENGTHS = {"a": (23, 47, 75, 141), "b": (9, 70, 35, 101), "c": (40, 130, 601, 215), "d": (12, 66, 31, 90), "e": (70, 150, 580, 310)}
PROMPTS = {"a": (3, 30, 41, 100), "b": (1, 64, 2, 67), "c": (8, 128, 560, 101), "d": (2, 40, 30, 51), "e": (50, 129, 540, 290)}


def write_folder(folder, cfg, weights, dtype):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    save_file({k: v.to(dtype).contiguous() for k, v in weights.items()}, os.path.join(folder, "model.safetensors"))


def make_model(tmp_path_factory, name, cfg, page, weights, lengths, prompts, seed=7):
    folders = {}
    for dtype in (torch.float32, torch.bfloat16):
        tag = "float32" if dtype == torch.float32 else "bfloat16"
        d = str(tmp_path_factory.mktemp(f"zuzenex_{name}_{tag}"))
        write_folder(d, cfg, weights, dtype)
        folders[tag] = d
    g = torch.Generator().manual_seed(seed)
    requests = {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}
    exact = {r: pz.forward(cfg, weights, ids) for r, ids in requests.items()}
    rounded = {r: pz.forward(cfg, weights, ids, round_to=torch.bfloat16) for r, ids in requests.items()}
    noise = float(np.sqrt(np.mean([float((rounded[r] - exact[r]).pow(2).mean()) for r in requests])))
    return dict(cfg=cfg, page=page, w=weights, folders=folders, requests=requests, exact=exact, rounded=rounded, noise=noise,
                prompt_lens={f"r{i}": n for i, n in enumerate(prompts)})


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return {name: make_model(tmp_path_factory, name, cfg, page, pz.random_weights(cfg, seed=len(name) + cfg["width"]),
                             LENGTHS[name], PROMPTS[name]) for name, (cfg, page) in CONFIGS.items()}


CLOSE_CALL = 0.01      # choice scores nearer than this: rounding to bfloat16 may choose either expert


def close_calls(cfg, weights, ids):
    """Per position: whether some router's last chosen score lies within
    CLOSE_CALL of the first one not chosen, here or at an earlier position
    (a choice that falls the other way also moves what the states carry on)."""
    margins = []
    pz.forward(cfg, weights, ids, margins_out=margins)
    if not margins:
        return np.zeros(len(ids), dtype=bool)
    close = (torch.stack(margins).amin(dim=0) < CLOSE_CALL).numpy()
    return np.maximum.accumulate(close)


def check(m, trace, dtype, out_dir, pool=None, what="", extra=()):
    """Runs the trace and compares every wanted place.  float32: tight.
    bfloat16: in units of what rounding activations to bfloat16 moves the plain
    implementation's own logits by (root mean square over all places): the
    median place within 1.5 units, no place beyond 30 (a key wrongly seen or
    missed, or a lost state, moves a place by 50 and more; where rounding
    alone flips a router's choice the plain implementation's own rounded run
    is as far off, and the place is measured from that run instead; places
    at or behind a router's close call are left out of this bound: no
    comparison rests on which way such a call falls), and no more loud places
    than twice what the plain implementation's own rounded run has (the same
    places left out; of all places a tenth at most)."""
    pool = pool or sum((len(v) + 63) // 64 * 64 for v in m["requests"].values())
    got = ru.run_trace(trace, m["folders"][dtype], dtype, str(out_dir), pool, m["page"], extra=extra)
    assert len(got) == sum(len(w) for w in trace.wanted)
    if dtype == "float32":
        return ru.compare(got, {r: v.float() for r, v in m["exact"].items()}, atol=3e-4, rtol=3e-4, what=what)
    units, own, near, clear = [], [], [], []
    close = m.setdefault("close", {})
    for (rid, p), row in sorted(got.items()):
        assert np.all(np.isfinite(row))
        if rid not in close:
            close[rid] = close_calls(m["cfg"], m["w"], m["requests"][rid])
        d = row.astype(np.float64) - m["exact"][rid][p].numpy()
        units.append(float(np.sqrt(np.mean(d * d))) / m["noise"])
        own.append(float((m["rounded"][rid][p] - m["exact"][rid][p]).pow(2).mean().sqrt()) / m["noise"])
        clear.append(not close[rid][p])
        d = row.astype(np.float64) - m["rounded"][rid][p].numpy()
        near.append(0.0 if close[rid][p] else min(units[-1], float(np.sqrt(np.mean(d * d))) / m["noise"]))
    worst = int(np.argmax(near))
    assert near[worst] <= 30.0, f"{what}: place {sorted(got)[worst]}: {near[worst]:.1f} units of rounding noise"
    assert float(np.median(units)) <= 1.5, f"{what}: the median place lies {np.median(units):.2f} units of rounding noise off"
    assert sum(u > 4.0 for u in units) <= 2 * sum(u > 4.0 for u in own) + max(2, len(units) // 10), what
    loud, loud_own = (sum(u > 4.0 and c for u, c in zip(us, clear)) for us in (units, own))
    assert loud <= 2 * loud_own + max(2, len(units) // 50), \
        f"{what}: {loud} of {len(units)} places above 4 units of rounding noise (the plain rounded run: {loud_own})"
    return float(np.median(units))


def test_what_is_left_out_or_one_off_would_show(models):
    """The plain implementation without its sinks, with a temperature that
    steps one position later, with one pass over the loop less or with every
    decay a little smaller moves the logits by far more than the comparisons
    allow."""
    m = models["a"]
    ids, exact = m["requests"]["r3"], m["exact"]["r3"]

    def moved(cfg=m["cfg"], w=m["w"]):
        return (pz.forward(cfg, w, ids) - exact).abs().amax(dim=-1)

    w = dict(m["w"])
    for name in w:
        if name.endswith(".sink"):
            w[name] = torch.full_like(w[name], -1e9)
    assert float(moved(w=w).median()) > 10 * 3e-4
    cfg = copy.deepcopy(m["cfg"])
    for layer in cfg["layers"]:
        if layer["type"] == "attention":
            layer["mixer"]["q_temp"]["every"] += 1
    late = moved(cfg)
    assert float(late[:9].max()) == 0.0 and float(late[10]) > 10 * 3e-4 and float(late[40:].median()) > 10 * 3e-4
    cfg = copy.deepcopy(m["cfg"])
    cfg["loop"]["times"] -= 1
    assert float(moved(cfg).median()) > 10 * 3e-4
    cfg = copy.deepcopy(m["cfg"])
    for layer in cfg["layers"]:
        if layer["type"] == "lightning":
            layer["mixer"]["decay"] = [d - 0.002 for d in layer["mixer"]["decay"]]
    assert float(moved(cfg)[40:].median()) > 10 * 3e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(models, name, dtype, tmp_path):
    m = models[name]
    check(m, ru.whole_trace(m["requests"]), dtype, tmp_path, what=f"{name} {dtype} whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_then_token_by_token(models, name, dtype, tmp_path):
    m = models[name]
    check(m, ru.tail_trace(m["requests"], tail=44), dtype, tmp_path, what=f"{name} {dtype} decode")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_down_to_two_tokens(models, name, dtype, tmp_path):
    m = models[name]
    check(m, ru.portions_trace(m["requests"]), dtype, tmp_path, what=f"{name} {dtype} portions")
    check(m, ru.portions_trace(m["requests"], sizes=(2, 2, 3, 2, 129, 2, 258)), dtype, tmp_path,
          what=f"{name} {dtype} small portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_mixed_batches_on_a_pool_that_is_used_again(models, name, dtype, tmp_path):
    """Twice the requests, up to four live on four state slots, on a pool that
    just holds the peak: late requests get pages and state rows that others
    gave back with their keys and state still in them."""
    m = models[name]
    requests, prompts, exact, rounded = dict(m["requests"]), dict(m["prompt_lens"]), dict(m["exact"]), dict(m["rounded"])
    g = torch.Generator().manual_seed(11)
    for rid, ids in list(m["requests"].items()):
        requests[rid + "x"] = torch.randint(0, m["cfg"]["vocab"], (min(len(ids), 150),), generator=g).tolist()
        prompts[rid + "x"] = min(m["prompt_lens"][rid], 120)
        exact[rid + "x"] = pz.forward(m["cfg"], m["w"], requests[rid + "x"])
        rounded[rid + "x"] = pz.forward(m["cfg"], m["w"], requests[rid + "x"], round_to=torch.bfloat16)
    trace = ru.mixed_trace(requests, prompts, chunk=16, max_live=4, seed=5)
    assert any(len(s["entries"]) >= 3 for s in trace.steps)
    m2 = dict(m, requests=requests, exact=exact, rounded=rounded)
    check(m2, trace, dtype, tmp_path, pool=ru.peak_pool_tokens(trace, m["page"]), what=f"{name} {dtype} mixed",
          extra=("--max-num-seqs", "4"))
    pages = ru.read_pages(str(tmp_path))
    assert pages["allocations"] > pages["pool_pages"] and pages["reuses"] > 0, pages


@pytest.mark.parametrize("name", ["c", "e"])
def test_a_batch_of_unequal_requests_against_each_alone(models, name, tmp_path):
    """Four requests whose portions have 1 to 300 tokens in one step (segments
    of one request beside single tokens of others, and the list of segments goes from one request to
    another and back): the logits of each alone."""
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
    for dtype in ("float32", "bfloat16"):
        check(m, trace, dtype, tmp_path / dtype, what=f"{name} unequal {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "d"])
def test_first_tokens_and_long_decoding(models, name, dtype, tmp_path):
    """One request token by token from its first token on, past many pages and
    every step of the temperature (the captured decode step serves it; the
    states pass from step to step 170 times), beside a second request that
    joins late."""
    m = models[name]
    g = torch.Generator().manual_seed(3)
    ids = torch.randint(0, m["cfg"]["vocab"], (170,), generator=g).tolist()
    other = m["requests"]["r1"]
    exact = {"long": pz.forward(m["cfg"], m["w"], ids), "r1": m["exact"]["r1"]}
    rounded = {"long": pz.forward(m["cfg"], m["w"], ids, round_to=torch.bfloat16), "r1": m["rounded"]["r1"]}
    t = ru.Trace()
    for i, tok in enumerate(ids):
        entries = [("long", [tok], [0])]
        j = i - 100
        if 0 <= j < len(other):
            entries.append(("r1", [other[j]], [0]))
        t.step(entries, end=(["long"] if i == len(ids) - 1 else []) + (["r1"] if j == len(other) - 1 else []))
    check(dict(m, requests={"long": ids, "r1": other}, exact=exact, rounded=rounded, close={}), t, dtype, tmp_path, pool=256,
          what=f"{name} {dtype} long decoding")
    assert ru.read_pages(str(tmp_path))["graph_steps"] > 100


def far_models():
    """(config, weights, the place that matters) of two one-layer models in
    which what an early token was moves the last logits through one mechanism."""
    cfg = config(40, 32, [lightning(16, 16, (0.999, 0.9995), None)], eps=1e-6)
    yield "state", cfg, pz.random_weights(cfg, seed=9), 5
    cfg = config(40, 32, [attention(2, 1, 16, 16, 1.0, (0.2, 40), None)], eps=1e-6)
    w = pz.random_weights(cfg, seed=5, sharp=6.0)
    yield "key", cfg, w, 33


def test_a_far_token_decides(tmp_path_factory, tmp_path):
    """Hundreds of positions on, what one early token was still moves the
    logits by many times what the comparison allows (through the state alone;
    through one key that a query singles out).  The engine must agree with the
    plain implementation in a whole prompt, in portions and token by token."""
    for what, cfg, w, place in far_models():
        g = torch.Generator().manual_seed(2)
        ids = torch.randint(1, 40, (402,), generator=g).tolist()
        if what == "key":
            # one token of its own kind at `place`: the queries of the last positions score it far above the others
            ids[place] = 0
            e = w["embed"]
            q, k = w["l0.mix.q"], w["l0.mix.k"]
            target = pz.unit_rms(e[ids[-1]], 1e-6) * w["l0.norm1"]
            e[0] = torch.linalg.lstsq(k, (q @ target)[:16]).solution.to(torch.bfloat16).double()
        m = make_model(tmp_path_factory, "far_" + what, cfg, 8, w, (1,), (1,))
        m["requests"] = {"far": ids}
        m["exact"] = {"far": pz.forward(cfg, w, ids)}
        m["rounded"] = {"far": pz.forward(cfg, w, ids, round_to=torch.bfloat16)}
        lost = list(ids)
        lost[place] = (ids[place] + 3) % 40
        moved = (pz.forward(cfg, w, lost)[401] - m["exact"]["far"][401]).abs().max()
        assert float(moved) > 10 * 3e-4, what
        for dtype in ("float32", "bfloat16"):
            for k, trace in enumerate((ru.whole_trace(m["requests"]), ru.tail_trace(m["requests"], tail=12),
                                       ru.portions_trace(m["requests"], sizes=(3, 130, 2, 64, 200, 2)))):
                check(m, trace, dtype, tmp_path / f"{what}{dtype}{k}", what=f"far {what} {dtype} {k}")


def test_state_rows_and_pages_are_given_back_and_zeroed(models, tmp_path):
    """Two state slots for five requests: every late request starts in a row
    that still holds an earlier request's state, and must start from zero."""
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


@pytest.mark.parametrize("name", ["b", "c", "d"])
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


def test_the_stream_after_every_layer_run(models):
    """The residual stream after every layer run (what is still pending
    entered) against the plain implementation; a looped layer counts each time."""
    from lyapunov_engine_b200 import build
    from lyapunov_engine_b200.cache import DeviceCache
    from lyapunov_engine_b200.engine.llm_engine import load_model
    from lyapunov_engine_b200.engine.step import ModelRunner
    from lyapunov_engine_b200.parts.base import SecondAddend
    m = models["a"]
    host = build.load_host()
    loaded = load_model(m["folders"]["float32"], "float32", "cuda:0", max_model_len=128)
    cache = DeviceCache(loaded.model, loaded.runtime, 32, m["page"], 1)
    runner = ModelRunner(loaded.model, cache, loaded.runtime, 128, 1, 128, use_cuda_graphs=False, check_status=True)
    ids = m["requests"]["r1"]
    seen = []

    def whole(y):
        return (y.sum(0) if y.dim() == 3 else y).float()

    def observe(index, stream):
        x = stream.resid.clone()
        if stream.pending is not None:
            x = x + whole(stream.pending)
        if isinstance(stream.update, SecondAddend):
            x = x + whole(stream.update.other)
        seen.append(x.cpu())

    forward = loaded.model.forward
    loaded.model.forward = lambda ctx, c: forward(ctx, c, observe=observe)
    seq = host.Sequence(0, ids, host.SamplingParams())
    assert cache.manager.grow(seq, len(ids))
    runner.step([host.StepEntry(seq, 0, len(ids), [0])])
    want = []
    pz.forward(m["cfg"], m["w"], ids, layers_out=want)
    assert len(seen) == len(want) == 8
    for got, ref in zip(seen, want):
        torch.testing.assert_close(got, ref.float(), atol=2e-4, rtol=2e-4)


def draw_config(rng):
    """A configuration with every size and the order of the layers drawn at random."""
    def mlp():
        r = rng.random()
        if r < 0.15:
            return None
        if r < 0.4:
            return dense(rng.choice([64, 96, 200, 256]))
        experts, identity = rng.choice([2, 4, 8, 12]), rng.choice([0, 1, 2, 4])
        return moe(rng.choice([64, 96, 128, 200]), experts, identity, rng.choice([t for t in (1, 2, 3, 4) if t <= experts + identity]),
                   rng.choice([0, 64, 96, 160]))

    def a_lightning():
        heads = rng.choice([1, 2, 3, 4, 6, 8])
        return lightning(rng.choice([16, 32, 48, 80, 96, 128]), rng.choice([16, 32, 72, 80, 128]),
                         [rng.choice([0.3, 0.8, 0.95, 0.99, 0.999, 0.9997]) for _ in range(heads)], mlp())

    def an_attention():
        heads, dim = rng.choice([2, 4, 6, 8]), rng.choice([24, 32, 64, 96, 128])
        return attention(heads, rng.choice([g for g in (1, 2, 3, 4, 8) if heads % g == 0]), dim, rng.choice([dim, dim // 2, 40, 16]),
                         rng.uniform(0.08, 0.25), rng.choice([None, (0.1, 16), (0.4, 50), (0.8, 200)]), mlp())

    n = rng.choice([3, 4, 5])
    kinds = [a_lightning, an_attention] + [rng.choice([a_lightning, an_attention]) for _ in range(n - 2)]
    rng.shuffle(kinds)
    start = rng.randrange(n)
    loop = rng.choice([None, (start, rng.randrange(start, n) + 1, rng.choice([1, 2, 3]))])
    return config(rng.choice([300, 512, 777, 1000]), rng.choice([128, 192, 320, 384]), [kind() for kind in kinds], loop=loop,
                  eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", [41, 42, 43])
def test_configurations_drawn_at_random(seed, tmp_path_factory, tmp_path):
    """Sizes, layer order, loop and page size drawn at random: whole prompts,
    portions and a mixed batch on a pool that just holds the peak, both types."""
    import random
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
    """`generate --random-weights` builds a Zuzenex model from a config.json alone."""
    import subprocess
    import sys
    cfg = CONFIGS["b"][0]
    folder = tmp_path / "cfg"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "lyapunov"), "generate", "--model", str(folder),
                           "--random-weights", "--prompt-ids", "1,2,3", "--max-tokens", "4", "--temperature", "0"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
