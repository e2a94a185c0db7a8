"""A plain, slow implementation of the Zuzenex decoder for the tests: whole
sequences, no cache, no state carried between calls, one function per
mechanism, on the CPU in the type asked for (float64 as the yardstick).  It
shares no code with the package.

``round_to``: activations are rounded to that type (and widened again) after
every matrix product and after every norm or gate whose output feeds one,
which is where a pipeline that computes in that type rounds; everything the
design keeps 32-bit (the stream, norms, scores, softmax, routers, the
recurrence) stays wide.

The model is given as a config dictionary (the keys of config.json) and a
dictionary of tensors by checkpoint name.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ small pieces
def _r(x, round_to):
    return x if round_to is None else x.to(round_to).to(x.dtype)


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


# ------------------------------------------------------------------ attention
def query_temperature(positions, coef, every):
    """One factor per position: it steps up each `every` positions."""
    steps = torch.div(positions + 1, every, rounding_mode="floor").to(torch.float64)
    return 1.0 + coef * torch.log(steps + 1.0)


def attend_with_sink(q, k, v, scale, sink):
    """q [T, H, d], k [T, G, d], v [T, G, e], sink [H]: causal softmax whose
    denominator has one more term exp(sink_h)."""
    T, H, _ = q.shape
    share = H // k.shape[1]
    causal = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for h in range(H):
        g = h // share
        s = (q[:, h] @ k[:, g].T) * scale
        s = torch.where(causal, s, torch.full_like(s, -math.inf))
        top = torch.maximum(s.amax(dim=-1), sink[h])
        e = torch.exp(s - top[:, None])
        total = e.sum(-1) + torch.exp(sink[h] - top)
        out.append((e / total[:, None]) @ v[:, g])
    return torch.stack(out, dim=1)


def attention(h, w, p, m, eps, round_to=None):
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = _r(h @ w[p + "q"].T, round_to).view(T, H, d)
    k = _r(h @ w[p + "k"].T, round_to).view(T, G, d)
    v = _r(h @ w[p + "v"].T, round_to).view(T, G, e)
    q = unit_rms(q, eps) * w[p + "q.norm"]
    k = unit_rms(k, eps) * w[p + "k.norm"]
    if m.get("q_temp") is not None:
        factor = query_temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])
        q = q * factor.to(q.dtype)[:, None, None]
    o = attend_with_sink(_r(q, round_to), _r(k, round_to), v, m["scale"], w[p + "sink"])
    return _r(_r(o, round_to).reshape(T, H * e) @ w[p + "o"].T, round_to)


# ------------------------------------------------------------------ the linear recurrence
def decayed_memory(q, k, v, decay):
    """q, k [T, H, d], v [T, H, e], decay [H]: S <- decay S + k v^T, o = S^T q."""
    T, H, d = q.shape
    S = q.new_zeros(H, d, v.shape[-1])
    rate = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    out = []
    for t in range(T):
        S = S * rate + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out)


def lightning(h, w, p, m, eps, round_to=None):
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q = silu(_r(h @ w[p + "q"].T, round_to)).view(T, H, d)
    k = silu(_r(h @ w[p + "k"].T, round_to)).view(T, H, d)
    v = silu(_r(h @ w[p + "v"].T, round_to)).view(T, H, e)
    o = decayed_memory(_r(q, round_to), _r(k, round_to), _r(v, round_to), m["decay"]).reshape(T, H * e)
    gate = torch.sigmoid(_r(h @ w[p + "g"].T, round_to))
    o = _r(unit_rms(o, eps) * w[p + "norm"] * gate, round_to)
    return _r(o @ w[p + "o"].T, round_to)


# ------------------------------------------------------------------ feed-forward
def plain_ff(h, w, p, round_to=None):
    """down(relu(up h)^2)"""
    a = _r(relu_squared(h @ w[p + "up"].T), round_to)
    return a @ w[p + "down"].T


def route(h, w, p, m):
    """(chosen ids [T, top], their weights [T, top], how far the last chosen
    one's choice score lies above the first not chosen one's)."""
    top = m["router"]["top"]
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    choice = s + w[p + "correction"]
    order = torch.argsort(choice, dim=-1, descending=True, stable=True)
    ids = order[:, :top]
    ranked = torch.gather(choice, 1, order)
    margin = ranked[:, top - 1] - ranked[:, top] if top < choice.shape[1] else torch.full((h.shape[0],), math.inf, dtype=h.dtype)
    picked = torch.gather(s, 1, ids)
    return ids, picked / (picked.sum(-1, keepdim=True) + 1e-20), margin


def routed_experts(h, w, p, m, round_to=None, margins_out=None):
    real = m["router"]["experts"]
    ids, share, margin = route(h, w, p, m)
    if margins_out is not None:
        margins_out.append(margin)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            e = int(ids[t, j])
            y = h[t] if e >= real else plain_ff(h[t:t + 1], w, f"{p}e{e}.", round_to)[0]
            out[t] += share[t, j] * y
    if m.get("shared") is not None:
        out = out + _r(plain_ff(h, w, p + "shared.", round_to), round_to)
    return _r(out, round_to)


def feed_forward(h, w, p, m, round_to=None, margins_out=None):
    if m["kind"] == "dense":
        return _r(plain_ff(h, w, p, round_to), round_to)
    return routed_experts(h, w, p, m, round_to, margins_out)


# ------------------------------------------------------------------ the model
def run_order(config):
    n = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return list(range(n))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n))


def forward(config, weights, tokens, dtype=torch.float64, round_to=None, layers_out=None, margins_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that
    receives the stream after every layer run.  ``margins_out``: a list that
    receives every routed layer run's margins (see route)."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i in run_order(config):
        layer, p = config["layers"][i], f"l{i}."
        h = _r(unit_rms(x, eps) * w[p + "norm1"], round_to)
        mixer = {"attention": attention, "lightning": lightning}[layer["type"]]
        y = mixer(h, w, p + "mix.", layer["mixer"], eps, round_to)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, p + "mlp.", layer["mlp"], round_to, margins_out)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(unit_rms(x, eps) * w["final.norm"], round_to) @ w["head"].T


def greedy(config, weights, prompt, n):
    ids = list(prompt)
    out = []
    for _ in range(n):
        nxt = int(forward(config, weights, ids)[-1].argmax())
        out.append(nxt)
        ids.append(nxt)
    return out


# ------------------------------------------------------------------ tensors
def tensor_shapes(config):
    W, V = config["width"], config["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        H, d, e = m["heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = (W,)
        if layer["type"] == "attention":
            G = m["kv_heads"]
            shapes.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * e, W), q + "o": (W, H * e),
                           q + "q.norm": (d,), q + "k.norm": (d,), q + "sink": (H,)})
        else:
            shapes.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * e, W), q + "g": (H * e, W),
                           q + "o": (W, H * e), q + "norm": (H * e,)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        f = p + "mlp."
        if mlp["kind"] == "dense":
            shapes.update({f + "up": (mlp["ff"], W), f + "down": (W, mlp["ff"])})
            continue
        F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
        for x in range(E):
            shapes.update({f"{f}e{x}.up": (F, W), f"{f}e{x}.down": (W, F)})
        total = E + mlp["router"].get("identity", 0)
        shapes.update({f + "router": (total, W), f + "correction": (total,)})
        if mlp.get("shared") is not None:
            S = mlp["shared"]["ff"]
            shapes.update({f + "shared.up": (S, W), f + "shared.down": (W, S)})
    return shapes


def random_weights(config, seed, sharp=3.0):
    """Values of bfloat16 precision (so that a folder stored in either type
    holds the same model).  Matrices N(0, 1 / fan-in) times a factor; norm
    weights of queries and keys are large enough that single keys decide a
    softmax (``sharp``: roughly the spread of the scores before the config's
    scale and temperature, over sqrt(dim)); sinks take a large part of the
    short contexts' sums; routers are wide apart."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        tail = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
        n = lambda: torch.randn(shape, generator=g)
        if tail in ("norm1", "mix.norm") or name == "final.norm":
            t = 1.0 + 0.2 * n()
        elif tail in ("mix.q.norm", "mix.k.norm"):
            t = math.sqrt(sharp) * (1.0 + 0.3 * n())
        elif tail == "mix.sink":
            t = 1.0 + 1.5 * n()
        elif tail == "mlp.correction":
            t = 0.15 * n()
        elif name == "embed":
            t = n()
        else:
            t = n() / math.sqrt(shape[1])
            if tail == "mlp.router":
                t = t * 3.0
            if tail.endswith(".o") or tail.endswith(".down"):
                t = t * 0.5
        out[name] = t.to(torch.bfloat16).to(torch.float64)
    return out
