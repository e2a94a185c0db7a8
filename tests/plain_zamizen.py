"""A plain, slow implementation of the Zamizen decoder for the tests: whole
sequences, no cache, no state carried between calls, one function per
mechanism, on the CPU in the type asked for (float64 as the yardstick).  It
shares no code with the package.

``round_to``: activations are rounded to that type (and widened again) after
every matrix product and after everything whose output feeds one, which is
where a pipeline that computes in that type rounds; everything the design
keeps 32-bit (the stream, norms, angles, scores, softmax) stays wide.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ small pieces
def _r(x, round_to):
    return x if round_to is None else x.to(round_to).to(x.dtype)


def layer_norm(x, w, b, eps):
    mean = x.mean(-1, keepdim=True)
    var = (x - mean).pow(2).mean(-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * w + b


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(u, taps):
    """u [T, C], taps [C, n] with the last column the current token's; zeros before the start."""
    T, C = u.shape
    n = taps.shape[1]
    padded = torch.cat([u.new_zeros(n - 1, C), u], dim=0)
    return sum(padded[j:j + T] * taps[:, j][None, :] for j in range(n))


def plain_rates(rot, base):
    i = torch.arange(rot // 2, dtype=torch.float64)
    return torch.as_tensor(float(base), dtype=torch.float64) ** (-2.0 * i / max(rot, 1))


def yarn_rates(rot, base, scaling):
    """(rates, factor on cosines and sines)."""
    f = plain_rates(rot, base)
    if not scaling:
        return f, 1.0

    def dim_of(t):
        return rot * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), rot - 1)
    out = []
    for i in range(rot // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(float(f[i]) / scaling["factor"] * ramp + float(f[i]) * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(scaling["factor"]) + 1.0


def turn_pairs(x, positions, rot, base):
    """x [T, heads, n]: entries (2i, 2i + 1) below ``rot`` turn by positions * base^(-2i / rot)."""
    if rot == 0:
        return x
    angle = positions.to(torch.float64)[:, None, None] * plain_rates(rot, base)[None, None, :]
    c, s = torch.cos(angle).to(x.dtype), torch.sin(angle).to(x.dtype)
    a, b = x[..., 0:rot:2], x[..., 1:rot:2]
    out = x.clone()
    out[..., 0:rot:2] = a * c - b * s
    out[..., 1:rot:2] = b * c + a * s
    return out


def turn_halves(x, positions, rot, base, scaling=None):
    """x [T, heads, n]: entries i and i + rot / 2, i < rot / 2, turn together."""
    if rot == 0:
        return x
    rates, magnitude = yarn_rates(rot, base, scaling)
    angle = positions.to(torch.float64)[:, None, None] * rates[None, None, :]
    c, s = (torch.cos(angle) * magnitude).to(x.dtype), (torch.sin(angle) * magnitude).to(x.dtype)
    h = rot // 2
    a, b = x[..., :h], x[..., h:rot]
    out = x.clone()
    out[..., :h] = a * c - b * s
    out[..., h:rot] = b * c + a * s
    return out


def softmax_attention(q, k, v, scale):
    """q [T, d], k [T, d], v [T, e]; position i sees j <= i."""
    T = q.shape[0]
    i = torch.arange(T)
    s = (q @ k.T) * scale
    s = s.masked_fill(i[None, :] > i[:, None], -math.inf)
    return torch.softmax(s, dim=-1) @ v


# ------------------------------------------------------------------ mixers
def convolved(h, w, name, round_to=None):
    """The projection with its bias, then the short convolution of every channel over time."""
    u = _r(h @ w[name].T, round_to) + w[name + ".b"][None]
    return causal_conv(u, w[name + ".conv"])


def keys_and_values(h, w, p, m, eps, positions, round_to=None):
    T, G, d, e = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = convolved(h, w, p + "k", round_to).view(T, G, d)
    v = _r(convolved(h, w, p + "v", round_to), round_to).view(T, G, e)
    k = _r(unit_rms(turn_pairs(k, positions, m["rot"]["dims"], m["rot"]["base"]), eps), round_to)
    return k, v


def attention_mixer(h, w, p, m, eps, positions, shared=None, round_to=None):
    """``shared``: another layer's (keys, values); (output, this layer's keys and values)."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = convolved(h, w, p + "q", round_to).view(T, H, d)
    q = _r(unit_rms(turn_pairs(q, positions, m["rot"]["dims"], m["rot"]["base"]), eps), round_to)
    k, v = shared if shared is not None else keys_and_values(h, w, p, m, eps, positions, round_to)
    heads = [softmax_attention(q[:, j], k[:, j // (H // G)], v[:, j // (H // G)], m["scale"]) for j in range(H)]
    o = _r(torch.stack(heads, dim=1), round_to)
    return _r(o.reshape(T, H * e) @ w[p + "o"].T, round_to) + w[p + "o.b"][None], (k, v)


def latent_mixer(h, w, p, m, eps, positions, round_to=None):
    T = h.shape[0]
    H, d, rd, e, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base, scaling = m["rot"]["base"], m["rot"].get("scaling")
    q = _r(h @ w[p + "q"].T, round_to).view(T, H, d + rd)
    down = _r(h @ w[p + "dkv"].T, round_to)
    c = _r(unit_rms(down[:, :r], eps) * w[p + "dkv.norm"][None], round_to)
    q_turned = _r(turn_halves(q[..., d:].contiguous(), positions, rd, base, scaling), round_to)
    k_turned = _r(turn_halves(down[:, r:].reshape(T, 1, rd), positions, rd, base, scaling)[:, 0], round_to)
    k_plain = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, e)
    heads = [softmax_attention(torch.cat([q[:, j, :d], q_turned[:, j]], dim=-1), torch.cat([k_plain[:, j], k_turned], dim=-1),
                               v[:, j], m["scale"]) for j in range(H)]
    o = _r(torch.stack(heads, dim=1).reshape(T, H * e), round_to)
    gate = torch.sigmoid(_r(h @ w[p + "g"].T, round_to))
    return _r(_r(o * gate, round_to) @ w[p + "o"].T, round_to)


def dense_feed_forward(h, w, p, round_to=None):
    g, u = h @ w[p + "gate"].T, h @ w[p + "up"].T
    return _r(_r(silu(g) * u, round_to) @ w[p + "down"].T, round_to)


# ------------------------------------------------------------------ the model
def forward(cfg, weights, ids, dtype=torch.float64, round_to=None, layers_out=None):
    """Logits [T, vocab] for the whole sequence ``ids``."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    ids = torch.as_tensor(ids, dtype=torch.long)
    positions = torch.arange(len(ids))
    x = w["embed"][ids]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]

        def norm(x, name):
            return layer_norm(x, w[p + name], w[p + name + ".b"], eps)

        h = _r(norm(x, "norm1"), round_to)
        if layer["type"] == "attention":
            shared = kept[m["kv_from"]] if m.get("kv_from") is not None else None
            y, kept[i] = attention_mixer(h, w, p + "mix.", m, eps, positions, shared, round_to)
        else:
            y = latent_mixer(h, w, p + "mix.", m, eps, positions, round_to)
        x = x + mult * norm(y, "norm1b")
        if layer.get("mlp"):
            y = dense_feed_forward(_r(norm(x, "norm2"), round_to), w, p + "mlp.", round_to)
            x = x + mult * norm(y, "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(layer_norm(x, w["final.norm"], w["final.norm.b"], eps), round_to) @ w["head"].T


def greedy(cfg, weights, prompt, n):
    ids, out = list(prompt), []
    for _ in range(n):
        nxt = int(forward(cfg, weights, ids)[-1].argmax())
        out.append(nxt)
        ids.append(nxt)
    return out


# ------------------------------------------------------------------ tensors
def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,), "final.norm.b": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer.get("mlp") else ()):
            shapes[p + n] = shapes[p + n + ".b"] = (W,)
        if layer["type"] == "attention":
            H, G, d, e, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            rows = {"q": H * d}
            if m.get("kv_from") is None:
                rows.update(k=G * d, v=G * e)
            for name, r in rows.items():
                shapes.update({p + "mix." + name: (r, W), p + f"mix.{name}.b": (r,), p + f"mix.{name}.conv": (r, n)})
            shapes.update({p + "mix.o": (W, H * e), p + "mix.o.b": (W,)})
        else:
            H, d, rd, e, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            shapes.update({p + "mix.q": (H * (d + rd), W), p + "mix.dkv": (r + rd, W), p + "mix.dkv.norm": (r,),
                           p + "mix.uk": (H * d, r), p + "mix.uv": (H * e, r), p + "mix.g": (H * e, W), p + "mix.o": (W, H * e)})
        if layer.get("mlp"):
            F = layer["mlp"]["ff"]
            shapes.update({p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return shapes


def random_weights(cfg, seed, sharp=3.0):
    """Values of bfloat16 precision (so that a folder stored in either type
    holds the same model).  Matrices N(0, 1 / fan-in) times a factor; those
    that make the scores of latent attention are larger, so that single keys
    decide a softmax (``sharp``: roughly the spread of the scores)."""
    g = torch.Generator().manual_seed(seed)
    latent = [layer["type"] == "latent_attention" for layer in cfg["layers"]]
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        tail = name.split(".", 1)[1] if name[0] == "l" else name
        if tail.endswith(".conv"):
            t = 0.6 * torch.randn(shape, generator=g)
        elif len(shape) == 1 and tail.endswith(".b"):
            t = 0.3 * torch.randn(shape, generator=g)
        elif len(shape) == 1:
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
            if tail in ("mix.q", "mix.uk") and latent[int(name[1:name.index(".")])]:
                t = t * math.sqrt(sharp)
        out[name] = t.to(torch.bfloat16).to(torch.float64)
    return out
