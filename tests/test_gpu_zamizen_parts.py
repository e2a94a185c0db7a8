"""Each mechanism of the Zamizen design alone, the kernel against the plain
function of tests/plain_zamizen.py in 64 bits: an output that enters the stream
through a norm of its own with the norm of the stream behind it; bias, short
convolution, turn of pairs, norm per head and cache write under every cut of a
sequence into steps (state rows used again); the latent's norm with the turned
parts of keys and queries, alone and as one launch with the queries' product;
the per-head products between wider heads and with a gate per entry."""
import math

import pytest
import torch

import plain_zamizen as pz

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def tol_of(dtype, tight=1e-5, loose=2e-2):
    return dict(atol=tight, rtol=tight) if dtype == torch.float32 else dict(atol=loose, rtol=loose)


# ------------------------------------------------------------------ norms around the addition
def plain_addend_norm(x, y, b_in, wy, by, eps_y, centered_y, w, b, eps, centered):
    def norm(v, w, b, eps, centered):
        n = pz.layer_norm(v, w, 0.0, eps) if centered else pz.unit_rms(v, eps) * w
        return n + b if b is not None else n
    if y is not None:
        x = x + norm(y + b_in if b_in is not None else y, wy, by, eps_y, centered_y)
    return x, norm(x, w, b, eps, centered)


@BOTH
@pytest.mark.parametrize("rows,W", [(1, 64), (3, 100), (5, 33), (7, 1024), (2, 2048), (150, 2048), (9, 3072), (200, 3072), (3, 5000),
                                    (2, 8192), (160, 8192), (2, 9000), (4, 4),
                                    (300, 1000), (4600, 600), (2300, 2048)])
def test_output_norm_addition_and_next_norm(rows, W, dtype):
    """Layer norms and root mean square norms in every combination, with and
    without biases, outputs as one tensor and as 1 to 5 partial sums, for all
    rows and for a list of them; a mean far from zero costs no digits."""
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(rows + W)
    rn = lambda *s: torch.randn(*s, generator=g)
    eps, eps_y = 1e-5, 1e-3
    w, b, wy, by, b_in = (1 + 0.3 * rn(W), rn(W), 1 + 0.3 * rn(W), rn(W), rn(W))
    for k, (parts, centered_y, centered, with_b, with_in) in enumerate([
            (0, True, True, True, True), (1, True, True, True, False), (2, True, True, True, True), (3, False, True, False, True),
            (4, True, False, False, False), (5, True, True, True, True), (-1, True, True, True, False), (-1, False, False, False, False)]):
        x = rn(rows, W) + 300.0 * (k == 0)
        y = None if parts < 0 else (rn(rows, W).to(dtype) if parts == 0 else rn(parts, rows, W))
        if k == 2:
            y = y + 500.0
        y64 = None if y is None else (y.double() if y.dim() == 2 else y.double().sum(0))
        bb = b if with_b else None
        bby = by if with_b else None
        bi = b_in if with_in else None
        want_x, want = plain_addend_norm(x.double(), y64, None if bi is None else bi.double(), wy.double(),
                                         None if bby is None else bby.double(), eps_y, centered_y, w.double(),
                                         None if bb is None else bb.double(), eps, centered)
        dev = lambda t: None if t is None else t.to(DEV)
        kw = dict(addend=dev(y), addend_bias=dev(bi) if y is not None else None, addend_weight=dev(wy) if y is not None else None,
                  addend_norm_bias=dev(bby) if y is not None else None, addend_eps=eps_y, addend_centered=centered_y)
        out = torch.empty(rows, W, dtype=dtype, device=DEV)
        resid = x.to(DEV)
        ops.addend_norm(out, resid, dev(w), dev(bb), eps, centered, **kw)
        loose = 1e-3 if k in (0, 2) else 3e-5          # (values of 300 and 500 carry 2^-24 of themselves)
        torch.testing.assert_close(resid.cpu(), want_x.float(), atol=loose, rtol=2e-5)
        torch.testing.assert_close(out.float().cpu(), want.float(), **tol_of(dtype, loose, 3e-2))
        # a list of rows: the stream stays
        pick = [rows - 1, 0] if rows > 1 else [0]
        some = torch.empty(len(pick), W, dtype=dtype, device=DEV)
        kept = x.to(DEV)
        ops.addend_norm(some, kept, dev(w), dev(bb), eps, centered, rows=i32(pick), **kw)
        assert torch.equal(kept.cpu(), x)
        torch.testing.assert_close(some.float().cpu(), want[pick].float(), **tol_of(dtype, loose, 3e-2))


# ------------------------------------------------------------------ bias, convolution, turn, norm, cache write
def plain_conv_turn(u, bias, taps, sizes, rot, base, unit_eps):
    """u [T, real channels]; sizes = (heads, kv_heads, d, e): q, k, v after everything."""
    H, G, d, e = sizes
    T = u.shape[0]
    y = pz.causal_conv(u + bias[None], taps)
    pos = torch.arange(T)
    q, k, v = y[:, :H * d].view(T, H, d), y[:, H * d:(H + G) * d].view(T, G, d), y[:, (H + G) * d:].view(T, G, e)
    q, k = pz.turn_pairs(q, pos, rot, base), pz.turn_pairs(k, pos, rot, base)
    if unit_eps is not None:
        q, k = pz.unit_rms(q, unit_eps), pz.unit_rms(k, unit_eps)
    return q, k, v


def padded_channels(t, sizes, hd):
    """[real channels, n] -> [padded channels, n]"""
    H, G, d, e = sizes
    out, at = [], 0
    for heads, size in ((H, d), (G, d), (G, e)):
        block = torch.zeros(heads, hd, t.shape[1], dtype=t.dtype)
        block[:, :size] = t[at:at + heads * size].view(heads, size, -1)
        out.append(block.view(heads * hd, -1))
        at += heads * size
    return torch.cat(out)


CONV_SIZES = [((4, 2, 32, 32), 16, 3), ((3, 1, 24, 10), 8, 4), ((2, 2, 64, 48), 64, 2), ((4, 1, 20, 28), 20, 3), ((2, 1, 128, 128), 32, 4),
              ((1, 1, 80, 96), 0, 3), ((2, 1, 16, 16), 16, 1), ((2, 2, 48, 48), 10, 6), ((1, 1, 200, 176), 50, 3), ((1, 1, 300, 40), 8, 17),
              ((6, 3, 9, 16), 8, 2), ((33, 2, 16, 16), 16, 3)]


@BOTH
@pytest.mark.parametrize("unit", [True, False])
@pytest.mark.parametrize("sizes,rot,taps", CONV_SIZES)
def test_convolution_turn_norm_and_store_under_every_cut(sizes, rot, taps, unit, dtype):
    """Four requests in cuts of unequal sizes (down to one token, shorter than
    the taps, over the kernel's tiles) on state rows that others left full;
    queries, stored keys and values equal those of the whole sequences."""
    run_conv_turn(sizes, rot, taps, unit, dtype, [[1, 1, 2, 1, 33, 1, 31], [2, 1, 1, 1], [40, 1], [16, 2]], [2, 0, 4, 3])


@BOTH
@pytest.mark.parametrize("sizes,rot,taps", [((32, 8, 64, 64), 32, 4), ((24, 4, 80, 64), 64, 3)])
def test_the_same_with_enough_tokens_for_whole_tiles_to_a_block(sizes, rot, taps, dtype):
    run_conv_turn(sizes, rot, taps, True, dtype, [[450, 3, 467], [1, 2, 330], [18, 1, 29]], [4, 2, 0])


def run_conv_turn(sizes, rot, taps, unit, dtype, cuts, slots_of):
    from lyapunov_engine_b200 import ops
    H, G, d, e = sizes
    hd = (max(d, e) + 15) // 16 * 16
    base, eps, page = 3e3, 1e-5, 8
    g = torch.Generator().manual_seed(H * 100 + d + taps)
    real = H * d + G * (d + e)
    w, bias = 0.6 * torch.randn(real, taps, generator=g), 0.5 * torch.randn(real, generator=g)
    lens = [sum(c) for c in cuts]
    u = [torch.randn(n, real, generator=g).to(dtype) for n in lens]
    want = [plain_conv_turn(x.double(), bias.double(), w.double(), sizes, rot, base, eps if unit else None) for x in u]
    wide = [padded_channels(x.t().contiguous(), sizes, hd).t().contiguous() for x in u]
    C = (H + 2 * G) * hd
    w_dev = padded_channels(w, sizes, hd).t().contiguous().to(DEV)
    bias_dev = padded_channels(bias[:, None], sizes, hd).view(-1).contiguous().to(DEV)
    R = len(cuts)
    state = torch.full((6, max(taps - 1, 1), C), 7.0, device=DEV) if taps > 1 else None
    per = (max(lens) + page - 1) // page
    pages = R * per + 1
    order = torch.randperm(pages - 1, generator=g).view(R, per).to(torch.int32)
    kc = torch.full((pages, G, page, hd), 3.0, dtype=dtype, device=DEV)
    vc = torch.full_like(kc, 3.0)
    rates = pz.plain_rates(max(rot, 2), base).to(DEV)
    status = ops.new_status(DEV)
    at = [0] * R
    got_q = [[] for _ in range(R)]
    for step in range(max(map(len, cuts))):
        live = [r for r in (2, 0, 3, 1) if r < R and step < len(cuts[r])]
        q_lens = [cuts[r][step] for r in live]
        src = torch.cat([wide[r][at[r]:at[r] + n] for r, n in zip(live, q_lens)])
        src = torch.cat([src, torch.zeros(src.shape[0], 8, dtype=dtype)], dim=1).to(DEV)     # (rows wider than the channels)
        if taps > 1:
            ops.zero_fresh_state(state, i32(slots_of[r] for r in live), i32(at[r] for r in live), len(live))
        positions = i32(p for r, n in zip(live, q_lens) for p in range(at[r], at[r] + n))
        table = order[live].to(DEV).contiguous()
        cu = i32([0] + torch.tensor(q_lens).cumsum(0).tolist())
        if all(n == 1 for n in q_lens):
            tiles = (None, None, len(live))
        else:
            pairs = [(b, s) for b, n in enumerate(q_lens) for s in range(0, n, ops.SHORT_CONV_TILE)]
            tiles = (i32(b for b, _ in pairs), i32(s for _, s in pairs), len(pairs))
        q_out = torch.full((src.shape[0], H * hd), 5.0, dtype=dtype, device=DEV)
        ops.conv_turn_store(q_out, src, bias_dev, w_dev, state, i32(slots_of[r] for r in live), cu, *tiles, rates, rot, 1.0,
                            eps if unit else None, d, kc, vc, positions, table, H, G, hd, page, True, status)
        o = 0
        for r, n in zip(live, q_lens):
            got_q[r].append(q_out[o:o + n].float().cpu().view(n, H, hd))
            o += n
            at[r] += n
    ops.check_status(status)
    tol = tol_of(dtype, 3e-5)
    for r, n in enumerate(lens):
        q = torch.cat(got_q[r])
        torch.testing.assert_close(q[..., :d], want[r][0].float(), **tol)
        assert float(q[..., d:].abs().sum()) == 0.0
        pg = order[r, torch.arange(n) // page].long()
        keys, values = (p[pg.to(DEV), :, (torch.arange(n) % page).to(DEV)].float().cpu() for p in (kc, vc))
        torch.testing.assert_close(keys[..., :d], want[r][1].float(), **tol)
        torch.testing.assert_close(values[..., :e], want[r][2].float(), **tol)
        assert float(keys[..., d:].abs().sum()) == 0.0 == float(values[..., e:].abs().sum())
        if taps > 1:
            tail = torch.cat([torch.zeros(taps, C), wide[r].float() + bias_dev.cpu()[None]])[-(taps - 1):]
            torch.testing.assert_close(state[slots_of[r]].cpu(), tail, atol=1e-6, rtol=1e-6)
    if taps > 1:
        assert float(state[1].min()) == 7.0 == float(state[5].min())                 # rows of no request stay as they are


@BOTH
@pytest.mark.parametrize("taps", [1, 3, 5])
def test_queries_alone_rows_of_no_request_and_a_page_outside_the_pool(taps, dtype):
    """A layer without keys: the same queries, nothing stored.  Rows with slot
    -1 see zeros before them and keep nothing.  A page outside the pool is
    refused, not followed."""
    from lyapunov_engine_b200 import ops
    H, hd, rot, T = 3, 32, 16, 4
    g = torch.Generator().manual_seed(taps)
    u = torch.randn(T, H * hd, generator=g).to(dtype)
    w = torch.randn(taps, H * hd, generator=g)
    state = torch.randn(3, max(taps - 1, 1), H * hd, generator=g).to(DEV) if taps > 1 else None
    before = state.clone() if taps > 1 else None
    rates = pz.plain_rates(rot, 100.0).to(DEV)
    status = ops.new_status(DEV)
    table = torch.zeros(T, 2, dtype=torch.int32, device=DEV)
    q = torch.empty(T, H * hd, dtype=dtype, device=DEV)
    slots = i32([1, -1, 0, -1])
    pos = i32([9, 4, 0, 1000003])
    ops.conv_turn_store(q, u.to(DEV), None, w.to(DEV), state, slots, i32(range(T + 1)), None, None, T, rates, rot, 1.25, 1e-6, hd,
                        None, None, pos, table, H, 0, hd, 8, False, status)
    ops.check_status(status)
    for t in range(T):
        past = torch.zeros(taps - 1, H * hd, dtype=torch.float64)
        if taps > 1 and int(slots[t]) >= 0:
            past = before[int(slots[t])].double().cpu()
        y = (torch.cat([past, u[t:t + 1].double()]) * w.double()).sum(0).view(1, H, hd)
        turned = pz.turn_pairs(y, pos[t:t + 1].cpu().long(), rot, 100.0)
        turned[..., :rot] *= 1.25
        want = pz.unit_rms(turned, 1e-6)
        torch.testing.assert_close(q[t].float().cpu().view(1, H, hd), want.float(), **tol_of(dtype, 2e-5))
    if taps > 1:
        assert torch.equal(state[2], before[2])
        for t in (0, 2):
            row = state[int(slots[t])].cpu()
            torch.testing.assert_close(row, torch.cat([before[int(slots[t])].cpu()[1:], u[t:t + 1].float()]))
    kc = torch.zeros(3, 1, 8, hd, dtype=dtype, device=DEV)
    q1 = torch.empty(T, hd, dtype=dtype, device=DEV)
    table.fill_(77)
    st = state if taps > 1 else None
    ops.conv_turn_store(q1, u.to(DEV), None, w.to(DEV), st, slots, i32(range(T + 1)), None, None, T, rates, rot, 1.0, None, hd, kc,
                        kc.clone(), i32([0, 1, 2, 3]), table, 1, 1, hd, 8, True, status)
    with pytest.raises(ops.KernelError):
        ops.check_status(status)
    assert float(kc.float().abs().max()) == 0.0


# ------------------------------------------------------------------ latent attention's turned parts and products
LATENT_SIZES = [(3, 24, 8, 48), (8, 32, 16, 112), (2, 16, 6, 20), (4, 40, 24, 72), (5, 7, 10, 33), (2, 64, 64, 64)]


@BOTH
@pytest.mark.parametrize("rows", [1, 9, 32, 70])
@pytest.mark.parametrize("heads,d,rot,rank", LATENT_SIZES)
def test_latent_norm_turned_parts_and_the_queries_way(heads, d, rot, rank, rows, dtype):
    """The latent's norm, the keys' turned part and the cache write; the
    queries' turned parts behind their products in the latent space, in the
    launches of many rows and, where it exists, in the one of few rows."""
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(heads + rank + rows)
    padded = (rank + rot + 15) // 16 * 16
    qh = d + rot
    col = (heads * qh + 7) // 8 * 8
    src = torch.randn(rows, (col + rank + rot + 7) // 8 * 8 + 8, generator=g).to(dtype)
    w_into = (torch.randn(heads, rank, d, generator=g) / math.sqrt(d)).to(dtype)
    weight = 1.0 + 0.3 * torch.randn(rank, generator=g)
    scaling = {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 0.5}
    rates, magnitude = pz.yarn_rates(rot, 500.0, scaling)
    page, eps = 4, 1e-5
    first = 5
    pages = (first + rows) // page + 2
    positions = torch.arange(first, first + rows, dtype=torch.int32)
    table = torch.randperm(pages, generator=g).to(torch.int32).view(1, -1)
    order = torch.arange(rot).view(2, rot // 2).t().reshape(-1)             # pairs from halves
    back = torch.argsort(order)
    q = src[:, :heads * qh].double().view(rows, heads, qh)
    want_q = torch.einsum("thk,hnk->thn", q[..., :d], w_into.double())
    want_turn = pz.turn_halves(q[..., d:][..., back], positions.long(), rot, 500.0, scaling)[..., order]
    c = src[:, col:col + rank].double()
    want_c = pz.unit_rms(c, eps) * weight.double()[None]
    kr = src[:, col + rank:col + rank + rot].double().view(rows, 1, rot)
    want_kr = pz.turn_halves(kr[..., back], positions.long(), rot, 500.0, scaling)[..., order][:, 0]
    dev = src.to(DEV)
    place = (positions.to(DEV), i32([0] * rows), table.to(DEV), page)
    status = ops.new_status(DEV)
    forms = ["many"] + (["few"] if ops.latent_prepare_applies(dev, d, rot) else [])
    assert ("few" in forms) == (rows <= 32 and d % 8 == 0 and rot % 8 == 0) or dtype == torch.float32
    for form in forms:
        cache = torch.full((pages + 1, 1, page, padded), 3.0, dtype=dtype, device=DEV)
        q_latent = torch.full((rows, heads * padded), 4.0, dtype=dtype, device=DEV)
        if form == "many":
            ops.latent_rope_store(dev, col, rank, rot, padded, weight.to(DEV), eps, rates.to(DEV), cache, *place, status,
                                  magnitude=magnitude, queries=(d, qh, heads, q_latent))
            ops.gemm_heads(q_latent, dev[:, :heads * qh], w_into.to(DEV), a_head=qh, out_head=padded)
        else:
            ops.latent_prepare(q_latent, dev, w_into.to(DEV), col, rank, weight.to(DEV), eps, cache, *place, status, rot=rot,
                               rates=rates.to(DEV), magnitude=magnitude)
        ops.check_status(status)
        got = q_latent.float().cpu().view(rows, heads, padded)
        torch.testing.assert_close(got[..., :rank], want_q.float(), **tol_of(dtype, 2e-5))
        torch.testing.assert_close(got[..., rank:rank + rot], want_turn.float(), **tol_of(dtype, 2e-5))
        assert float(got[..., rank + rot:].abs().sum()) == 0.0
        for t in range(rows):
            p = int(positions[t])
            row = cache[int(table[0, p // page]), 0, p % page].float().cpu()
            torch.testing.assert_close(row[:rank], want_c[t].float(), **tol_of(dtype, 2e-5))
            torch.testing.assert_close(row[rank:rank + rot], want_kr[t].float(), **tol_of(dtype, 2e-5))
            assert float(row[rank + rot:].abs().sum()) == 0.0
        assert float(cache[pages].float().min()) == 3.0


@BOTH
@pytest.mark.parametrize("rows,heads,N,K", [(1, 4, 32, 128), (7, 3, 20, 48), (40, 2, 70, 33), (32, 5, 1, 16), (100, 4, 48, 64)])
def test_a_gate_per_entry_in_the_per_head_products(rows, heads, N, K, dtype):
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(rows + N)
    a = torch.randn(rows, heads * K, generator=g).to(dtype)
    w = (torch.randn(heads, N, K, generator=g) / math.sqrt(K)).to(dtype)
    gate = (2 * torch.randn(rows, heads * N + 3, generator=g)).to(dtype)
    want = torch.einsum("thk,hnk->thn", a.double().view(rows, heads, K), w.double())
    want = want * torch.sigmoid(gate[:, 2:2 + heads * N].double().view(rows, heads, N))
    out = torch.empty(rows, heads * N, dtype=dtype, device=DEV)
    ops.gemm_heads(out, a.to(DEV), w.to(DEV), gate.to(DEV)[:, 2:2 + heads * N])
    torch.testing.assert_close(out.float().cpu().view(rows, heads, N), want.float(), **tol_of(dtype))
