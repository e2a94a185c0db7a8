"""Each mechanism of the Zuzenex design alone, the kernel against a plain
function in 64 bits (the building blocks of tests/plain_zuzenex.py and the
recurrence written out here): lightning attention token by token and over
chunks under every cut of a sequence into steps, with state rows used again and
a far token that decides; sinks on all attention kernels with scores made so
that the sink matters; the norm per head with the query temperature and the
cache write; two outputs that enter the stream beside one another in the norm's
kernel; the norm over all heads at once; products with relu squared
or silu on some of their columns; the router's corrected choice; experts without a gate and identity
experts."""
import math

import pytest
import torch

import plain_zuzenex as pz

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def tiles(q_lens, size, only=None):
    req, q0 = [], []
    for b, n in enumerate(q_lens):
        if only is not None and b not in only:
            continue
        for s in range(0, n, size):
            req.append(b)
            q0.append(s)
    return i32(req), i32(q0), len(req)


def tol_of(dtype, tight=2e-5, loose=2e-2):
    return dict(atol=tight, rtol=tight) if dtype == torch.float32 else dict(atol=loose, rtol=loose)


# ------------------------------------------------------------------ lightning attention
def run_in_cuts(seqs, cuts, state_rows, H, d, e, decay, dtype, chunks, poison=7.0):
    """Feeds sequences (rows q | k | v before silu) in their cuts, the live
    requests of a step as one batch; requests take the lowest free state row
    and give it back when they end.  Returns their outputs and the last states."""
    from lyapunov_engine_b200 import ops
    parts, powers = ops.lightning_tables(decay, DEV)
    state = torch.full((state_rows + 1, H, e, d), poison, device=DEV)     # (the last row belongs to nobody)
    q_col, k_col, v_col = 0, H * d, 2 * H * d
    free, slot_of, at = list(range(state_rows)), {}, [0] * len(seqs)
    got, last = [[] for _ in seqs], {}
    seg = ops.lightning_segment()
    step = 0
    while any(step < len(c) for c in cuts):
        live = [r for r in range(len(seqs)) if step < len(cuts[r])]
        for r in live:
            if r not in slot_of:
                slot_of[r] = free.pop(0)
                state[slot_of[r]].zero_()
        q_lens = [cuts[r][step] for r in live]
        rows = torch.cat([seqs[r][at[r]:at[r] + n] for r, n in zip(live, q_lens)]).to(dtype).to(DEV)
        ops.activate(rows[:, :v_col + H * e], rows[:, :v_col + H * e], ops.ACT_SILU)
        out = torch.full((rows.shape[0], H * e), -5.0, device=DEV)
        cu, slots = i32([0] + torch.tensor(q_lens).cumsum(0).tolist()), i32(slot_of[r] for r in live)
        multi = [b for b, n in enumerate(q_lens) if n > 1]
        single = [b for b, n in enumerate(q_lens) if n == 1]
        if chunks and multi:
            # the order of a step's list: by the keys a tile of attention sees, the requests' segments between one another
            listed = sorted(((b, s) for b in multi for s in range(0, q_lens[b], seg)), key=lambda x: at[live[x[0]]] + x[1])
            tr, tq, n = i32(b for b, _ in listed), i32(s for _, s in listed), len(listed)
            scratch = torch.full((n, H, e, d), 3.0, device=DEV) if n > len(multi) else None
            ops.lightning_chunks(out, rows, q_col, k_col, v_col, powers, state, scratch, slots, cu, tr, tq, n, H, d, e)
            if single:
                ops.lightning_scan(out, rows, q_col, k_col, v_col, parts, state, slots, cu, len(single), H, d, e,
                                   requests=i32(single), single=True)
        else:
            ops.lightning_scan(out, rows, q_col, k_col, v_col, parts, state, slots, cu, len(live), H, d, e,
                               single=max(q_lens) == 1)
        t0 = 0
        for r, n in zip(live, q_lens):
            got[r].append(out[t0:t0 + n].double().cpu())
            t0 += n
            at[r] += n
            if at[r] == seqs[r].shape[0]:
                last[r] = state[slot_of[r]].double().cpu()
                free.append(slot_of.pop(r))
        step += 1
    assert bool((state[-1] == poison).all())
    return [torch.cat(o) for o in got], last


def lightning_reference(rows, H, d, e, decay, dtype):
    act = lambda z: pz.silu(z).to(dtype).double()
    q = act(rows[:, :H * d].double()).view(-1, H, d)
    k = act(rows[:, H * d:2 * H * d].double()).view(-1, H, d)
    v = act(rows[:, 2 * H * d:2 * H * d + H * e].double()).view(-1, H, e)
    T = rows.shape[0]
    S = torch.zeros(H, d, e, dtype=torch.float64)
    rate = torch.tensor(decay, dtype=torch.float64)[:, None, None]
    out = []
    for t in range(T):
        S = S * rate + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out).reshape(T, H * e), S.transpose(1, 2)


SHAPES = [
    # heads, dim, vdim, decays
    (2, 16, 16, [0.3, 0.97]),
    (3, 40, 72, [0.0, 0.9, 0.999]),            # sizes that are padded; a decay of 0 remembers nothing
    (1, 128, 128, [0.995]),
    (2, 96, 24, [1.0, 0.6]),                   # a decay of 1 forgets nothing
    (2, 13, 9, [0.8, 0.99]),                   # no 16-byte pieces
    (1, 64, 200, [0.98]),
]
LENS = (700, 70, 1, 531)
CUTS = [((700,), (70,), (1,), (531,)),
        ((1, 2, 61, 64, 65, 257, 250), (2,) * 35, (1,), (128, 1, 2, 400)),
        ((256, 256, 188), (1,) * 70, (1,), (463, 1, 1, 66)),
        ((513, 1, 1, 185), (64, 1, 5), (1,), (3, 528))]


@pytest.mark.parametrize("cut", range(len(CUTS)))
@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: f"{s[0]}x{s[1]}x{s[2]}")
@pytest.mark.parametrize("form", ["scan32", "scan16", "chunks"])
def test_lightning_under_cuts(form, shape, cut):
    H, d, e, decay = shape
    dtype = torch.float32 if form == "scan32" else torch.bfloat16
    g = torch.Generator().manual_seed(d + e)
    width = (2 * H * d + H * e + 7) // 8 * 8
    seqs = [torch.randn(n, width, generator=g).to(dtype).float() for n in LENS]
    # two state rows for the four requests where the cuts leave room: rows are used again
    got, last = run_in_cuts(seqs, CUTS[cut], 4, H, d, e, decay, dtype, chunks=form == "chunks")
    for r, rows in enumerate(seqs):
        want, S = lightning_reference(rows, H, d, e, decay, dtype)
        size = float(want.abs().max())
        # (the chunked form's products keep 16 bits of the 32-bit operands)
        tol = 2e-5 if form != "chunks" else 6e-5
        torch.testing.assert_close(got[r] / size, want / size, atol=tol, rtol=0)
        torch.testing.assert_close(last[r] / S.abs().max(), S / S.abs().max(), atol=tol, rtol=0)


def test_lightning_rows_are_used_again():
    """Six requests one after the other on two state rows, each starting in a
    row that holds another's state."""
    H, d, e, decay = 2, 32, 48, [0.9, 0.998]
    g = torch.Generator().manual_seed(1)
    lens = (300, 5, 66, 129, 2, 40)
    seqs = [torch.randn(n, 2 * H * d + H * e, generator=g).to(torch.bfloat16).float() for n in lens]
    for r in range(0, 6, 2):
        pair = [seqs[r], seqs[r + 1]]
        cuts = ((lens[r] - 1, 1), (1, lens[r + 1] - 1))
        got, _ = run_in_cuts(pair, cuts, 2, H, d, e, decay, torch.bfloat16, chunks=True, poison=1e3)
        for o, rows in zip(got, pair):
            want, _ = lightning_reference(rows, H, d, e, decay, torch.bfloat16)
            torch.testing.assert_close(o / want.abs().max(), want / want.abs().max(), atol=6e-5, rtol=0)


@pytest.mark.parametrize("chunks", [False, True])
def test_a_far_token_decides_through_the_state(chunks):
    """One loud key and value at position 3; hundreds of tokens on, a query
    that matches it gives that value, through the state alone, whatever the cut
    (chunk and segment borders lie between)."""
    H, d, e, decay = 1, 16, 16, [0.999]
    T = 600
    rows = torch.full((T, 48), -20.0)                  # silu(-20): next to nothing
    rows[3, 16], rows[3, 32:48] = 30.0, torch.arange(1.0, 17.0)
    rows[T - 1, 0] = 5.0
    rows = rows.to(torch.bfloat16).float()
    want, _ = lightning_reference(rows, H, d, e, decay, torch.bfloat16)
    assert float(want[T - 1].abs().min()) > 50 * float(want[:3].abs().max() + 1e-3)
    for cuts in ((T,), (4, T - 4), (256, 256, 88), (2, 62, 1, 300, 234, 1), (T - 1, 1)):
        got, _ = run_in_cuts([rows], (cuts,), 1, H, d, e, decay, torch.bfloat16, chunks)
        torch.testing.assert_close(got[0][T - 1], want[T - 1], atol=1e-4 * float(want[T - 1].max()), rtol=1e-4)


def test_requests_without_a_state_row_leave_everything_alone():
    """Slot -1 (padding of a fixed-shape step): zeros out, no state touched."""
    from lyapunov_engine_b200 import ops
    H, d, e = 2, 16, 24
    parts, _ = ops.lightning_tables([0.9, 0.5], DEV)
    state = torch.full((3, H, e, d), 4.0, device=DEV)
    rows = torch.randn(4, 2 * H * d + H * e, device=DEV).to(torch.bfloat16)
    out = torch.full((4, H * e), 9.0, device=DEV)
    ops.lightning_scan(out, rows, 0, H * d, 2 * H * d, parts, state, i32([-1, -1, -1, -1]), i32([0, 1, 2, 3, 4]), 4, H, d, e, single=True)
    assert float(out.abs().max()) == 0.0 and bool((state == 4.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 520, 1000, 2048, 6000])
def test_one_norm_and_a_gate_over_all_heads(width, dtype):
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(width)
    T = 5
    o, w = 3 * torch.randn(T, width, generator=g), 1 + 0.2 * torch.randn(width, generator=g)
    gate = torch.randn(T, width + 8, generator=g).to(dtype)
    out = torch.zeros(T, width, dtype=dtype, device=DEV)
    for sigmoid in (True, False):
        ops.head_norm_gate(out, o.to(DEV), gate.to(DEV)[:, 8:], w.to(DEV), 1e-5, 1, width, sigmoid=sigmoid, out_scale=0.7)
        z = gate.double()[:, 8:]
        want = pz.unit_rms(o.double(), 1e-5) * w.double() * (torch.sigmoid(z) if sigmoid else pz.silu(z)) * 0.7
        torch.testing.assert_close(out.double().cpu(), want, **tol_of(dtype))


# ------------------------------------------------------------------ attention with a sink
def build_attention(dtype, nh, nkv, hd, page, q_lens, ctx_before, seed, scale, sink):
    g = torch.Generator().manual_seed(seed)
    B, T = len(q_lens), sum(q_lens)
    most = max(c + n for c, n in zip(ctx_before, q_lens))
    per = (most + page - 1) // page
    perm = torch.randperm(B * per + 3, generator=g)
    table = torch.zeros(B, per, dtype=torch.int32)
    k_cache, v_cache = (torch.randn(B * per + 4, nkv, page, hd, generator=g).to(dtype) for _ in range(2))
    q = torch.randn(T, nh * hd, generator=g).to(dtype)
    want = torch.zeros(T, nh * hd, dtype=torch.float64)
    t0 = 0
    for b in range(B):
        table[b] = perm[b * per:(b + 1) * per].to(torch.int32)
        n = ctx_before[b] + q_lens[b]
        at = torch.arange(n)
        k = k_cache[table[b][at // page].long(), :, at % page].double()
        v = v_cache[table[b][at // page].long(), :, at % page].double()
        # one sequence whose first tokens' queries are of no interest
        qq = torch.zeros(n, nh, hd, dtype=torch.float64)
        qq[ctx_before[b]:] = q[t0:t0 + q_lens[b]].double().view(-1, nh, hd)
        full = pz.attend_with_sink(qq, k, v, scale, sink.double())
        want[t0:t0 + q_lens[b]] = full[ctx_before[b]:].reshape(q_lens[b], nh * hd)
        t0 += q_lens[b]
    return dict(q=q.to(DEV), k=k_cache.to(DEV), v=v_cache.to(DEV), table=table.to(DEV),
                cu=i32([0] + torch.tensor(q_lens).cumsum(0).tolist()), ctx=i32(ctx_before), want=want, T=T)


SINKS = [
    # nh, nkv, hd, page, q_lens, ctx_before, scale, sinks (cycled over the heads)
    (4, 2, 16, 4, [5, 1, 17, 1], [0, 9, 30, 0], 0.4, [0.0, 3.0, -4.0, 1.0]),
    (6, 2, 64, 16, [200, 1, 1, 130, 1], [0, 120, 2, 150, 700], 0.11, [2.0, 5.0, -1.0, 7.0, 0.5, 90.0]),
    (8, 2, 32, 8, [33, 1, 1, 2], [100, 69, 0, 300], 0.3, [1.0, -90.0, 4.0]),
    (2, 1, 128, 32, [140, 1], [120, 513], 0.09, [4.0, 6.0]),
    (3, 3, 80, 2, [9, 1], [30, 77], 0.1, [0.0, 5.0, -2.0]),
    (20, 1, 48, 16, [3, 1], [40, 300], 0.2, [1.0, 6.0]),          # more heads to a key head than a tile has rows
]


def sinks_of(case):
    return torch.tensor([case[7][h % len(case[7])] for h in range(case[0])], dtype=torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", SINKS, ids=lambda c: f"hd{c[2]}")
def test_a_sink_on_the_32_bit_pipes(case, dtype):
    from lyapunov_engine_b200 import ops
    nh, nkv, hd, page, q_lens, ctx_before, scale, _ = case
    sink = sinks_of(case)
    c = build_attention(dtype, nh, nkv, hd, page, q_lens, ctx_before, hd, scale, sink)
    out = torch.zeros(c["T"], nh * hd, dtype=dtype, device=DEV)
    status = ops.new_status(DEV)
    tr, tq, n = tiles(q_lens, 16)
    ops.attention_generic(out, c["q"], c["q"].stride(0), c["k"], c["v"], c["table"], c["cu"], c["ctx"], tr, tq, n, nh, nkv, hd,
                          page, 0, scale, status, sink=sink.to(DEV))
    ops.check_status(status)
    torch.testing.assert_close(out.double().cpu(), c["want"], **tol_of(dtype, tight=1e-4))
    # without it the result is another one
    plain = torch.zeros_like(out)
    ops.attention_generic(plain, c["q"], c["q"].stride(0), c["k"], c["v"], c["table"], c["cu"], c["ctx"], tr, tq, n, nh, nkv,
                          hd, page, 0, scale, status)
    assert float((plain.double().cpu() - c["want"]).abs().max()) > 0.2


@pytest.mark.parametrize("splits", [1, 2, 5, 11])
@pytest.mark.parametrize("case", SINKS, ids=lambda c: f"hd{c[2]}")
def test_a_sink_on_the_tensor_cores(case, splits):
    """Requests with several tokens on the mma.sync and (where it exists) the
    tcgen05 prefill kernel, single tokens on the split-key decode kernel: one
    split, splits merged by a cluster, more splits than a cluster merges; the
    sink must count once."""
    from lyapunov_engine_b200 import ops
    nh, nkv, hd, page, q_lens, ctx_before, scale, _ = case
    sink = sinks_of(case)
    dtype = torch.bfloat16
    c = build_attention(dtype, nh, nkv, hd, page, q_lens, ctx_before, hd + 1, scale, sink)
    status = ops.new_status(DEV)
    multi = [b for b, n in enumerate(q_lens) if n > 1]
    single = [b for b, n in enumerate(q_lens) if n == 1]
    prefills = [ops.attention_prefill_bf16]
    if ops.attention_tc_available(hd, page):
        prefills.append(ops.attention_prefill_tc_bf16)
    req, q0, n = tiles(q_lens, 128, only=multi)
    for prefill in prefills:
        out = torch.zeros(c["T"], nh * hd, dtype=dtype, device=DEV)
        prefill(out, c["q"], c["q"].stride(0), c["k"], c["v"], c["table"], c["cu"], c["ctx"], req, q0, n, nh, nkv, hd, page, 0,
                scale, status, sink=sink.to(DEV))
        floats = ops.attention_decode_scratch_floats(hd, len(single), nh, splits)
        scratch = torch.zeros(max(floats, 1), device=DEV)
        ops.attention_decode_bf16(out, scratch, c["q"], c["q"].stride(0), c["k"], c["v"], c["table"], c["cu"], c["ctx"],
                                  i32(single), len(single), nh, nkv, hd, page, 0, scale, splits, status, sink=sink.to(DEV))
        ops.check_status(status)
        torch.testing.assert_close(out.double().cpu(), c["want"], atol=2e-2, rtol=2e-2)


# ------------------------------------------------------------------ norm per head, query temperature, cache write
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,real,padded,page,temp", [(4, 2, 16, 16, 8, (0.4, 7)), (6, 3, 40, 48, 16, (0.25, 1)),
                                                                 (2, 1, 11, 16, 4, None), (3, 3, 18, 18, 2, (1.5, 64)),
                                                                 (8, 1, 128, 128, 32, (0.1, 5))])
def test_head_norm_temperature_and_store(heads, kv_heads, real, padded, page, temp, dtype):
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(real)
    positions = [0, 1, 5, 6, 7, 62, 63, 64, 300, 4097]
    T, eps = len(positions), 1e-5
    width = (heads + 2 * kv_heads) * padded
    rows = torch.zeros(T, heads + 2 * kv_heads, padded)
    rows[:, :, :real] = 2 * torch.randn(T, heads + 2 * kv_heads, real, generator=g)
    rows = rows.view(T, width).to(dtype)
    wq, wk = torch.zeros(padded), torch.zeros(padded)
    wq[:real], wk[:real] = 1 + 0.3 * torch.randn(real, generator=g), 1 + 0.3 * torch.randn(real, generator=g)
    per = 4097 // page + 1
    table = torch.arange(per, dtype=torch.int32).flip(0).view(1, -1)
    k_cache, v_cache = (torch.full((per + 1, kv_heads, page, padded), 5.0, dtype=dtype, device=DEV) for _ in range(2))
    x = rows.clone().to(DEV)
    status = ops.new_status(DEV)
    ops.rope_norm_store(x, k_cache, v_cache, None, i32(positions), i32([0] * T), table.to(DEV), heads, kv_heads, padded, 0, 0,
                        eps, real, page, True, False, status, w_q=wq.to(DEV), w_k=wk.to(DEV), temperature=temp, store_values=True)
    ops.check_status(status)
    r = rows.double().view(T, -1, padded)[:, :, :real]
    factor = torch.ones(T, dtype=torch.float64)
    if temp:
        factor = pz.query_temperature(torch.tensor(positions), *temp)
    want_q = pz.unit_rms(r[:, :heads], eps) * wq[:real].double() * factor[:, None, None]
    want_k = pz.unit_rms(r[:, heads:heads + kv_heads], eps) * wk[:real].double()
    got = x.double().cpu().view(T, -1, padded)
    torch.testing.assert_close(got[:, :heads, :real], want_q, **tol_of(dtype))
    pages, places = table[0][torch.tensor(positions) // page].long(), torch.tensor(positions) % page
    torch.testing.assert_close(k_cache.double().cpu()[pages, :, places][:, :, :real], want_k, **tol_of(dtype))
    assert torch.equal(v_cache.cpu()[pages, :, places], rows.view(T, -1, padded)[:, heads + kv_heads:])
    assert float(got[:, :heads, real:].abs().sum()) == 0.0 and int((k_cache.cpu() != 5.0).any(-1).sum()) == T * kv_heads
    # a layer that reads another's cache: queries only
    y = rows.clone().to(DEV)
    ops.rope_norm_store(y, None, None, None, i32(positions), i32([0] * T), table.to(DEV), heads, kv_heads, padded, 0, 0, eps,
                        real, page, False, False, status, w_q=wq.to(DEV), w_k=wk.to(DEV), temperature=temp, store_values=True)
    assert torch.equal(y.view(T, -1, padded)[:, :heads], x.view(T, -1, padded)[:, :heads])
    assert torch.equal(y.cpu().view(T, -1, padded)[:, heads:], rows.view(T, -1, padded)[:, heads:])


# ------------------------------------------------------------------ two outputs side by side into the stream
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("parts", [(0, 0), (3, 0), (0, 2), (1, 4)])
@pytest.mark.parametrize("width", [96, 101, 2048, 9000])
def test_two_addends_in_the_norms_kernel(width, parts, dtype):
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(width)
    T = 4
    resid, w = torch.randn(T, width, generator=g), 1 + 0.1 * torch.randn(width, generator=g)
    ys = [torch.randn(p, T, width, generator=g) if p else torch.randn(T, width, generator=g).to(dtype) for p in parts]
    total = resid.double() + sum(y.double().sum(0) if y.dim() == 3 else y.double() for y in ys)
    want = pz.unit_rms(total, 1e-5) * w.double()
    r, out = resid.clone().to(DEV), torch.zeros(T, width, dtype=dtype, device=DEV)
    ops.rmsnorm_pair(out, None, r, w.to(DEV), None, 1e-5, addend=ys[0].to(DEV), addend2=ys[1].to(DEV))
    torch.testing.assert_close(r.double().cpu(), total, atol=1e-5, rtol=1e-5)
    torch.testing.assert_close(out.double().cpu(), want, **tol_of(dtype))
    r2, out2 = resid.clone().to(DEV), torch.zeros(2, width, dtype=dtype, device=DEV)
    ops.rmsnorm_pair(out2, None, r2, w.to(DEV), None, 1e-5, addend=ys[0].to(DEV), addend2=ys[1].to(DEV), rows=i32([3, 1]))
    torch.testing.assert_close(out2.double().cpu(), want[[3, 1]], **tol_of(dtype))
    assert torch.equal(r2.cpu(), resid)


# ------------------------------------------------------------------ relu squared
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,inner", [(1, 64, 48), (7, 128, 96), (20, 256, 200), (40, 64, 72), (300, 192, 520), (5, 50, 33),
                                             (600, 512, 1024)])
def test_relu_squared_in_the_products_epilogue(rows, width, inner, dtype):
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(rows)
    x, w = torch.randn(rows, width, generator=g).to(dtype), (torch.randn(inner, width, generator=g) / math.sqrt(width)).to(dtype)
    out = torch.zeros(rows, inner, dtype=dtype, device=DEV)
    status = ops.new_status(DEV)
    ops.activated_linear(out, x.to(DEV), w.to(DEV), ops.ACT_RELU_SQUARED, status)
    ops.check_status(status)
    want = pz.relu_squared(x.double() @ w.double().T)
    torch.testing.assert_close(out.double().cpu(), want, **tol_of(dtype, tight=5e-5))
    if dtype == torch.bfloat16 and ops.tc_applies(x.to(DEV), w.to(DEV)):        # the activation in the tcgen05 product's epilogue
        ops.gemm_tc(out, x.to(DEV), w.to(DEV), status=status, activation=(ops.ACT_RELU_SQUARED, 1.0, 0.0))
        ops.check_status(status)
        torch.testing.assert_close(out.double().cpu(), want, **tol_of(dtype))
    assert float((out == 0).float().mean()) > 0.3                      # (about half of the products are negative)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,inner,columns", [(1, 64, 48, 32), (12, 128, 96, 96), (20, 256, 200, 1), (300, 192, 520, 390),
                                                      (5, 50, 33, 20), (600, 512, 1024, 700)])
def test_silu_on_the_first_columns_of_a_product(rows, width, inner, columns, dtype):
    from lyapunov_engine_b200 import ops
    g = torch.Generator().manual_seed(rows)
    x, w = torch.randn(rows, width, generator=g).to(dtype), (torch.randn(inner, width, generator=g) / math.sqrt(width)).to(dtype)
    out = torch.zeros(rows, inner, dtype=dtype, device=DEV)
    status = ops.new_status(DEV)
    ops.activated_linear(out, x.to(DEV), w.to(DEV), ops.ACT_SILU_COLUMNS, status, columns=columns)
    ops.check_status(status)
    z = x.double() @ w.double().T
    want = torch.cat([pz.silu(z[:, :columns]), z[:, columns:]], dim=1)
    torch.testing.assert_close(out.double().cpu(), want, **tol_of(dtype, tight=5e-5))
    if dtype == torch.bfloat16 and ops.tc_applies(x.to(DEV), w.to(DEV)):
        ops.gemm_tc(out, x.to(DEV), w.to(DEV), status=status, activation=(ops.ACT_SILU_COLUMNS, 1.0, float(columns)))
        ops.check_status(status)
        torch.testing.assert_close(out.double().cpu(), want, **tol_of(dtype))


# ------------------------------------------------------------------ router, experts, identity experts
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", [(5, 48, 6, 2), (70, 64, 70, 5), (3, 20, 1, 1), (9, 32, 4, 4)])
def test_router_scores_over_all_with_a_corrected_choice(shape, dtype):
    from lyapunov_engine_b200 import ops
    T, W, E, top = shape
    g = torch.Generator().manual_seed(T + E)
    h, wr = torch.randn(T, W, generator=g).to(dtype), 2 * torch.randn(E, W, generator=g) / math.sqrt(W)
    cor = 0.5 * torch.randn(E, generator=g)
    w = {"m.router": wr.double(), "m.correction": cor.double()}
    for correction in (cor, None):
        if correction is None:
            w["m.correction"] = torch.zeros(E, dtype=torch.float64)
        ids, share = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV)
        ops.moe_route(ids, share, None, h.to(DEV), wr.to(DEV), None, None, top, scoring=ops.MOE_SOFTMAX_ALL,
                      correction=correction.to(DEV) if correction is not None else None)
        want_ids, want, _ = pz.route(h.double(), w, "m.", {"router": {"top": top}})
        assert torch.equal(ids.cpu().long(), want_ids)
        torch.testing.assert_close(share.double().cpu(), want, atol=1e-5, rtol=1e-5)


EXPERTS = [
    # tokens, width, ff, experts, identity, top, shared ff
    (5, 48, 40, 6, 2, 2, 24),
    (1, 64, 32, 4, 3, 4, 0),
    (300, 128, 128, 4, 2, 2, 64),           # rows enough for the tcgen05 product over sorted rows
    (700, 64, 96, 3, 1, 1, 0),
    (3, 20, 12, 1, 1, 1, 8),                # no 16-byte pieces
    (9, 40, 18, 2, 0, 2, 10),
    (4, 32, 16, 1, 4, 5, 16),               # every choice is taken
]


def experts_case(shape, dtype, bias=None):
    from lyapunov_engine_b200.engine.runtime import Runtime
    from lyapunov_engine_b200.parts.base import FEED_FORWARDS, PartSpec
    T, W, F, E, I, top, S = shape
    g = torch.Generator().manual_seed(T + E)
    sizes = {f"m.e{e}.{part}": s for e in range(E) for part, s in (("up", (F, W)), ("down", (W, F)))}
    if S:
        sizes.update({"m.shared.up": (S, W), "m.shared.down": (W, S)})
    w = {n: (torch.randn(*s, generator=g) / math.sqrt(s[1])).to(torch.bfloat16).double() for n, s in sizes.items()}
    w["m.router"] = (3 * torch.randn(E + I, W, generator=g) / math.sqrt(W)).to(torch.bfloat16).double()
    w["m.correction"] = (0.2 * torch.randn(E + I, generator=g)).to(torch.bfloat16).double()
    if bias is not None:
        w["m.correction"] += torch.tensor(bias, dtype=torch.float64)
    shared = PartSpec("relu_squared", {"hidden_size": W, "intermediate_size": S, "up_name": "m.shared.up",
                                       "down_name": "m.shared.down"}) if S else None
    part = FEED_FORWARDS.build(PartSpec("routed_experts", {
        "hidden_size": W, "intermediate_size": F, "num_experts": E, "identity": I, "top": top, "router_name": "m.router",
        "router_bias_name": None, "correction_name": "m.correction", "expert_names": "m.e{expert}.{part}",
        "activation": "relu_squared", "scoring": "softmax_all", "shared": shared}))
    rt = Runtime(DEV, dtype)
    part.bind(lambda name: w[name].to(torch.float32 if name in ("m.router", "m.correction") else dtype).to(DEV), rt)
    cfg = {"router": {"experts": E, "identity": I, "top": top}, "expert": {"ff": F}}
    if S:
        cfg["shared"] = {"ff": S}
    return part, rt, w, cfg, torch.randn(T, W, generator=g).to(dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", EXPERTS, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("lean", [0.0, 50.0, -50.0])
def test_experts_without_a_gate_and_identity_experts(shape, lean, dtype):
    """``lean``: a correction that sends every token to the identity experts
    first (50), to none where the others suffice (-50), or leaves the choice
    mixed; the weights stay what the uncorrected scores say."""
    from lyapunov_engine_b200 import ops
    E, I = shape[3], shape[4]
    part, rt, w, cfg, h = experts_case(shape, dtype, bias=[0.0] * E + [lean] * I)

    class Ctx:
        workspace, status = rt.workspace, rt.status
    out = part.forward(h.to(DEV), Ctx)
    ops.check_status(rt.status)
    margins = []
    want = pz.routed_experts(h.double(), w, "m.", cfg, None, margins)
    ids, _, _ = pz.route(h.double(), w, "m.", cfg)
    if I and lean > 0:
        assert bool((ids[:, 0] >= E).all())
    clear = margins[0] > 1e-5
    assert int(clear.sum()) >= len(clear) - 1
    torch.testing.assert_close(out.double().cpu()[clear], want[clear], **tol_of(dtype, tight=1e-4, loose=6e-2))
