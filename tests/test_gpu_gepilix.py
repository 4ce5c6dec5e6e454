"""The Gepilix decoder on the GPU: every new kernel and every new option of an older one against the plain PyTorch
statement of its operator (tests/torch_ops.py), attention inputs made so that one key stands out at the edges of windows,
chunks and pages, and the engine -- whole prompts, decoding, portions, mixed batches, captured steps, generation, the
trace runner -- against tests/plain_gepilix.py."""
import json
import random
import subprocess
from types import SimpleNamespace

import pytest
import torch

import plain_gepilix as plain
import traces
from conftest import ROOT, random_tokens
from torch_ops import TorchOps

pytestmark = pytest.mark.gpu
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL32 = 2e-4


@pytest.fixture(scope="module")
def ops():
    from pytriton_llama_b200.ops.cuda import CudaOps
    return CudaOps(torch.device("cuda:0"))


def _ctx(q_lens, starts, slots, device):
    t = lambda v: torch.tensor(v, dtype=torch.int32, device=device)
    q_start = [0]
    for n in q_lens:
        q_start.append(q_start[-1] + n)
    return SimpleNamespace(num_requests=len(q_lens), num_tokens=q_start[-1], q_start=t(q_start), state_slot=t(slots), max_q_len=max(q_lens),
                           max_ctx_len=max(s + n for s, n in zip(starts, q_lens)), work={},
                           tok_req=t([r for r, n in enumerate(q_lens) for _ in range(n)]),
                           positions=t([s + i for s, n in zip(starts, q_lens) for i in range(n)]))


# portions beside single tokens, requests that start and that go on, slots out of order; single tokens alone
STEPS = {"portions": ([70, 1, 9, 1, 33, 2], [0, 40, 17, 0, 5, 1], [2, 0, 3, 1, 6, 5]), "single": ([1] * 5, [0, 40, 17, 3, 1], [4, 0, 3, 1, 2])}


def _both(step):
    q_lens, starts, slots = STEPS[step]
    return _ctx(q_lens, starts, slots, "cuda:0"), _ctx(q_lens, starts, slots, "cpu"), sum(q_lens)


def _close(got, ref, dtype, what, scale=None, tol=None):
    got, ref = got.double().cpu(), ref.double().cpu()
    assert torch.isfinite(got).all(), what
    scale = scale or max(1.0, float(ref.abs().max()))
    tol = tol or (2e-5 if dtype == "float32" else 1.2e-2)
    assert (got - ref).abs().max() <= tol * scale, f"{what}: {(got - ref).abs().max():.3e} of {scale:.2f}"


def _rand(gen, *shape, scale=1.0):
    return torch.randn(*shape, generator=gen) * scale


def _cuda(t):
    return None if t is None else t.cuda()


# ---------------------------------------------------------------------------- norm without statistics
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [40, 256, 1030, 33, 2048, 4096, 8200])
def test_scaled_add_and_tanh_norm(ops, dtype, width):
    g = torch.Generator().manual_seed(width)
    dt, T, ref = DTYPES[dtype], 13, TorchOps()
    a, b = _rand(g, T, width).to(dt), _rand(g, T, width, scale=3.0).to(dt)
    norm = (0.6, 1 + 0.2 * _rand(g, width), 0.3 * _rand(g, width))
    dnorm = (0.6, norm[1].cuda(), norm[2].cuda())
    scale, res = 1 + 0.5 * _rand(g, width), _rand(g, T, width)
    wa, wb = 1 + 0.2 * _rand(g, width), 1 + 0.2 * _rand(g, width)
    rows = torch.tensor([12, 0, 5], dtype=torch.int32)
    cases = {"an output": dict(x=a), "a float32 output": dict(x=a.float() * 1.001), "nothing": dict(x=None),
             "two members": dict(x=None, members=([(a, wa), (b, wb)], 1e-5)), "one member": dict(x=None, members=([(b, wb)], 1e-3))}
    for what, c in cases.items():
        for sc in (scale, None):
            m = c.get("members")
            dm = None if m is None else ([(x.cuda(), w.cuda()) for x, w in m[0]], m[1])
            ra, rb = res.clone().cuda(), res.clone()
            ya, ra2 = ops.add_tanh_norm(_cuda(c["x"]), ra, dnorm, scale=_cuda(sc), dtype=dt, members=dm)
            yb, _ = ref.add_tanh_norm(c["x"], rb, norm, scale=sc, dtype=dt, members=m)
            assert ra2 is ra
            _close(ra, rb, "float32", f"{what}: stream", tol=3e-6)
            _close(ya, yb, dtype, f"{what}: norm", tol=3e-6 if dtype == "float32" else 5e-3)
            yp, none = ops.add_tanh_norm(_cuda(c["x"]), res.cuda(), dnorm, scale=_cuda(sc), rows=rows.cuda(), dtype=dt, members=dm)
            assert none is None
            _close(yp, yb[rows.long()], dtype, f"{what}: picked rows", tol=3e-6 if dtype == "float32" else 5e-3)
    ya, ra = ops.add_tanh_norm(a.cuda(), None, dnorm, dtype=dt)
    yb, rb = ref.add_tanh_norm(a, None, norm, dtype=dt)
    _close(ra, rb, "float32", "a new stream", tol=1e-7)
    _close(ya, yb, dtype, "a new stream's norm", tol=3e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [1, 5, 8, 9, 16, 30, 64, 65, 200])
@pytest.mark.parametrize("N,K", [(256, 192), (1000, 520), (96, 4096), (37, 72), (2048, 64), (50, 27)])
def test_products_with_the_tail_and_with_the_square_of_relu(ops, dtype, T, N, K):
    g = torch.Generator().manual_seed(T + N)
    dt, ref = DTYPES[dtype], TorchOps()
    x, w = _rand(g, T, K).to(dt), _rand(g, N, K, scale=K ** -0.5).to(dt)
    norm, scale, res = (0.5, 1 + 0.2 * _rand(g, N), 0.3 * _rand(g, N)), 1 + 0.5 * _rand(g, N), _rand(g, T, N)
    ra, rb = res.clone().cuda(), res.clone()
    ya = ops.linear_add_tanh_norm(x.cuda(), w.cuda(), ra, (0.5, norm[1].cuda(), norm[2].cuda()), scale.cuda())
    yb = ref.linear_add_tanh_norm(x, w, rb, norm, scale)
    _close(ra, rb, dtype, "stream", tol=2e-5 if dtype == "float32" else 1e-2)
    _close(ya, yb, dtype, "norm", tol=2e-5 if dtype == "float32" else 1.5e-2)
    assert ops.gemm_tc_status() == 0
    _close(ops.linear_relu2(x.cuda(), w.cuda()), ref.linear_relu2(x, w), dtype, "square of relu", tol=2e-5 if dtype == "float32" else 1.5e-2)
    xs, ws = _rand(g, 3, T, K).to(dt), _rand(g, 3, N, K, scale=K ** -0.5).to(dt)
    _close(ops.linear_each(xs.cuda(), ws.cuda()), ref.linear_each(xs, ws), dtype, "a matrix each")


# ---------------------------------------------------------------------------- token shift
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("step", sorted(STEPS))
@pytest.mark.parametrize("width", [40, 33, 2048, 4100])
def test_token_shift_and_its_state(ops, dtype, step, width):
    g = torch.Generator().manual_seed(width)
    dt, ref = DTYPES[dtype], TorchOps()
    cd, cc, T = _both(step)
    h, mu, last = _rand(g, T, width).to(dt), torch.rand(5, width, generator=g), _rand(g, 8, width)
    la, lb = last.clone().cuda(), last.clone()
    a, b = ops.token_shift(h.cuda(), mu.cuda(), la, cd), ref.token_shift(h, mu, lb, cc)
    _close(a, b, dtype, "mixes", tol=1e-6 if dtype == "float32" else 5e-3)
    assert torch.equal(la.cpu(), lb)            # the kept rows are the rows themselves, and no other slot was touched


# ---------------------------------------------------------------------------- short convolution with a bias on its input
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("step", sorted(STEPS))
@pytest.mark.parametrize("channels,taps,column,ld", [(64, 4, 16, 96), (300, 3, 0, 300), (2, 2, 4, 8), (33, 4, 1, 40), (48, 1, 0, 48), (40, 9, 8, 64),
                                                    (1030, 4, 2, 1100), (26, 5, 0, 26)])
def test_causal_convolution_with_input_bias(ops, dtype, step, channels, taps, column, ld):
    g = torch.Generator().manual_seed(channels + taps)
    dt, ref = DTYPES[dtype], TorchOps()
    cd, cc, T = _both(step)
    x, w, b, ib = _rand(g, T, ld).to(dt), _rand(g, channels, taps), _rand(g, channels), _rand(g, channels)
    state = _rand(g, 8, max(taps - 1, 1), channels)
    for bias in (ib, None):
        for silu in (False, True):
            sa, sb = state.clone().cuda(), state.clone()
            a = ops.causal_conv(x.cuda(), column, channels, w.cuda(), b.cuda(), sa, cd, silu=silu, in_bias=_cuda(bias))
            r = ref.causal_conv(x, column, channels, w, b, sb, cc, silu=silu, in_bias=bias)
            _close(a, r, dtype, "result", tol=3e-6 if dtype == "float32" else 5e-3)
            _close(sa, sb, "float32", "state", tol=1e-6)


# ---------------------------------------------------------------------------- recurrences
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("step", sorted(STEPS) + ["long"])
@pytest.mark.parametrize("n,blocks,scale,extra", [(64, 4, 1.0, 0), (24, 3, 0.7, 8), (15, 5, 1.0, 3), (1024, 4, 1.0, 0), (40, 1, -0.5, 8), (600, 2, 1.0, 0)])
def test_gated_linear_recurrence(ops, dtype, step, n, blocks, scale, extra):
    g = torch.Generator().manual_seed(n)
    dt, ref = DTYPES[dtype], TorchOps()
    if step == "long":
        q_lens, starts, slots = [700, 1, 257], [0, 3, 50], [1, 2, 0]
        cd, cc, T = _ctx(q_lens, starts, slots, "cuda:0"), _ctx(q_lens, starts, slots, "cpu"), sum(q_lens)
    else:
        cd, cc, T = _both(step)
    s = n // blocks
    u, wg = _rand(g, T, n).to(dt), _rand(g, blocks, 2 * s, s, scale=s ** -0.5).to(dt)
    gb, rate = 0.5 * _rand(g, 2, n), torch.exp(torch.empty(n).uniform_(-7.0, 2.0, generator=g))       # from hardly any decay to e^-7 a token
    yx, yb, state = _rand(g, T, n + extra).to(dt), 0.3 * _rand(g, n), _rand(g, 8, n)
    oa, ob = torch.zeros(T, n + 2 * extra, dtype=dt).cuda(), torch.zeros(T, n + 2 * extra, dtype=dt)
    sa, sb = state.clone().cuda(), state.clone()
    ops.gated_lru(u.cuda(), wg.cuda(), gb.cuda(), rate.cuda(), yx.cuda(), yb.cuda(), sa, cd, oa, extra, scale)
    ref.gated_lru(u, wg, gb, rate, yx, yb, sb, cc, ob, extra, scale)
    _close(oa, ob, dtype, "result", tol=1e-5 if dtype == "float32" else 1e-2)
    _close(sa, sb, "float32", "state", tol=1e-5)


def test_a_channel_that_hardly_decays_keeps_what_it_should(ops):
    """A decay of 1 - 1e-5 over 4,000 tokens: a rounded once per token would lean by up to 1e-7 each time."""
    n, T = 16, 4000
    cd = _ctx([T], [0], [0], "cuda:0")
    u = torch.ones(T, n)
    wg, gb = torch.zeros(1, 2 * n, n), torch.zeros(2, n)
    gb[0] = 30.0                                          # r = 1: log a = -rate
    rate = torch.logspace(-6, -4, n)
    out, state = torch.zeros(T, n).cuda(), torch.zeros(1, n).cuda()
    ops.gated_lru(u.cuda(), wg.cuda(), gb.cuda(), rate.cuda(), torch.ones(T, n).cuda(), torch.zeros(n).cuda(), state, cd, out, 0, 1.0)
    r64 = rate.double()
    want = torch.sqrt(-torch.expm1(-2 * r64)) * 0.5 * torch.expm1(-T * r64) / torch.expm1(-r64)     # i = 1/2, a geometric series
    assert ((state[0].cpu().double() - want) / want).abs().max() < 2e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("step", sorted(STEPS))
@pytest.mark.parametrize("H,G,n,dv", [(4, 2, 16, 32), (6, 1, 48, 20), (2, 2, 128, 64), (3, 3, 200, 33), (8, 4, 64, 8), (1, 1, 3, 100)])
def test_state_space_walk_and_the_gated_norm_in_parts(ops, dtype, step, H, G, n, dv):
    g = torch.Generator().manual_seed(H * 10 + n)
    dt, ref = DTYPES[dtype], TorchOps()
    cd, cc, T = _both(step)
    xbc, steps = _rand(g, T, H * dv + 2 * G * n, scale=0.7).to(dt), _rand(g, T, H)
    bias, rate, D, state = _rand(g, H), torch.exp(2 * _rand(g, H)), _rand(g, H), _rand(g, 8, H, n, dv, scale=0.3)
    sa, sb = state.clone().cuda(), state.clone()
    a = ops.state_space_scan(xbc.cuda(), steps.cuda(), bias.cuda(), rate.cuda(), D.cuda(), sa, cd, H, G, n, dv)
    b = ref.state_space_scan(xbc, steps, bias, rate, D, sb, cc, H, G, n, dv)
    _close(a, b, "float32", "read-outs", tol=1e-5)
    _close(sa, sb, "float32", "states", tol=1e-5)
    inner = H * dv
    for groups in [k for k in (1, 2, 3, inner) if inner % k == 0]:
        for column, extra in ((0, 0), (8, 16), (3, 5)):
            gate, w = _rand(g, T, inner + 7 * bool(column)).to(dt), 1 + 0.2 * _rand(g, inner)
            oa, ob = torch.zeros(T, inner + column + extra, dtype=dt).cuda(), torch.zeros(T, inner + column + extra, dtype=dt)
            ops.gated_group_norm(b.cuda(), gate.cuda(), 0, w.cuda(), 1e-4, groups, oa, column, 0.6)
            ref.gated_group_norm(b, gate, 0, w, 1e-4, groups, ob, column, 0.6)
            _close(oa, ob, dtype, f"{groups} parts", tol=1e-5 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("len_", [4096, 8192, 9000, 1001])
def test_a_long_part_of_the_gated_norm(ops, len_):
    g = torch.Generator().manual_seed(len_)
    y, gate, w = _rand(g, 3, 2 * len_), _rand(g, 3, 2 * len_), 1 + 0.2 * _rand(g, 2 * len_)
    oa, ob = torch.zeros(3, 2 * len_).cuda(), torch.zeros(3, 2 * len_)
    ops.gated_group_norm(y.cuda(), gate.cuda(), 0, w.cuda(), 1e-5, 2, oa, 0, 1.0)
    TorchOps().gated_group_norm(y, gate, 0, w, 1e-5, 2, ob, 0, 1.0)
    _close(oa, ob, "float32", "part", tol=5e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("step", sorted(STEPS))
@pytest.mark.parametrize("H,d", [(3, 32), (2, 64), (1, 128), (2, 200), (4, 8), (1, 20), (5, 12)])
def test_wkv_walk_with_its_bonus(ops, dtype, step, H, d):
    g = torch.Generator().manual_seed(H * 10 + d)
    dt, ref = DTYPES[dtype], TorchOps()
    cd, cc, T = _both(step)
    n = H * d
    rkvg, inner, w2 = _rand(g, 4, T, n, scale=0.7).to(dt), _rand(g, T, 7), _rand(g, n, 7, scale=0.4)
    bias, u, state = torch.empty(n).uniform_(-9.0, 1.0, generator=g), _rand(g, n), _rand(g, 8, H, d, d, scale=0.3)
    da, db = ops.lowrank_tanh_linear(inner.cuda(), 0, w2.cuda(), decay_bias=bias.cuda()), ref.lowrank_tanh_linear(inner, 0, w2, decay_bias=bias)
    _close(da, db, "float32", "decays", tol=3e-7)
    sa, sb = state.clone().cuda(), state.clone()
    a = ops.wkv_scan(rkvg.cuda(), da, u.cuda(), sa, cd, H, d)
    b = ref.wkv_scan(rkvg, db, u, sb, cc, H, d)
    _close(a, b, "float32", "read-outs", tol=1e-5)
    _close(sa, sb, "float32", "states", tol=1e-5)
    assert torch.equal(sa[7].cpu(), state[7])                     # a slot of no request in the step


# ---------------------------------------------------------------------------- attention: cap, chunks, a gate per head
def _paged(gen, q_lens, starts, page, pages, width):
    """Block tables over shuffled pages and the slots of the step's tokens."""
    perm = torch.randperm(pages, generator=gen).tolist()
    bt = torch.full((len(q_lens), width), -1, dtype=torch.int32)
    slots, k = [], 0
    for r, (n, s) in enumerate(zip(q_lens, starts)):
        for b in range(-(-(s + n) // page)):
            bt[r, b] = perm[k]
            k += 1
        slots += [int(bt[r, p // page]) * page + p % page for p in range(s, s + n)]
    return bt, torch.tensor(slots, dtype=torch.int32)


ATTENTION = [   # H, G, d, dv, page, window, chunk, cap, gate per head, result factor
    (4, 2, 64, 64, 16, 0, 20, 5.0, True, 1.0), (6, 3, 48, 80, 8, 9, 0, 3.0, False, 0.7), (2, 1, 24, 40, 4, 0, 1, 8.0, True, 1.0),
    (8, 2, 128, 128, 16, 40, 0, 6.0, True, -0.5), (3, 3, 16, 16, 4, 0, 33, 4.0, False, 1.0), (5, 1, 72, 8, 32, 0, 100, 50.0, True, 1.0),
    (8, 2, 64, 40, 16, 100, 0, 10.0, True, 1.2), (4, 4, 128, 128, 8, 0, 64, 7.0, True, 1.0), (6, 2, 64, 64, 16, 0, 130, 30.0, True, 1.3),
    (2, 2, 64, 64, 16, 0, 0, 2.0, False, 1.0), (4, 1, 128, 128, 16, 1, 0, 5.0, False, 1.0), (4, 2, 64, 64, 4, 0, 7, 0.0, True, 1.0),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,page,window,chunk,cap,gate,factor", ATTENTION)
def test_capped_attention_in_windows_and_chunks(ops, dtype, H, G, d, dv, page, window, chunk, cap, gate, factor):
    g = torch.Generator().manual_seed(H * 100 + d + chunk)
    dt, ref = DTYPES[dtype], TorchOps()
    q_lens, starts = [300, 1, 37, 1, 2], [0, 190, 61, 3, 254]
    R, T = len(q_lens), sum(q_lens)
    cd, cc = _ctx(q_lens, starts, list(range(R)), "cuda:0"), _ctx(q_lens, starts, list(range(R)), "cpu")
    pages = sum(-(-(s + n) // page) for s, n in zip(starts, q_lens)) + 3
    bt, _ = _paged(g, q_lens, starts, page, pages, width=-(-300 // page) + 2)
    gate_col = H * d + G * (d + dv)
    proj = _rand(g, T, -(-(gate_col + H) // 8) * 8, scale=1.5).to(dt)
    cache = _rand(g, pages, G * page * (d + dv)).to(dt)
    kw = dict(softcap=cap, chunk=chunk, out_scale=factor, **(dict(gate_column=gate_col, gate_per_head=True) if gate else {}))
    scale = 2.0 * d ** -0.5                # scores of a few units, beside the small caps
    want = ref.window_attention(proj, cache, bt, cc.tok_req, cc.positions, H, G, d, dv, page, scale, window, 0, **kw)
    hints = ops.hints_for(q_lens, [s + n for s, n in zip(starts, q_lens)])
    args = (proj.cuda(), cache.cuda(), bt.cuda(), cd.tok_req, cd.positions, H, G, d, dv, page, scale)
    out = ops.window_attention(*args, window, 0, hints=hints, **kw)
    _close(out, want, dtype, "as the engine calls it", tol=2e-5 if dtype == "float32" else 2e-2)
    whole = torch.full((T, H * dv + 24), 7.0, dtype=dt, device="cuda:0")
    ops.window_attention(*args, window, 0, hints=hints, out=whole, column=8, **kw)
    assert torch.equal(whole[:, 8:8 + H * dv], out) and bool((whole[:, :8] == 7).all()) and bool((whole[:, 8 + H * dv:] == 7).all())
    for splits in (1, 3):
        out = torch.empty((T, H * dv), dtype=dt, device="cuda:0")
        ops._window_attention_simt(out, *args, window, 0, splits, None, (0, 0, 0.0, 1, 0.0, gate_col if gate else -1, 0, None, None, 0, 0, None,
                                                                         cap, chunk, int(gate), factor))
        _close(out, want, dtype, f"{splits} parts", tol=2e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,page,q_len", [(64, 16, 1), (64, 4, 5), (64, 16, 140), (128, 16, 140), (32, 8, 140), (32, 8, 1)])
@pytest.mark.parametrize("kind", ["chunk", "window"])
def test_a_key_that_stands_out_is_seen_where_its_chunk_or_window_says(ops, dtype, d, page, q_len, kind):
    """One key with a score far above the others and a value of its own, at the last place of a chunk and at the first: the
    result is that value exactly where the query sees the key."""
    H, G, size, n = 2, 1, 24, 140
    dt, ref = DTYPES[dtype], TorchOps()
    for spike in (47, 48):
        g = torch.Generator().manual_seed(page + q_len)
        start = n - q_len
        cd, cc = _ctx([q_len], [start], [0], "cuda:0"), _ctx([q_len], [start], [0], "cpu")
        pages = -(-n // page) + 2
        bt, _ = _paged(g, [n], [0], page, pages, width=pages)
        keys, values = _rand(g, n, d, scale=0.05), _rand(g, n, d, scale=0.1)
        keys[spike, 0] = 6.0
        values[spike] = 50.0
        cache = torch.zeros(pages, G * page * 2 * d).to(dt)
        for p in range(n):
            kp, vp = TorchOps._page_views(cache, int(bt[0, p // page]), G, page, d, d)
            kp[0, p % page], vp[0, p % page] = keys[p].to(dt), values[p].to(dt)
        q = torch.zeros(q_len, H * d + G * 2 * d)
        q[:, 0] = q[:, d] = 4.0
        q = q.to(dt)
        kw = dict(softcap=20.0, **({"chunk": size} if kind == "chunk" else {"window": size}))
        want = ref.window_attention(q, cache, bt, cc.tok_req, cc.positions, H, G, d, d, page, 1.0, **kw)
        got = ops.window_attention(q.cuda(), cache.cuda(), bt.cuda(), cd.tok_req, cd.positions, H, G, d, d, page, 1.0,
                                   hints=ops.hints_for([q_len], [n]), **kw)
        _close(got, want, dtype, "spiked key", tol=1e-4 if dtype == "float32" else 2e-2)
        for i in range(q_len):
            p = start + i
            seen = p >= spike and (p // size == spike // size if kind == "chunk" else p - spike < size)
            assert (float(got[i, 0]) > 45) == seen, (p, float(got[i, 0]))


# ---------------------------------------------------------------------------- experts: router bias, sum with the tail
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,W,ff,E,top,shared", [(45, 64, 32, 8, 4, True), (3, 96, 64, 16, 1, False), (200, 48, 24, 6, 2, True), (17, 33, 16, 9, 9, False),
                                                 (400, 128, 96, 64, 6, True), (5, 32, 8, 1, 1, True), (9, 2050, 16, 130, 5, False)])
def test_experts_with_a_router_bias_and_the_tail(ops, dtype, T, W, ff, E, top, shared):
    g = torch.Generator().manual_seed(T + E)
    dt, ref = DTYPES[dtype], TorchOps()
    x, logits, bias = _rand(g, T, W).to(dt), _rand(g, T, E, scale=2.0), _rand(g, E, scale=2.0)
    w_gu, w_d = _rand(g, E, 2 * ff, W, scale=W ** -0.5).to(dt), _rand(g, E, W, ff, scale=ff ** -0.5).to(dt)
    sh = _rand(g, T, W).to(dt) if shared else None
    norm, scale, res = (0.5, 1 + 0.2 * _rand(g, W), 0.3 * _rand(g, W)), 1 + 0.5 * _rand(g, W), _rand(g, T, W)
    opts = dict(score="softmax", renormalise=True)
    rows = ops.expert_rows(x.cuda(), logits.cuda(), w_gu.cuda(), w_d.cuda(), top, logit_bias=bias.cuda(), **opts)
    # the softmax over the chosen logits alone
    biased = (logits + bias).double()
    chosen = biased.topk(top).values
    weights = rows.weights.view(T, top).cpu().double()
    _close(weights.sort(dim=1).values, torch.softmax(chosen, 1).sort(dim=1).values, "float32", "weights", tol=2e-6)
    ra, rb = res.clone().cuda(), res.clone()
    ya = ops.combine_experts_tanh_norm(rows, _cuda(sh), ra, (0.5, norm[1].cuda(), norm[2].cuda()), scale.cuda())
    yb = ref.combine_experts_tanh_norm(ref.expert_rows(x, logits, w_gu, w_d, top, logit_bias=bias, **opts), sh, rb, norm, scale)
    _close(ra, rb, dtype, "stream", tol=2e-5 if dtype == "float32" else 2e-2)
    _close(ya, yb, dtype, "norm", tol=2e-5 if dtype == "float32" else 2e-2)


# ---------------------------------------------------------------------------- the engine
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, dtype, cfg=None, seed=5):
        if (name, dtype) not in made:
            folder = tmp_path_factory.mktemp(f"gepilix_{name}_{dtype}")
            plain.write_model(folder, cfg or plain.TINY[name], seed, DTYPES[dtype])
            made[(name, dtype)] = folder
        return made[(name, dtype)]
    return get


def _engine(folder, dtype, page, pages, max_seq_len=512, slots=4, **extra):
    from pytriton_llama_b200.config import EngineConfig
    from pytriton_llama_b200.engine.engine import Engine
    return Engine(folder, EngineConfig(dtype=dtype, page_size=page, max_gpu_num_blocks=pages, max_seq_len=max_seq_len,
                                       max_num_seqs=slots, **extra), device="cuda:0")


def _reference(folder, seqs):
    from pytriton_llama_b200.weights import read_folder
    cfg = json.loads((folder / "config.json").read_text())
    W = read_folder(folder)
    return {r: plain.forward(cfg, W, s) for r, s in seqs.items()}


def _assert_logits(got, ref, dtype, what):
    diff = (got.double().cpu() - ref).abs()
    if dtype == "float32":
        assert diff.max() < TOL32 * max(1.0, float(ref.abs().max())), f"{what}: {diff.max():.3e}"
    else:
        centred = (got.double().cpu() - ref) - (got.double().cpu() - ref).mean(-1, keepdim=True)
        rms = centred.pow(2).mean(-1).sqrt() / ref.std()
        # Rounding alone moves the typical row of these models by 0.005 to 0.06 of the logits' spread.  A row where a
        # router's logits lie within rounding of each other may take another expert than the float64 computation does, and
        # the rows after it feel that through the mixers: such rows are allowed, as long as they are few.  A fault of a
        # mechanism shows in float32, where the bound is 2e-4.
        off = int((rms > 0.4).sum())
        assert rms.median() < 0.1 + 0.06 * (rms.numel() < 4) and off <= max(1, rms.numel() // 10), \
            f"{what}: median row {rms.median():.3f} of the logits' spread, {off} of {rms.numel()} rows beyond 0.4"


# Heads of 64 and 128, widths that are multiples of 64, windows and chunks that prompts pass, a state space with real sizes.
WIDE = plain.config(300, 192, [
    plain.layer("parallel", plain.parallel(plain.attention(4, 2, 64, 64, 0.125, 20.0, 40), plain.linear_unit(160, 2, 4)), plain.moe(64, 8, 2, shared=64)),
    plain.layer("parallel_2", plain.parallel_2(plain.attention(2, 1, 128, 128, 0.09, 15.0, 33, rot=plain.rotation(64, 500.0, (4.0, 1.0, 4.0, 64))),
                                               plain.state_space(4, 64, 128, 2, 1, 4), 0.7, 1.1), plain.dense(256)),
    plain.layer("wkv", {"heads": 3, "dim": 32}, plain.moe(32, 4, 1)),
    plain.layer("parallel", plain.parallel(plain.attention(8, 1, 32, 48, 0.17, 30.0, 70), plain.linear_unit(96, 1, 3)), None),
    plain.layer("parallel_2", plain.parallel_2(plain.attention(3, 3, 64, 64, 0.12, 9.0, 50, rot=plain.rotation(64, 1.0e4)),
                                               plain.state_space(6, 32, 16, 1, 3, 2), 1.0, 1.0), plain.dense(136)),
])


def _config(name):
    return WIDE if name == "WIDE" else plain.TINY[name]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page", [("A", 4), ("B", 8), ("C", 16), ("WIDE", 16)])
def test_every_cut_gives_the_whole_sequence_logits(folders, dtype, name, page):
    folder = folders(name, dtype, _config(name))
    seqs = {f"r{i}": random_tokens(n, _config(name)["vocab"], 700 + i) for i, n in enumerate([1, 9, 33, 150, 12, 27, 64])}
    ref = _reference(folder, seqs)
    for family in (traces.whole, traces.prefill_then_decode, traces.portions, traces.mixed):
        steps = family(seqs)
        eng = _engine(folder, dtype, page, -(-traces.max_live_tokens(steps, 16) // page))
        got = traces.replay(eng, steps)
        for r in seqs:
            _assert_logits(got[r], ref[r][traces.wanted_positions(steps, r)], dtype, f"{family.__name__} {r}")
        eng.check_device_status()
        eng.cache.check_invariants()
        assert eng.cache.free_slots() == 4 and all(eng.cache.free_pages(g) == eng.cache.groups[g].pool.num_pages for g in eng._paged_groups())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_steps_from_captured_graphs(folders, dtype):
    folder = folders("WIDE", dtype, WIDE)
    seqs = {f"g{i}": random_tokens(n, 300, 300 + i) for i, n in enumerate([80, 7, 55, 21, 33])}
    ref = _reference(folder, seqs)
    eng = _engine(folder, dtype, 16, 40, compiled_model=True)
    for turn in range(3):           # the same steps again: shapes seen twice are captured, then replayed
        for family in (traces.prefill_then_decode, traces.mixed):
            steps = family(seqs)
            got = traces.replay(eng, steps)
            for r in seqs:
                _assert_logits(got[r], ref[r][traces.wanted_positions(steps, r)], dtype, f"turn {turn} {family.__name__} {r}")
    assert any(not isinstance(k, tuple) for k in eng._graphs)             # decode steps were captured
    eng.check_device_status()


@pytest.mark.parametrize("switch", ["PTL_PARALLEL_STREAMS", "PTL_WINDOW_TC", "fuses_next_norm", "small_products", "library_products", "moe_tensor_cores"])
def test_the_switches_change_nothing_but_rounding(folders, monkeypatch, switch):
    folder = folders("WIDE", "bfloat16", WIDE)
    seqs = {f"s{i}": random_tokens(n, 300, 60 + i) for i, n in enumerate([130, 9, 41])}
    ref = _reference(folder, seqs)
    if switch.startswith("PTL_"):
        monkeypatch.setenv(switch, "0")
    eng = _engine(folder, "bfloat16", 16, 40)
    if not switch.startswith("PTL_"):
        setattr(eng.ops, switch, False)
    steps = traces.mixed(seqs)
    got = traces.replay(eng, steps)
    for r in seqs:
        _assert_logits(got[r], ref[r][traces.wanted_positions(steps, r)], "bfloat16", f"{switch} {r}")
    eng.check_device_status()


def _random_config(seed):
    """Sizes drawn freely: head sizes that are no power of two, one to three kv heads, windows and chunks of 1 to 60
    positions, part of a head or all of it rotated, layers in any order, with and without feed-forwards and shared experts."""
    rng = random.Random(seed)
    width = rng.choice([48, 56, 64, 72, 88, 100, 61])
    layers = []
    for i in range(rng.randint(2, 5)):
        mlp = None
        if rng.random() > 0.2:
            E = rng.randint(1, 12)
            mlp = plain.dense(rng.choice([8, 24, 100, 33])) if rng.random() < 0.5 else \
                plain.moe(rng.choice([8, 24, 40]), E, rng.randint(1, E), shared=rng.choice([0, 16, 40]))
        kind = rng.choice(["parallel", "parallel_2", "wkv"])
        if kind == "wkv":
            layers.append(plain.layer("wkv", {"heads": rng.randint(1, 4), "dim": rng.choice([8, 12, 20, 32, 36, 64])}, mlp))
            continue
        G, d = rng.randint(1, 3), rng.choice([8, 16, 24, 40, 64])
        size, cap = rng.choice([rng.randint(1, 60), rng.randint(1, 12)]), rng.choice([3.0, 10.0, 50.0])
        rot = None
        if kind == "parallel_2" and rng.random() > 0.2:
            rot = plain.rotation(rng.choice([2, d // 2 // 2 * 2, d]), rng.choice([30.0, 10000.0]),
                                 None if rng.random() < 0.4 else (rng.choice([2.0, 8.0]), 1.0, rng.choice([2.0, 4.0]), rng.choice([16, 64, 1024])))
        left = plain.attention(G * rng.choice([1, 2, 4]), G, d, rng.choice([8, 16, 24, 40, 64]), rng.uniform(0.1, 0.4), cap, size, rot)
        if kind == "parallel":
            blocks = rng.randint(1, 5)
            layers.append(plain.layer(kind, plain.parallel(left, plain.linear_unit(blocks * rng.choice([3, 8, 16, 24]), blocks, rng.randint(1, 6))), mlp))
        else:
            groups = rng.randint(1, 3)
            H, e = groups * rng.randint(1, 3), rng.choice([4, 12, 24, 40])
            parts = rng.choice([k for k in (1, 2, 3, 4, H) if H * e % k == 0])
            layers.append(plain.layer(kind, plain.parallel_2(left, plain.state_space(H, e, rng.choice([4, 9, 16, 40]), groups, parts, rng.randint(1, 6)),
                                                             rng.uniform(-1, 1.5), rng.uniform(0.3, 1.5)), mlp))
    return plain.config(rng.randint(50, 300), width, layers, eps=rng.choice([1e-6, 1e-5, 1e-3]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(16))
def test_random_configurations(tmp_path, dtype, seed):
    cfg = _random_config(seed)
    plain.write_model(tmp_path, cfg, seed, weights=plain.random_weights(cfg, seed, DTYPES[dtype], rank=random.Random(seed).choice([4, 16, 33])))
    seqs = {f"r{i}": random_tokens(n, cfg["vocab"], 40 * seed + i) for i, n in enumerate([90, 1, 33, 14])}
    ref = _reference(tmp_path, seqs)
    page = random.Random(seed).choice([4, 8, 16, 32])
    for family in (traces.whole, traces.mixed):
        steps = family(seqs)
        eng = _engine(tmp_path, dtype, page, -(-traces.max_live_tokens(steps, 32) // page) + 1)
        got = traces.replay(eng, steps)
        for r in seqs:
            _assert_logits(got[r], ref[r][traces.wanted_positions(steps, r)], dtype, f"seed {seed} {family.__name__} {r}")
        eng.check_device_status()


@pytest.mark.parametrize("seed", [1, 2, 3])
def test_random_traces_in_float32(folders, seed):
    folder = folders("A", "float32")
    rng = random.Random(seed)
    seqs = {f"t{i}": random_tokens(rng.randint(1, 200), 97, 900 + 10 * seed + i) for i in range(7)}
    ref = _reference(folder, seqs)
    steps = traces.random_trace(seqs, rng)
    for graphs in (False, True):
        eng = _engine(folder, "float32", 4, -(-traces.max_live_tokens(steps, 4) // 4), compiled_model=graphs)
        got = traces.replay(eng, steps)
        for r in got:
            _assert_logits(got[r], ref[r][traces.wanted_positions(steps, r)], "float32", f"trace {seed} {r}")
        eng.cache.check_invariants()


def test_batch_does_not_change_a_request(folders):
    from pytriton_llama_b200.engine.engine import StepEntry
    folder = folders("WIDE", "float32", WIDE)
    seqs = {"a": random_tokens(137, 300, 1), "b": random_tokens(8, 300, 2), "c": random_tokens(61, 300, 3)}
    eng = _engine(folder, "float32", 16, 40)
    together = eng.step([StepEntry(r, s, list(range(len(s)))) for r, s in seqs.items()]).logits
    eng.finish_all()
    at = 0
    for r, s in seqs.items():
        alone = eng.step([StepEntry(r, s, list(range(len(s))))]).logits
        eng.finish(r)
        assert torch.allclose(together[at:at + len(s)], alone, atol=5e-5, rtol=1e-5), r
        at += len(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, dtype):
    from pytriton_llama_b200.engine.engine import StepEntry
    folder = folders("WIDE", dtype, WIDE)
    toks = random_tokens(400, 300, 21)
    ref = _reference(folder, {"a": toks})["a"]
    eng = _engine(folder, dtype, 16, 9)           # 9 pages for 400 tokens: pages that windows and chunks have passed come back
    rows = [eng.step([StepEntry("a", toks[:3], [0, 1, 2])]).logits] + [eng.step([StepEntry("a", [t], [0])]).logits for t in toks[3:]]
    _assert_logits(torch.cat(rows), ref, dtype, "400 tokens, one by one")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(folders, dtype):
    from pytriton_llama_b200 import LLM, EngineConfig, SamplingParams
    folder = folders("A", dtype)
    prompts = [random_tokens(n, 97, 40 + i) for i, n in enumerate([5, 23, 2, 14, 9, 31])]
    cfg = EngineConfig(dtype=dtype, page_size=4, max_gpu_num_blocks=60, max_seq_len=64, max_num_seqs=3, max_batched_tokens=16)
    outs = LLM(folder, cfg).generate(prompts, SamplingParams(temperature=0.0, max_gen_len=8))
    far = []
    for p, o in zip(prompts, outs):
        assert len(o) == 8
        logits = _reference(folder, {"x": p + o})["x"]
        slack = 1e-3 if dtype == "float32" else 0.1 * float(logits.std())
        for i, tok in enumerate(o):
            row = logits[len(p) + i - 1]
            if row[tok] < row.max() - slack:
                far.append((i, tok, int(row.argmax())))
    # in 16 bits a router's close call may send a token to another expert than the float64 computation does, and what is
    # generated after it differs: a few such tokens are allowed; in float32 none
    assert not far if dtype == "float32" else len(far) <= 4, far


def test_trace_runner_and_command_line(folders, tmp_path):
    folder = folders("WIDE", "bfloat16", WIDE)
    seqs = {"a": random_tokens(90, 300, 1), "b": random_tokens(13, 300, 2)}
    steps = traces.mixed(seqs)
    lines = "\n".join(json.dumps(s) for s in steps) + "\n"
    for dtype in ("bfloat16", "float32"):
        out = tmp_path / dtype
        proc = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                               "--max-tokens", str(traces.max_live_tokens(steps))], input=lines, text=True, capture_output=True,
                              timeout=900)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
        ref = _reference(folder, seqs)
        fed = {r: 0 for r in seqs}
        got, want = [], []
        for s in steps:
            rows = torch.frombuffer(bytearray((out / f"{s['step']}.f32").read_bytes()), dtype=torch.float32).view(-1, 300)
            at = 0
            for e in s["entries"]:
                for w in e["want"]:
                    got.append(rows[at])
                    want.append(ref[e["id"]][fed[e["id"]] + w])
                    at += 1
                fed[e["id"]] += len(e["tokens"])
        _assert_logits(torch.stack(got), torch.stack(want), dtype, f"{dtype} replay")
    import sys
    proc = subprocess.run([sys.executable, str(ROOT / "cli.py"), "--checkpoints_dir", str(folder), "--temperature", "0",
                           "--max_gen_len", "5", "--max_seq_len", "64", "--page_size", "16", "--prompt_ids", "3", "1", "4", "1", "5"],
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert len(proc.stdout.split()) == 5
