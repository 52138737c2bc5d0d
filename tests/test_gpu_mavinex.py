"""The Mavinex design on the GPU against the plain float64 model of tests/plain_mavinex.py: every mechanism's kernels alone,
every layer by itself, whole prompts, token-by-token decoding, prompts in pieces down to two tokens, ragged batches, reused
slots and pages, keys far away, at page borders and at the windows' edges under a peaked softmax, layers on another layer's
weights, sizes of real models, and greedy generation through Engine.generate and the command lines."""
import random
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import helpers
import mavinex_models as mm
import plain_mavinex as pm

pytestmark = pytest.mark.gpu

# A position's error is the root mean square over the vocabulary of the difference of its logits, relative to
# the root mean square of the request's logits.  float32: rounding of a few hundred fused multiply-adds per
# value; bfloat16: activations rounded to 2^-9 relative at every product, a few dozen products deep.
TOL = {"float32": 1e-4, "bfloat16": 5e-2}
# bfloat16 moves a router's logits by a few hundredths (they are several units); a choice that hangs on less than this is a
# close call, and such positions are left out of the bfloat16 comparison
CLOSE_CALL = 0.08


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (raw, seed) in mm.ALL.items():
        d = mm.write(tmp_path_factory.mktemp(f"mavinex_{name}"), raw, seed)
        out[name] = (d, pm.PlainMavinex(d))
    return out


def _engine(folder, dtype, **kw):
    from oracle_engine_b200.engine.engine import Engine
    kw.setdefault("max_tokens", 1024)
    return Engine.from_pretrained(folder, dtype=dtype, **kw)


def _compare(got, plain, requests, tol, what, cache={}):
    """float32 (a tolerance below 1e-3): every position is within the tolerance.  bfloat16: close calls of a router
    are left out, nine positions in ten are within the tolerance and none is beyond six times it."""
    left_out = total = 0
    for i, toks in enumerate(requests):
        key = (id(plain), tuple(toks))
        if key not in cache:
            cache[key] = (plain.logits(toks).numpy(), plain.close_calls(toks, CLOSE_CALL), plain)
        want, close, _ = cache[key]
        assert np.isfinite(got[i]).all(), f"{what}: request {i} has positions without logits"
        err = np.sqrt(((got[i] - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean())
        total += len(toks)
        if tol < 1e-3:
            assert err.max() < tol, f"{what}: request {i} (len {len(toks)}) first bad position " \
                                    f"{int((err >= tol).argmax())}, worst {int(err.argmax())}: {err.max()}"
            continue
        err[sorted(close)] = 0.0
        left_out += len(close)
        assert err.max() < 6 * tol, f"{what}: request {i} (len {len(toks)}) position {int(err.argmax())}: {err.max()}"
        assert (err >= tol).sum() <= 0.1 * len(toks), \
            f"{what}: request {i} (len {len(toks)}): {int((err >= tol).sum())} positions over {tol}, first {int((err >= tol).argmax())}"
    assert total < 50 or left_out <= 0.5 * total, f"{what}: {left_out} of {total} positions are close calls: the test's weights are too even"


def _run(eng, tmp, steps, requests):
    got = helpers.collect(steps, helpers.TraceRunner(eng, tmp).run(steps), requests)
    eng.cache.check()
    assert eng.cache.slots.n_free == eng.cache.n_slots
    return got


def _i32(x):
    return torch.as_tensor(x, dtype=torch.int32).cuda()


def _step(lens, slots, starts=None):
    """What a kernel reads of a step that brings lens[b] tokens of sequences in the given slots (-1: a padding sequence)."""
    starts = starts or [0] * len(lens)
    seq, pos, cu = [], [], [0]
    for b, n in enumerate(lens):
        seq += [b] * n
        pos += list(range(starts[b], starts[b] + n))
        cu.append(cu[-1] + n)
    return SimpleNamespace(tok_seq=_i32(seq), tok_pos=_i32(pos), cu_q=_i32(cu), seq_slot=_i32(slots), seq_start=_i32(starts),
                           seq_qlen=_i32(lens), n_seqs=len(lens), n_tokens=cu[-1], max_qlen=max(lens),
                           max_kvlen=max(s + n for s, n in zip(starts, lens)), all_decode=all(n == 1 for n in lens),
                           context_class=0)


def _close(got, want, tol, what=""):
    err = (got.double().cpu() - want).abs().max().item()
    assert err < tol * max(1e-6, want.abs().max().item()), (what, err, want.abs().max().item())


# ------------------------------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("cast", [False, True])
@pytest.mark.parametrize("two", [False, True])
@pytest.mark.parametrize("rows,D", [(5, 100), (3, 7), (1, 2048), (9, 9000), (300, 96), (33, 4096), (2, 4100)])
def test_norm_of_a_sum(rows, D, two, cast):
    """x <- N(alpha x + y), and with the sum of two outputs that are normed with weights of their own; an eps of the values'
    size; widths in registers and beyond."""
    from oracle_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(rows + D)
    r = lambda *s: torch.randn(*s, generator=g)                            # noqa: E731
    x, y0, y1, w, w0, w1 = r(rows, D), r(rows, D) * 2, r(rows, D) * 0.3, r(D), r(D), r(D)
    eps, alpha = 0.2, 1.3
    d = lambda t: t.double()                                               # noqa: E731
    s = 0.5 * (pm.rms(d(y0), eps) * d(w0) + pm.rms(d(y1), eps) * d(w1)) if two else d(y0)
    want = pm.rms(alpha * d(x) + s, eps) * d(w)
    got = x.cuda()
    out = torch.empty(rows, D, dtype=torch.bfloat16, device="cuda") if cast else None
    parts = [(y0.cuda(), w0.cuda()), (y1.cuda(), w1.cuda())] if two else [(y0.cuda(), None)]
    ops.rmsnorm_sum(got, parts, w.cuda(), alpha, eps, 0.5, out)
    _close(got, want, 1e-6)
    if cast:
        assert torch.equal(out, got.bfloat16())


# (dtype, H, G, dk, dv, turned, pairing): the pieces' form needs bfloat16 and multiples of 8
ROWS = [("bfloat16", 6, 2, 40, 96, 40, "interleaved"), ("bfloat16", 16, 4, 128, 128, 128, "interleaved"),
        ("bfloat16", 40, 8, 128, 64, 64, "interleaved"), ("bfloat16", 3, 1, 20, 12, 10, "interleaved"),
        ("bfloat16", 4, 2, 32, 48, 16, "halves"), ("bfloat16", 4, 4, 32, 32, 0, "interleaved"),
        ("float32", 6, 3, 40, 56, 24, "interleaved"), ("float32", 3, 1, 7, 9, 4, "halves"), ("float32", 5, 5, 20, 12, 0, "halves")]


@pytest.mark.parametrize("normed", [True, False])
@pytest.mark.parametrize("dtype,H,G,dk,dv,dims,pairing", ROWS)
def test_row_norm_turn_and_cache_write(dtype, H, G, dk, dv, dims, pairing, normed):
    """Queries and keys normed over the whole projection, turned, and written over scattered pages; a padding token, rows of
    a wider buffer whose other columns stay."""
    from oracle_engine_b200.csrc import ops
    from oracle_engine_b200.csrc.ops import PAGE
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(H * dk)
    n, start, eps = 70, 40, 0.1
    width = (H + G) * dk + G * dv
    rows = (torch.randn(n, width, generator=g) * (1 + torch.arange(n)[:, None] / 20)).to(tdt)
    qw, kw = torch.randn(H * dk, generator=g), torch.randn(G * dk, generator=g)
    rot = mm.rot(dims, 100.0)
    pos = torch.arange(start, start + n)
    x = rows.double()
    q, k, v = x[:, :H * dk], x[:, H * dk:(H + G) * dk], x[:, (H + G) * dk:]
    if normed:
        q, k = pm.rms(q, eps) * qw.double(), pm.rms(k, eps) * kw.double()
    q = pm.turn(q.reshape(n, H, dk), pos, rot, pairing == "halves")
    k = pm.turn(k.reshape(n, G, dk), pos, rot, pairing == "halves")
    tables = None
    if dims:
        ang = torch.arange(200, dtype=torch.float64)[:, None] * torch.tensor(pm.frequencies(dims, 100.0, None)[0], dtype=torch.float64)
        tables = (torch.cos(ang).float().cuda(), torch.sin(ang).float().cuda())
    pages = [5, 2, 7]
    wide = torch.full((n + 1, width + 24), 3.0, dtype=tdt, device="cuda")
    wide[:n, :width] = rows.cuda()
    kc, vc = torch.zeros(8, G, PAGE, dk, dtype=tdt, device="cuda"), torch.zeros(8, G, PAGE, dv, dtype=tdt, device="cuda")
    ops.qkv_row_norm_rot_write(wide[:, :width], kc, vc, (qw.cuda(), kw.cuda()) if normed else None, eps, tables, dims, pairing,
                               _i32([pages]), _i32([0] * n + [-1]), _i32(pos.tolist() + [0]), H, G, dk, dv)
    tol = 2e-6 if dtype == "float32" else 5e-3
    _close(wide[:n, :H * dk], q.reshape(n, -1), tol, "q")
    assert (wide[n] == 3.0).all() and (wide[:n, width:] == 3.0).all()
    where = [(pages[p // PAGE], p % PAGE) for p in pos.tolist()]
    _close(torch.stack([kc[a, :, o] for a, o in where]), k, tol, "k")
    assert torch.equal(torch.stack([vc[a, :, o] for a, o in where]).cpu(), rows[:, (H + G) * dk:].reshape(n, G, dv))
    assert int((kc != 0).any(-1).any(1).sum()) == n                # nothing else was written


@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("dtype,proj", [("float32", "float32"), ("bfloat16", "bfloat16"), ("bfloat16", "float32")])
def test_latent_rows(dtype, proj, halves):
    """The latent's norm and the turned parts by tables whose magnitude is not one, from projections of either type."""
    from oracle_engine_b200.csrc import ops
    from oracle_engine_b200.csrc.ops import PAGE
    T = lambda s: torch.float32 if s == "float32" else torch.bfloat16      # noqa: E731
    n, H, dk, r, rd, dims, start, eps = 9, 3, 10, 20, 8, 6, 60, 0.1
    rot = mm.rot(dims, 50.0, mm.yarn(8.0, 64, 8.0, 1.0))
    g = torch.Generator().manual_seed(1)
    d, q = torch.randn(n, r + rd, generator=g).to(T(proj)), torch.randn(n, H * (dk + rd), generator=g).to(T(dtype))
    w = torch.randn(r, generator=g)
    pos = torch.arange(start, start + n)
    f, mag = pm.frequencies(dims, 50.0, rot["scaling"])
    ang = torch.arange(100, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    tables = ((mag * torch.cos(ang)).float().cuda(), (mag * torch.sin(ang)).float().cuda())
    cache = torch.zeros(4, PAGE, r + rd, dtype=T(dtype), device="cuda")
    qfull = torch.zeros(n, H * (r + rd), dtype=T(dtype), device="cuda")
    ctx = _step([n], [0], [start])
    ops.latent_write(d.cuda(), w.cuda(), eps, q.cuda(), qfull, None, dims, cache, _i32([[3, 1]]), ctx, H, dk, r, rd, True,
                     tables_cs=tables, halves=halves)
    tol = 2e-6 if dtype == "float32" else 5e-3
    got = torch.stack([cache[[3, 1][p // PAGE], p % PAGE] for p in pos.tolist()])
    _close(got[:, :r], pm.rms(d.double()[:, :r], eps) * w.double(), tol)
    _close(got[:, r:], pm.turn(d.double()[:, None, r:], pos, rot, halves)[:, 0], tol)
    _close(qfull.view(n, H, r + rd)[:, :, r:], pm.turn(q.double().view(n, H, dk + rd)[..., dk:], pos, rot, halves), tol)


@pytest.mark.parametrize("T", [1, 40, 400])
@pytest.mark.parametrize("E,top", [(8, 2), (5, 5), (33, 3), (80, 2), (1, 1)])
def test_router_bias(T, E, top):
    """A bias of the logits' size moves the choice and the weights: the routing kernel, and the router in one launch."""
    from oracle_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(T + E)
    h, w = torch.randn(T, 96, generator=g).bfloat16(), (torch.randn(E, 96, generator=g) * 0.2).bfloat16()
    bias = torch.randn(E, generator=g) * 2
    z = h.double() @ w.double().T
    want, gap = pm.route(z + bias.double(), top)
    seq = torch.zeros(T, dtype=torch.int32, device="cuda")
    sure = gap > 1e-4
    assert sure.float().mean() > 0.9 and (T < 40 or E == top or (pm.route(z, top)[0] - want).abs().max() > 0.2)
    runs = {"route": lambda d: ops.moe_route(z.float().cuda(), E, top, False, d, seq, bias=bias.cuda())}
    if E <= 64:
        runs["router"] = lambda d: ops.moe_router(h.cuda(), w.cuda(), E, top, False, d, seq, "softmax", bias.cuda())
    for name, run in runs.items():
        dense = torch.full((T, E), 9.0, device="cuda")
        run(dense)
        assert (dense.double().cpu()[sure] - want[sure]).abs().max().item() < 2e-5, name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_scale(dtype):
    from oracle_engine_b200.csrc import ops
    table = torch.randn(50, 33).to(torch.float32 if dtype == "float32" else torch.bfloat16)
    x, err = torch.empty(3, 33, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.embed_gather(x, table.cuda(), _i32([4, 49, 0]), err, 17.3)
    _close(x, table.double()[[4, 49, 0]] * 17.3, 1e-6)


@pytest.mark.parametrize("dtype,C,taps", [("float32", 37, 4), ("bfloat16", 64, 4), ("bfloat16", 64, 3), ("bfloat16", 96, 2), ("float32", 20, 1),
                                          ("bfloat16", 50, 7), ("float32", 16, 32), ("bfloat16", 2048, 4)])
def test_convolution_over_cuts_and_slots(dtype, C, taps):
    """Three sequences in slots of their own, in steps of many sizes (whole, pieces shorter than the window, single tokens,
    batches that mix them), a slot that is used again: as the convolution of the whole sequences."""
    from oracle_engine_b200.csrc import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(C + taps)
    n = 700 if C > 1000 else 90
    seqs = [(torch.randn(n, C, generator=g)).to(tdt) for _ in range(4)]
    k, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    want = [pm.silu(pm.causal_conv(s.double(), k.double(), b.double())) for s in seqs]
    state = torch.full((5, max(taps - 1, 1), C), 7.0, device="cuda")
    slot_of, done, got = {0: 3, 1: 0, 2: 4}, [0] * 4, [torch.zeros(n, C) for _ in range(4)]

    def start(i, slot):
        slot_of[i] = slot
        state[slot] = 0
    for i in range(3):
        start(i, slot_of[i])

    def step(bring):
        lens = [m for _, m in bring]
        ctx = _step(lens, [slot_of[i] for i, _ in bring])
        wide = torch.full((ctx.n_tokens, C + 16), 9.0, dtype=tdt)
        wide[:, :C] = torch.cat([seqs[i][done[i]:done[i] + m] for i, m in bring])
        out = torch.zeros(ctx.n_tokens, C, dtype=tdt, device="cuda")
        ops.causal_conv(out, wide.cuda()[:, :C], k.T.contiguous().cuda(), b.cuda(), state, ctx)
        row = 0
        for i, m in bring:
            got[i][done[i]:done[i] + m] = out[row:row + m].float().cpu()
            done[i] += m
            row += m
    step([(0, 1), (1, n - 12), (2, 2)])
    for _ in range(3):
        step([(0, 1), (1, 1), (2, 1)])
    step([(0, 2), (2, 1), (1, 5)])
    step([(2, n - done[2]), (0, 33)])
    step([(1, n - done[1])])
    start(3, slot_of.pop(2))                              # the freed slot's next user
    step([(3, n), (0, n - done[0])])
    for i in range(4):
        _close(got[i], want[i], 2e-6 if dtype == "float32" else 6e-3, i)
    assert (state[[1, 2]] == 7.0).all()                    # slots nobody held


def _scan_inputs(T, C, N, tdt, g):
    r = lambda *s: torch.randn(*s, generator=g)                            # noqa: E731
    return SimpleNamespace(u=r(T, C).to(tdt), z=r(T, C).to(tdt), zdt=r(T, C), thin=r(T, 5 + 2 * N), bias=r(C) * 0.7 - 2.5,
                           A=-torch.exp(r(C, N) * 0.7 - 0.7), D=r(C))


def _scan_want(x, N):
    dt = torch.nn.functional.softplus(x.zdt.double() + x.bias.double())
    y = pm.scan(x.u.double(), dt, x.A.double(), x.thin.double()[:, 5:5 + N], x.thin.double()[:, 5 + N:])
    return (y + x.D.double() * x.u.double()) * pm.silu(x.z.double())


@pytest.mark.parametrize("dtype,C,N", [("float32", 37, 16), ("bfloat16", 100, 16), ("bfloat16", 64, 1), ("float32", 33, 5), ("bfloat16", 40, 32),
                                       ("bfloat16", 24, 100), ("float32", 20, 200), ("bfloat16", 16, 256), ("bfloat16", 3000, 64)])
def test_selective_scan_over_cuts_slots_and_segments(dtype, C, N):
    """The recurrence against the plain one: unequal sequences in slots out of order, cut into steps down to one token, a
    padding sequence beside them; in bfloat16 also as segments side by side (lengths that are and are not multiples of a
    segment, sequences shorter than one) and with the step sizes' product inside."""
    from oracle_engine_b200.csrc import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(C + N)
    lens = [70, 3, 40]
    xs = [_scan_inputs(n, C, N, tdt, g) for n in lens]
    for x in xs[1:]:
        x.bias, x.A, x.D = xs[0].bias, xs[0].A, xs[0].D
    want = [_scan_want(x, N) for x in xs]
    A2 = (xs[0].A.double() * 1.4426950408889634).float().cuda()
    bias, D = xs[0].bias.cuda(), xs[0].D.cuda()
    slots = [4, 1, 2]
    tol = 2e-5 if dtype == "float32" else 1e-2

    def run(cuts, segments=None, pad=False, fused=None):
        """cuts: per step, how many tokens each sequence brings."""
        state = torch.full((6, C, N), 5.0, device="cuda")
        state[slots] = 0
        got, at = [[] for _ in lens], [0] * 3
        for bring in cuts:
            who = [i for i in range(3) if bring[i]]
            ctx = _step([bring[i] for i in who] + ([0] if pad else []), [slots[i] for i in who] + ([-1] if pad else []))
            part = lambda name: torch.cat([getattr(xs[i], name)[at[i]:at[i] + bring[i]] for i in who]).cuda()   # noqa: E731
            T = ctx.n_tokens
            y, thin = torch.zeros(T, C, dtype=tdt, device="cuda"), part("thin").contiguous()
            z = torch.cat([part("u"), part("z")], 1)[:, C:]                    # columns of a wider buffer
            if segments:
                seg_len = segments
                n_seg = -(-ctx.max_qlen // seg_len)
                extra = (seg_len, n_seg, torch.empty(ctx.n_seqs * n_seg, C * N, device="cuda"), torch.empty(ctx.n_seqs * n_seg, C, device="cuda"))
            ops.selective_scan(y, state, part("u"), part("zdt"), bias, thin, 5, 5 + N, A2, D, z, ctx, segments=extra if segments else None)
            row = 0
            for i in who:
                got[i].append(y[row:row + bring[i]])
                row += bring[i]
                at[i] += bring[i]
        assert (state[[0, 3, 5]] == 5.0).all()
        return [torch.cat(p) for p in got], state
    whole, end = run([lens], pad=True)
    for i in range(3):
        _close(whole[i], want[i], tol, i)
    pieces, end2 = run([[20, 1, 0], [1, 1, 1], [1, 1, 1], [2, 0, 38], [46, 0, 0]])
    for i in range(3):
        _close(pieces[i], want[i], tol, i)
    if dtype == "float32":
        assert all(torch.equal(a, b) for a, b in zip(whole, pieces)) and torch.equal(end, end2)
        return
    _close(end2, end.double().cpu(), 1e-5)
    for seg in (8, 16, 24, 64):
        side, end3 = run([lens], segments=seg, pad=True)
        for i in range(3):
            _close(side[i], want[i], tol, (seg, i))
        _close(end3, end.double().cpu(), 1e-5)
    side, end3 = run([[30, 1, 0], [40, 2, 40]], segments=8)
    for i in range(3):
        _close(side[i], want[i], tol, i)


@pytest.mark.parametrize("dtype,C,N,rank,B", [("float32", 37, 16, 12, 3), ("bfloat16", 100, 16, 8, 1), ("bfloat16", 64, 1, 1, 5),
                                              ("bfloat16", 40, 32, 12, 40), ("bfloat16", 24, 100, 130, 6), ("float32", 20, 200, 5, 2),
                                              ("bfloat16", 4096, 16, 128, 33), ("bfloat16", 16, 256, 24, 7), ("bfloat16", 1000, 5, 40, 70)])
def test_one_token_with_the_step_sizes_inside(dtype, C, N, rank, B):
    """The one-launch step for batches of single tokens, in groups of sequences and alone, padding rows among them."""
    from oracle_engine_b200.csrc import ops
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(C + N + B)
    ld = -(-rank // 8) * 8
    x = _scan_inputs(B, C, N, tdt, g)
    w = (torch.randn(C, rank, generator=g) / rank ** 0.5).to(tdt)
    thin = torch.randn(B, ld + 2 * N, generator=g)
    S = torch.randn(B + 3, C, N, generator=g)
    slots = torch.randperm(B + 3, generator=g)[:B].tolist()
    live = [b for b in range(B) if b not in (2, B - 1) or B < 4]
    lens = [1 if b in live else 0 for b in range(B)]
    ctx = _step([1] * B, [slots[b] if lens[b] else -1 for b in range(B)])
    cu = np.concatenate([[0], np.cumsum(lens)])
    order = [b for b in range(B) if lens[b]]                   # a real sequence's row is the number of real ones before it
    ctx.cu_q = _i32(cu)
    rows = torch.tensor(order)
    pick = lambda t: torch.cat([t[rows], t[:B - len(order)]]).cuda()       # noqa: E731
    state, y = S.cuda(), torch.full((B, C), 3.0, dtype=tdt, device="cuda")
    A2 = (x.A.double() * 1.4426950408889634).float().cuda()
    ops.selective_step(y, state, pick(x.u), torch.nn.functional.pad(w, (0, ld - rank)).cuda(), 0, rank, x.bias.cuda(), pick(thin), ld,
                       ld + N, A2, x.D.cuda(), pick(x.z), ctx)
    dt = torch.nn.functional.softplus(thin.double()[:, :rank] @ w.double().T + x.bias.double())
    for k, b in enumerate(order):
        new = torch.exp(dt[b][:, None] * x.A.double()) * S[slots[b]].double() + (dt[b] * x.u[b].double())[:, None] * thin[b].double()[ld:ld + N]
        want = (new @ thin[b].double()[ld + N:] + x.D.double() * x.u[b].double()) * pm.silu(x.z[b].double())
        _close(y[k], want, 2e-5 if dtype == "float32" else 1e-2, b)
        _close(state[slots[b]], new, 1e-5, b)
    untouched = [s for s in range(B + 3) if s not in [slots[b] for b in order]]
    assert torch.equal(state.cpu()[untouched], S[untouched]) and (y[len(order):] == 3.0).all()


# (dtype, key size, value size, heads, key heads): tensor-core kernel and the one path
ATTENTION = [("float32", 20, 28, 4, 2), ("bfloat16", 48, 96, 6, 2), ("bfloat16", 128, 128, 8, 2), ("bfloat16", 24, 40, 4, 2), ("bfloat16", 32, 16, 20, 1)]
LATENT = [("float32", 20, 6, 3), ("bfloat16", 112, 48, 6), ("bfloat16", 192, 64, 16), ("bfloat16", 33, 4, 1), ("bfloat16", 272, 32, 5)]


def _edge_probes(n, window):
    return [window - 1, window, 130, 149, 180, 198, 199] if window < 130 else [window - 1, window, 170, 198, 199]


def _planted(q, k, probes, window, inside, at):
    """Query and key rows in which, per probe, one key stands out: the last one the window still holds, or the next."""
    chosen = []
    for a, t in enumerate(probes):
        j = t - window + (1 if inside else 0)
        chosen.append(j if j >= 0 else None)
        if j < 0:
            continue
        k[..., at + a] = 0
        q[t] = 0
        q[t, ..., at + a] = 8.0
        k[j, ..., at + a] = 5.0                              # a score of 40 against about one
    return chosen


@pytest.mark.parametrize("gate", ["value", "head", None])
@pytest.mark.parametrize("sink", [True, False])
@pytest.mark.parametrize("window", [70, 64, 140])
@pytest.mark.parametrize("dtype,dk,dv,H,G", ATTENTION)
def test_attention_with_one_key_that_stands_out(dtype, dk, dv, H, G, window, sink, gate):
    """Window, sink and gate over scattered pages, for queries in a prompt, in a second piece and decoded alone: the key just
    inside the window's edge decides the output, the one just outside is not seen; and the whole against the plain form."""
    from oracle_engine_b200.csrc.ops import PAGE
    from oracle_engine_b200.engine.runtime import Runtime
    from oracle_engine_b200.parts import attention_dispatch as ad
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    n, cuts = 200, [0, 150, 198, 199, 200]
    gen = torch.Generator().manual_seed(5)
    r = lambda *s: torch.randn(*s, generator=gen)                          # noqa: E731
    rt = Runtime(tdt, torch.device("cuda"), True)
    tables = torch.full((1, 6), -1, dtype=torch.int32)
    tables[0, :4] = torch.tensor([5, 2, 7, 0])
    probes = _edge_probes(n, window)
    sinks = r(H) * 2 + 1 if sink else None
    gates = None if gate is None else r(n, H * dv if gate == "value" else H).to(tdt)
    for inside in (True, False, None):
        q, k, v = r(n, H, dk) * 0.3, r(n, G, dk) * 0.3, r(n, G, dv)
        chosen = _planted(q, k, probes, window, inside, 3) if inside is not None else []
        q, k, v = (x.to(tdt) for x in (q, k, v))
        seen = pm.visible(n, window)
        want = torch.zeros(n, H, dv, dtype=torch.float64)
        for h in range(H):
            g = h // (H // G)
            s = (q[:, h].double() @ k[:, g].double().T).masked_fill(~seen, -float("inf"))
            want[:, h] = pm.softmax_with_sink(s, None if sinks is None else sinks[h].double()) @ v[:, g].double()
        bare = want.clone()
        if gates is not None:
            want *= torch.sigmoid(gates.double()).view(n, H, -1)
        kc, vc = torch.zeros(8, G, PAGE, dk, dtype=tdt, device="cuda"), torch.zeros(8, G, PAGE, dv, dtype=tdt, device="cuda")
        for j in range(n):
            kc[tables[0, j // PAGE], :, j % PAGE], vc[tables[0, j // PAGE], :, j % PAGE] = k[j].cuda(), v[j].cuda()
        got = torch.zeros(n, H * dv, dtype=tdt, device="cuda")
        for lo, hi in zip(cuts[:-1], cuts[1:]):
            ctx = _step([hi - lo], [0], [lo])
            out = torch.zeros(hi - lo, H * dv, dtype=tdt, device="cuda")
            gw = None
            if gates is not None:                             # columns of a wider buffer
                gw = torch.cat([gates[lo:hi, :8], gates[lo:hi]], 1).cuda()[:, min(8, gates.shape[1]):]
            ad.split_attend(rt, out, q[lo:hi].reshape(hi - lo, -1).cuda(), kc, vc, tables.cuda(), ctx, H, G, dk, dv, window, 1.0, 0.0,
                            None if sinks is None else sinks.cuda(), gate=gw)
            got[lo:hi] = out
        _close(got, want.reshape(n, -1), 2e-5 if dtype == "float32" else 2e-2, (inside,))
        for t, j in zip(probes, chosen):
            if j is None:
                continue
            o = bare[t] if gates is None else got[t].double().cpu().view(H, dv) / torch.sigmoid(gates[t].double()).view(H, -1)
            for h in range(H):
                d = (o[h] - v[j, h // (H // G)].double()).abs().max().item()
                assert (d < 0.2) == inside, (inside, t, h, d)


@pytest.mark.parametrize("window", [70, 64, 0])
@pytest.mark.parametrize("sink,gate", [(True, True), (False, True), (True, False)])
@pytest.mark.parametrize("dtype,r,rd,H", LATENT)
def test_latent_attention_with_one_key_that_stands_out(dtype, r, rd, H, sink, gate, window):
    """The same over rows of latents: the value is the key row's first part, read by every head."""
    from oracle_engine_b200.csrc.ops import PAGE
    from oracle_engine_b200.engine.runtime import Runtime
    from oracle_engine_b200.parts import attention_dispatch as ad
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    n, cuts, R = 200, [0, 150, 198, 199, 200], r + rd
    gen = torch.Generator().manual_seed(6)
    rnd = lambda *s: torch.randn(*s, generator=gen)                        # noqa: E731
    rt = Runtime(tdt, torch.device("cuda"), True)
    tables = torch.full((1, 6), -1, dtype=torch.int32)
    tables[0, :4] = torch.tensor([5, 2, 7, 0])
    probes = _edge_probes(n, window or 199)
    sinks = rnd(H) * 2 + 1 if sink else None
    gates = rnd(n, H).to(tdt) if gate else None
    for inside in (True, False):
        q, k = rnd(n, H, R) * 0.3, rnd(n, 1, R) * 0.3
        chosen = _planted(q, k, probes, window, inside, 3) if window else []
        q, k = q.to(tdt), k[:, 0].to(tdt)
        seen = pm.visible(n, window)
        want = torch.zeros(n, H, r, dtype=torch.float64)
        for h in range(H):
            s = (q[:, h].double() @ k.double().T).masked_fill(~seen, -float("inf"))
            want[:, h] = pm.softmax_with_sink(s, None if sinks is None else sinks[h].double()) @ k[:, :r].double()
        bare = want.clone()
        if gates is not None:
            want *= torch.sigmoid(gates.double())[:, :, None]
        rows = torch.zeros(8, PAGE, R, dtype=tdt, device="cuda")
        for j in range(n):
            rows[tables[0, j // PAGE], j % PAGE] = k[j].cuda()
        got = torch.zeros(n, H * r, dtype=tdt, device="cuda")
        for lo, hi in zip(cuts[:-1], cuts[1:]):
            ctx = _step([hi - lo], [0], [lo])
            out = torch.zeros(hi - lo, H * r, dtype=tdt, device="cuda")
            gw = None if gates is None else torch.cat([gates[lo:hi], gates[lo:hi]], 1).cuda()[:, H:]
            ad.latent_core(rt, out, q[lo:hi].reshape(hi - lo, -1).cuda(), rows, tables.cuda(), ctx, H, r, rd, 1.0, window,
                           None if sinks is None else sinks.cuda(), gw)
            got[lo:hi] = out
        _close(got, want.reshape(n, -1), 2e-5 if dtype == "float32" else 2e-2, (inside,))
        for t, j in zip(probes, chosen):
            if j is None:
                continue
            d = (bare[t] - k[j, :r].double()).abs().amax(1)
            assert ((d < 0.2) == inside).all(), (inside, t, d)


# ------------------------------------------------------------------------------------------ layers and schedules

@pytest.mark.parametrize("name", ["M1", "M2", "M3"])
def test_every_layer_by_itself_float32(models, name):
    """The stream that leaves each entry of the schedule for a whole prompt, in float32, against the plain model; then the
    same prompt's last 20 tokens one by one."""
    from oracle_engine_b200 import SequenceStep
    folder, plain = models[name]
    eng = _engine(folder, "float32", use_graphs=False)
    seen = []
    for layer in eng.model.layers:
        def fwd(x, *a, _orig=layer.forward, **k):
            _orig(x, *a, **k)
            seen.append(x.detach().double().cpu())
        layer.forward = fwd
    toks = helpers.random_tokens(150, plain.cfg["vocab"], 9)
    want = plain.layers(toks)
    slot = eng.alloc()
    eng.step([SequenceStep(slot, toks[:130], [129])])
    assert len(seen) == len(want) == len(plain.cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, want)):
        err = (a - b[:130]).abs().max().item()
        assert err < 1e-4 * max(1.0, b.abs().max().item()), f"{name}: layer {i} differs by {err}"
    for t in range(130, 150):
        seen.clear()
        eng.step([SequenceStep(slot, toks[t:t + 1], [0])])
        for i, (a, b) in enumerate(zip(seen, want)):
            err = (a[0] - b[t]).abs().max().item()
            assert err < 1e-4 * max(1.0, b.abs().max().item()), f"{name}: token {t} alone, layer {i} differs by {err}"
    eng.free(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2", "M3"])
def test_whole_decoded_pieces_and_batches_agree_with_plain(models, tmp_path, name, dtype):
    folder, plain = models[name]
    vocab = plain.cfg["vocab"]
    lens = [130, 65, 1, 200, 37, 2, 64, 129]
    requests = [helpers.random_tokens(n, vocab, 300 + i) for i, n in enumerate(lens)]
    eng = _engine(folder, dtype)
    runs = {}
    # each alone and whole; each alone decoded token by token from the first token (or after a prompt)
    runs["whole"] = helpers.whole_steps(requests)
    runs["decoded"] = helpers.tail_steps(requests, 1000)
    runs["tail"] = helpers.tail_steps(requests, 40)
    # in pieces down to two tokens and one
    runs["pieces"] = helpers.piece_steps(requests, [helpers.cut(n, [2, 37, 1, 64, 3, 65]) for n in lens], batch_size=1)
    runs["pairs"] = helpers.piece_steps(requests[1:3] + requests[4:6], [helpers.cut(n, [2]) for n in (65, 1, 37, 2)],
                                        batch_size=1)
    # ragged batches of three, prompts then one token each; the next batch takes the slots they leave
    runs["batched"] = helpers.batched_steps(requests, [max(1, n - 20) for n in lens], 3)
    # steps that mix a prompt piece of one request with single tokens of others
    runs["mixed"] = helpers.piece_steps(requests, [helpers.cut(n, [1, 1, 30, 1, 2, 70][i % 3:] + [5]) for i, n in enumerate(lens)],
                                        batch_size=3)
    got = {}
    for k, steps in runs.items():
        reqs = requests[1:3] + requests[4:6] if k == "pairs" else requests
        got[k] = _run(eng, tmp_path / k, steps, reqs)
        _compare(got[k], plain, reqs, TOL[dtype], f"{name} {dtype} {k}")
    if dtype == "float32":
        # a position's logits do not depend on the cut or the batch: the same instructions in the same order
        for k in got:
            reqs = [1, 2, 4, 5] if k == "pairs" else range(len(requests))
            for j, i in enumerate(reqs):
                assert np.array_equal(got["whole"][i], got[k][j]), f"{name} float32: {k} differs from whole, request {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_page_borders_and_window_edges_under_a_peaked_softmax(models, tmp_path, dtype):
    """Windows of 100, 64, 33 and 150 keys under scores so large that single keys decide: prompts that end just before, at
    and just after page borders and windows, decoded across the next ones.  (tests/test_mavinex_cpu.py shows that a window
    one position off moves most positions by ten tolerances.)"""
    folder, plain = models["SHARP"]
    toks = helpers.random_tokens(330, plain.cfg["vocab"], 77)
    lens = [32, 33, 34, 63, 64, 65, 66, 67, 99, 100, 101, 128, 129, 149, 150, 151, 199, 201, 330]
    requests = [toks[:n] for n in lens]
    eng = _engine(folder, dtype, max_tokens=2048)
    runs = {"whole": helpers.whole_steps(requests),
            "tail": helpers.tail_steps(requests, 6),
            "decoded": helpers.tail_steps(requests[-1:], 300),
            "pieces": helpers.piece_steps(requests, [helpers.cut(n, [62, 2, 1, 63, 64]) for n in lens], batch_size=2)}
    for kname, steps in runs.items():
        reqs = requests[-1:] if kname == "decoded" else requests
        got = _run(eng, tmp_path / kname, steps, reqs)
        _compare(got, plain, reqs, TOL[dtype] * 2, f"SHARP {dtype} {kname}")


def test_pages_behind_the_windows_are_given_back(models):
    """While a sequence decodes, every group holds the pages of its window and no more; a pool that could not hold the whole
    sequences serves them."""
    from oracle_engine_b200 import SequenceStep
    folder, plain = models["SHARP"]
    eng = _engine(folder, "float32", max_tokens=512)
    toks = helpers.random_tokens(400, plain.cfg["vocab"], 3)
    want = plain.logits(toks).numpy()
    slot = eng.alloc()
    eng.step([SequenceStep(slot, toks[:30], [])])
    for t in range(30, 400):
        got = eng.step([SequenceStep(slot, toks[t:t + 1], [0])])[0].cpu().numpy()
        err = np.sqrt(((got - want[t]) ** 2).mean()) / np.sqrt((want ** 2).mean())
        assert err < TOL["float32"], (t, err)
        for g in eng.cache.groups:
            first = max(0, t - g.need.window + 1) // 64
            held = np.nonzero(g.tables[slot] >= 0)[0].tolist()
            assert held == list(range(first, t // 64 + 1)), (t, g.need)
    eng.free(slot)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_real_sizes(tmp_path, dtype):
    """Heads of 128 beside 2,048 channels of 16 states, and latents of 192 + 64, at a width of 1,024: in bfloat16 the prompts
    go through the tensor-core products with the branches' joined input and the scan's segments, decoding through the
    kernels that split the keys and the one-launch scan."""
    folder = mm.write(tmp_path / "m", mm.REAL, 31, std=0.03, router_scale=6.0)
    plain = pm.PlainMavinex(folder)
    lens = [333, 70, 200, 530]
    requests = [helpers.random_tokens(n, 1000, 800 + i) for i, n in enumerate(lens)]
    eng = _engine(folder, dtype, max_tokens=2048)
    if dtype == "bfloat16":
        assert eng.model.layers[0].mixer.w_joined is not None
    runs = {"batched": helpers.batched_steps(requests, [n - 6 for n in lens], 4),
            "pieces": helpers.piece_steps(requests, [helpers.cut(n, [150, 2, 100]) for n in lens], batch_size=1)}
    for k, steps in runs.items():
        got = _run(eng, tmp_path / k, steps, requests)
        _compare(got, plain, requests, TOL[dtype], f"REAL {dtype} {k}")
    short = [r[:9] for r in requests]
    for k, steps in {"short_alone": helpers.tail_steps(short[:1], 1000),
                     "short_batch": helpers.batched_steps(short, [1, 2, 3, 4], 4)}.items():
        reqs = short[:1] if k == "short_alone" else short
        got = _run(eng, tmp_path / k, steps, reqs)
        _compare(got, plain, reqs, TOL[dtype], f"REAL {dtype} {k}")
    eng.check_device_errors()


@pytest.mark.parametrize("seed", [41, 42, 43, 44, 45, 46, 47, 48])
def test_configurations_drawn_at_random(tmp_path, seed):
    """Any number of layers, sizes that are and are not multiples of 16, optional parts present or absent, layers on any
    earlier layer's weights: whole prompts, a prompt and 34 single tokens, and a ragged batch, in both precisions."""
    raw = mm.random_config(random.Random(seed))
    folder = mm.write(tmp_path / "m", raw, seed, std=0.06, router_scale=3.0)
    plain = pm.PlainMavinex(folder)
    lens = [1, 45, 230, 131]
    requests = [helpers.random_tokens(n, raw["vocab"], 7 * seed + i) for i, n in enumerate(lens)]
    for dtype in ("float32", "bfloat16"):
        eng = _engine(folder, dtype, max_tokens=2048)
        runs = {"whole": helpers.whole_steps(requests), "tail": helpers.tail_steps(requests, 34),
                "batched": helpers.batched_steps(requests, [max(1, n - 20) for n in lens], 4)}
        for k, steps in runs.items():
            got = _run(eng, tmp_path / f"{dtype}{k}", steps, requests)
            _compare(got, plain, requests, TOL[dtype], f"random {seed} {dtype} {k}")
        eng.check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_are_used_again(models, tmp_path, dtype):
    """Two slots for six requests, in a cache of four pages a sequence: a request that starts in a slot and on pages
    another left reads nothing of it, neither keys nor states nor the convolution's inputs."""
    folder, plain = models["M1"]
    lens = [70, 40, 90, 66, 5, 120]
    requests = [helpers.random_tokens(n, plain.cfg["vocab"], 500 + i) for i, n in enumerate(lens)]
    eng = _engine(folder, dtype, max_tokens=256, n_slots=2)
    steps = helpers.batched_steps(requests, [max(1, n - 8) for n in lens], 2)
    got = _run(eng, tmp_path / "t", steps, requests)
    _compare(got, plain, requests, TOL[dtype], f"reuse {dtype}")
    assert eng.cache.slots.n_free == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2"])
def test_long_decoding_through_generate(models, name, dtype):
    """Greedy generation through Engine.generate (scheduler, sampler, step ahead) against the plain model."""
    from oracle_engine_b200 import GenParams
    folder, plain = models[name]
    vocab = plain.cfg["vocab"]
    eng = _engine(folder, dtype)
    prompts = [helpers.random_tokens(n, vocab, 40 + i) for i, n in enumerate((1, 9, 70))]
    n_new = 150
    got = eng.generate(prompts, GenParams.greedy(n_new, ignore_eos=True))
    assert [len(g) for g in got] == [n_new] * 3
    margin = 1e-3 if dtype == "float32" else 2 * TOL[dtype]
    for p, g in zip(prompts, got):
        lg = plain.logits(list(p) + list(g))
        close = plain.close_calls(list(p) + list(g), CLOSE_CALL) if dtype == "bfloat16" else set()
        scale = float(lg.pow(2).mean().sqrt())
        for j, tok in enumerate(g):
            if len(p) + j - 1 in close:
                continue
            row = lg[len(p) + j - 1]
            assert row.max().item() - row[tok].item() <= margin * max(1.0, scale), f"{dtype}: token {j} of a prompt of {len(p)}"
    # a budget of prompt tokens per step: the 70-token prompt goes through in portions beside decoding rows
    again = eng.generate(prompts, GenParams.greedy(12, ignore_eos=True), max_step_tokens=16)
    if dtype == "float32":
        assert again == [g[:12] for g in got]
    eng.cache.check()
    assert eng.cache.slots.n_free == eng.cache.n_slots


def test_command_lines(models, tmp_path):
    """bin/trace_run and bin/oracle load the design by its config.json."""
    folder, plain = models["M1"]
    vocab = plain.cfg["vocab"]
    requests = [helpers.random_tokens(n, vocab, 900 + i) for i, n in enumerate((20, 66))]
    steps = helpers.batched_steps(requests, [15, 60], 2)
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        helpers.run_trace_cli(folder, dtype, steps, out, 256)
        files = {s["step"]: np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab) for s in steps}
        got = helpers.collect(steps, files, requests)
        _compare(got, plain, requests, TOL[dtype], f"trace_run {dtype}")
    prompt = requests[0][:12]
    r = subprocess.run([sys.executable, str(helpers.ROOT / "bin" / "oracle"), "-m", folder, "--tokens",
                        ",".join(map(str, prompt)), "-n", "6", "--temp", "0", "--repeat-penalty", "1", "--dtype", "float32", "--ignore-eos"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()] == pm.generate(plain, prompt, 6)
