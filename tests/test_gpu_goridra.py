"""The Goridra design on the GPU against the plain float64 model of tests/plain_goridra.py: every mechanism's kernels
alone, every layer by itself, whole prompts, token-by-token decoding, prompts in pieces down to two tokens, ragged batches,
reused slots and pages, keys far away, at page borders and at the chunks' edges under a peaked softmax, layers that read
another layer's keys with a mask of their own, sizes of real models, and greedy generation through Engine.generate and the
command lines."""
import copy
import random
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import goridra_models as gm
import helpers
import plain_goridra as pg

pytestmark = pytest.mark.gpu

# A position's error is the root mean square over the vocabulary of the difference of its logits, relative to
# the root mean square of the request's logits.  float32: rounding of a few hundred fused multiply-adds per
# value; bfloat16: activations rounded to 2^-9 relative at every product, a few dozen products deep.
TOL = {"float32": 1e-4, "bfloat16": 5e-2}
# bfloat16 moves a router's logits by a few hundredths (they are scaled up to several units); a choice that hangs on less
# than this is a close call, and such positions are left out of the bfloat16 comparison
CLOSE_CALL = 0.08


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (raw, seed) in gm.ALL.items():
        d = gm.write(tmp_path_factory.mktemp(f"goridra_{name}"), raw, seed)
        out[name] = (d, pg.PlainGoridra(d))
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


# ------------------------------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,D", [(5, 100), (3, 7), (1, 2048), (9, 9000), (1100, 96), (1030, 1500), (1024, 3000), (1024, 4096)])
def test_layer_norm(dtype, rows, D):
    """Block per row (plain and in 16-byte pieces, also rows longer than its registers) and warp per row; a mean far above
    the deviations, and an eps of their size."""
    from oracle_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(rows + D)
    x = torch.randn(rows, D, generator=g) * 0.2 + 3.0
    w, b = torch.randn(D, generator=g), torch.randn(D, generator=g)
    y = torch.empty(rows, D, dtype=dtype, device="cuda")
    ops.layernorm(y, x.cuda(), w.cuda(), b.cuda(), 0.03)
    want = pg.layer_norm(x.double(), w.double(), b.double(), 0.03)
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    assert (y.double().cpu() - want).abs().max().item() < tol * want.abs().max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gelu_and_cap_kernels(dtype):
    from oracle_engine_b200.csrc import ops
    z = torch.linspace(-9, 9, 3001).to(dtype).double()
    a = z.to(dtype).cuda()
    ops.gelu_(a)
    err = (a.double().cpu() - pg.gelu(z)).abs()
    assert (err < (1e-6 if dtype == torch.float32 else 4e-3) * (1 + z.abs())).all()
    x = (z * 20).float().cuda()
    ops.softcap_rows(x, 7.5)
    assert (x.double().cpu() - 7.5 * torch.tanh(z.float().double() * 20 / 7.5)).abs().max().item() < 2e-6 * 7.5 + 1e-5


@pytest.mark.parametrize("E,top,groups", [(8, 2, None), (8, 4, (4, 2)), (6, 2, (6, 2)), (80, 3, (40, 5)), (33, 2, (11, 3)),
                                          (1024, 5, (512, 9)), (4, 4, (1, 1)), (16, 1, (2, 1)), (5, 1, None)])
def test_routing_kernel(E, top, groups):
    """The choice by groups and the weights over all experts' softmax, logits of several sizes, padding rows; ties go to
    the lower index and the lower group."""
    from oracle_engine_b200.csrc import ops
    T = 37
    z = torch.randn(T, E, generator=torch.Generator().manual_seed(E + top)) * 3.0
    z[5] *= 20                                            # far apart: the smaller scores underflow
    seq = torch.zeros(T, dtype=torch.int32)
    seq[11] = -1
    dense = torch.full((T, E), 9.0, device="cuda")
    idx, wt = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    ops.moe_route(z.cuda(), E, top, False, dense, seq.cuda(), idx=idx, wt=wt, weights="softmax_all", groups=groups)
    router = {"experts": E, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    want, gap = pg.route(z.double(), router)
    got = dense.double().cpu()
    assert got[11].abs().max().item() == 0
    rows = [t for t in range(T) if t != 11 and gap[t] > 1e-6]
    assert len(rows) > 30
    assert (got[rows] - want[rows]).abs().max().item() < 2e-6
    assert got[rows][want[rows] == 0].abs().max().item() == 0 if top < E else True      # an expert not chosen has no weight
    for t in rows:
        assert torch.allclose(dense[t][idx[t].long()], wt[t], atol=1e-7) and len(set(idx[t].tolist())) == top
    if groups:                                            # equal scores everywhere: the first groups' first experts
        dense.fill_(9.0)
        ops.moe_route(torch.zeros(T, E).cuda(), E, top, False, dense, torch.zeros(T, dtype=torch.int32).cuda(),
                      weights="softmax_all", groups=groups)
        assert (dense[:, :top] - 1.0 / top).abs().max().item() < 1e-6 and not dense[:, top:].any()
    with pytest.raises(ops.KernelError):
        ops.moe_route(z.cuda(), E, top, False, dense, seq.cuda(), weights="softmax_all", groups=(E, 0))


@pytest.mark.parametrize("T", [1, 7, 300, 1025])
@pytest.mark.parametrize("E,top,groups,gate,weights", [(8, 2, (4, 2), False, "softmax_all"), (5, 1, None, False, "softmax_all"),
                                                       (7, 3, None, True, "softmax"), (16, 4, (8, 4), False, "softmax_all"),
                                                       (12, 2, None, "one", "sigmoid"), (31, 3, None, True, "softmax"),
                                                       (64, 6, (16, 3), False, "softmax_all")])
@pytest.mark.parametrize("D", [64, 2056])
def test_router_in_one_launch(T, E, top, groups, gate, weights, D):
    """The router's product and the routing in one launch against the routing kernel on float64 logits: the same choice
    wherever it is no close call, whatever else is in the batch."""
    from oracle_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(T + E + D)
    rows = E + (1 if gate is True else 0)
    wide = torch.randn(T, D + 8, generator=g).bfloat16().cuda()
    h, w = wide[:, :D], (torch.randn(rows, D, generator=g) * 2 / D ** 0.5).bfloat16().cuda()
    seq = torch.zeros(T, dtype=torch.int32)
    if T > 5:
        seq[4] = -1
    bias = torch.randn(E, generator=g).cuda() * 0.1 if weights == "sigmoid" else None
    z = h.double() @ w.double().T
    want, got = (torch.full((T, E + int(bool(gate))), 9.0, device="cuda") for _ in range(2))
    ops.moe_route(z.float().contiguous(), E, top, gate, want, seq.cuda(), weights=weights, bias=bias, groups=groups)
    ops.moe_router(h, w, E, top, gate, got, seq.cuda(), weights, bias, groups)
    same = ((got > 0) == (want > 0)).all(1)
    assert same.float().mean().item() > 0.99 or (~same).sum().item() <= 1
    assert (got[same] - want[same]).abs().max().item() < 2e-5
    last = torch.full((1, got.shape[1]), 9.0, device="cuda")                     # the last token alone: the same bits
    ops.moe_router(h[-1:], w, E, top, gate, last, torch.zeros(1, dtype=torch.int32).cuda(), weights, bias, groups)
    assert torch.equal(last[0], got[-1])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff", [24, 10])
def test_squared_relu_experts_kernel(dtype, ff):
    from oracle_engine_b200.csrc import ops
    T, E = 9, 5
    g = torch.Generator().manual_seed(ff)
    u = torch.randn(T, E * ff, generator=g).to(dtype)
    dense = torch.rand(T, E, generator=g) * (torch.rand(T, E, generator=g) < 0.5)
    got = u.cuda()
    ops.moe_dense_relu2(got, dense.cuda(), ff)
    want = torch.relu(u.double()) ** 2 * dense.double().repeat_interleave(ff, 1)
    assert (got.double().cpu() - want).abs().max().item() < (1e-6 if dtype == torch.float32 else 8e-3) * want.max().item()


# products of the three kernels: weight streaming; one SM with swapped operands, K split in a cluster, narrow tiles,
# 128-row tiles; two SMs; with and without a plain part in front, groups that are and are not multiples of 16
@pytest.mark.parametrize("M,N0,F,K,ff", [(1, 64, 96, 128, 24), (8, 512, 1024, 512, 128), (13, 8, 200, 256, 40),
                                         (33, 768, 2048, 2048, 256), (64, 0, 16384, 1024, 1024), (100, 40, 264, 512, 8),
                                         (128, 256, 520, 1024, 40), (200, 24, 600, 128, 100), (300, 1280, 1024, 2048, 128),
                                         (700, 768, 2000, 512, 250), (2100, 512, 1536, 256, 96)])
@pytest.mark.parametrize("act", ["gelu", "relu2", "weighted"])
def test_activated_products(M, N0, F, K, ff, act):
    """act (and the groups' weights) in a product's epilogue, applied from column N0 on, against float64."""
    from oracle_engine_b200.csrc import ops_tc
    g = torch.Generator().manual_seed(M + F)
    a = torch.randn(M, K, generator=g).bfloat16()
    w = (torch.randn(N0 + F, K, generator=g) / K ** 0.5).bfloat16()
    n_groups = -(-F // ff)
    gw = torch.rand(M, n_groups + 1, generator=g) * (torch.rand(M, n_groups + 1, generator=g) < 0.6)
    wide = torch.full((M, N0 + F + 8), 7.0, dtype=torch.bfloat16, device="cuda")      # rows of a wider buffer
    out = wide[:, :N0 + F]
    weights = (gw.cuda(), ff) if act == "weighted" else None
    kernels = ["auto"] + (["tcgen05"] if M <= 16 or M > 128 else [])
    z = a.double() @ w.double().T
    want = z.clone()
    body = z[:, N0:]
    want[:, N0:] = pg.gelu(body) if act == "gelu" else torch.relu(body) ** 2
    if act == "weighted":
        want[:, N0:] *= gw.double().repeat_interleave(ff, 1)[:, :F]
    for kernel in kernels:
        out.fill_(3.0)
        ops_tc.gemm(out, a.cuda(), w.cuda(), kernel=kernel, act="gelu" if act == "gelu" else "relu2", act_from=N0,
                    group_weights=weights)
        err = (out.double().cpu() - want).abs()
        assert (err < 6e-3 * want.abs() + 2e-3).all(), (kernel, err.max().item())
    assert (wide[:, N0 + F:] == 7.0).all()
    assert ops_tc.device_error() == 0


# (head sizes, heads, the kernels that serve them)
ATTENTION = [("float32", 20, 20, 4, 2, {}), ("float32", 12, 36, 4, 2, {}), ("bfloat16", 64, 64, 4, 2, {}),
             ("bfloat16", 128, 128, 8, 2, {}), ("bfloat16", 64, 64, 4, 2, {"prompt_kernel": "mma", "decode_kernel": "split"}),
             ("bfloat16", 32, 32, 4, 1, {"decode_warps_cluster": 4}), ("bfloat16", 32, 32, 4, 1, {"decode_kernel": "split", "decode_splits": 3}),
             ("bfloat16", 48, 48, 4, 2, {}), ("bfloat16", 32, 32, 20, 1, {}), ("bfloat16", 10, 10, 2, 1, {}),
             ("bfloat16", 64, 32, 4, 2, {}), ("bfloat16", 32, 128, 4, 2, {}), ("bfloat16", 24, 40, 4, 2, {})]


@pytest.mark.parametrize("chunk", [70, 64, 33])
@pytest.mark.parametrize("dtype,dk,dv,H,G,pins", ATTENTION)
def test_attention_kernels_alone_with_one_key_that_stands_out(dtype, dk, dv, H, G, pins, chunk, pin):
    """Rotation, cache write and attention in chunks on hand-made projections over scattered pages: the first key of the
    query's chunk is made to dominate (the output is that key's value), then the last key of the chunk before (the output
    must not know it), for queries in a prompt, in a second piece and decoded alone; and the whole against the plain
    attention."""
    from oracle_engine_b200.csrc.ops import PAGE
    from oracle_engine_b200.engine.runtime import Runtime
    from oracle_engine_b200.parts import attention_dispatch as ad
    pin(**pins)
    tdt = torch.float32 if dtype == "float32" else torch.bfloat16
    rotd, base, n = 4, 100.0, 200
    cuts = [0, 150, 198, 199, 200]                          # a prompt, a second piece, two decoded tokens
    torch.manual_seed(5)
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 1.0, "mask": {"size": chunk}, "rot": {"dims": rotd, "base": base}}
    rt = Runtime(tdt, torch.device("cuda"), True)
    one_tensor = dk == dv
    pages = torch.tensor([5, 2, 7, 0], dtype=torch.int32)     # the sequence's pages, out of order, among 8
    tables = torch.full((1, 6), -1, dtype=torch.int32)
    tables[0, :4] = pages
    from oracle_engine_b200.parts.positions import Rotary
    rot = Rotary({"head_dim": dk if one_tensor else rotd, "dims": rotd, "theta": base, "max_positions": 256}, "", rt)
    cos, sin = rot.tables()
    order = rot.head_order() if one_tensor else None
    for inside in (True, False, None):
        q, k, v = torch.randn(n, H, dk) * 0.3, torch.randn(n, G, dk) * 0.3, torch.randn(n, G, dv)
        probes = [chunk + 1, 140, 149, 180, 198, 199]
        if inside is not None:
            for a, t in enumerate(probes):                   # a dimension of its own per probe, behind the turned ones
                j = t // chunk * chunk - (0 if inside else 1)
                k[:, :, rotd + a] = 0
                q[t, :, :] = 0
                q[t, :, rotd + a] = 8.0
                k[j, :, rotd + a] = 5.0                      # a score of 40 against about one
        q, k, v = (x.to(tdt).float() for x in (q, k, v))
        hq = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], 1).double()
        eye = torch.eye(hq.shape[1], dtype=torch.float64)
        wd = {"q": eye[:H * dk], "k": eye[H * dk:(H + G) * dk], "v": eye[(H + G) * dk:], "o": torch.eye(H * dv, dtype=torch.float64)}
        want = pg.attention(hq, pg.keys_values(hq, wd, "", m), wd, "", m)
        if order is not None:
            q, k = q[:, :, order], k[:, :, order]
        proj = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], 1).to(tdt).cuda()
        got = torch.zeros(n, H * dv, dtype=tdt, device="cuda")
        kv = torch.zeros(8, 2, G, PAGE, dk, dtype=tdt, device="cuda")
        kc, vc = torch.zeros(8, G, PAGE, dk, dtype=tdt, device="cuda"), torch.zeros(8, G, PAGE, dv, dtype=tdt, device="cuda")
        for lo, hi in zip(cuts[:-1], cuts[1:]):
            T = hi - lo
            ctx = SimpleNamespace(tok_seq=_i32([0] * T), tok_pos=_i32(list(range(lo, hi))), cu_q=_i32([0, T]),
                                  seq_start=_i32([lo]), seq_qlen=_i32([T]), n_seqs=1, n_tokens=T, max_qlen=T,
                                  max_kvlen=hi, all_decode=T == 1, context_class=0)
            rows = torch.zeros(T, proj.shape[1] + 8, dtype=tdt, device="cuda")          # rows of a wider buffer
            rows[:, :proj.shape[1]] = proj[lo:hi]
            rows = rows[:, :proj.shape[1]]
            out = torch.zeros(T, H * dv, dtype=tdt, device="cuda")
            tab = tables.cuda()
            if one_tensor:
                ad.mixer_core(rt, out, rows, cos, sin, SimpleNamespace(kv=kv, tables=tab), ctx, H, G, dk, -chunk, 1.0, True)
            else:
                ad.split_mixer_core(rt, out, rows, cos, sin, rotd, kc, vc, tab, ctx, H, G, dk, dv, -chunk, 1.0, 0.0, True)
            got[lo:hi] = out
        tol = 2e-5 if dtype == "float32" else 3e-2
        err = (got.double().cpu() - want).abs().max().item()
        assert err < tol * max(1.0, want.abs().max().item()), (dtype, dk, dv, inside, err)
        if inside is not None:
            for t in probes:
                j = t // chunk * chunk - (0 if inside else 1)
                for hh in range(H):
                    o = got[t, hh * dv:(hh + 1) * dv].double().cpu()
                    d = (o - v[j, hh // (H // G)].double()).abs().max().item()
                    assert (d < 0.06) == inside, (dtype, dk, dv, inside, t, hh, d)


# ------------------------------------------------------------------------------------------ layers and schedules

@pytest.mark.parametrize("name", ["G1", "G2", "G3"])
def test_every_layer_by_itself_float32(models, name):
    """The stream that leaves each layer of a whole prompt, in float32, against the plain model; then the same prompt's
    last 20 tokens one by one."""
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
    assert len(seen) == len(want)
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
@pytest.mark.parametrize("name", ["G1", "G2", "G3"])
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
def test_far_keys_page_borders_and_chunk_edges_under_a_peaked_softmax(models, tmp_path, dtype):
    """Chunks of 100, 64, 33 and 150 keys (two of them over keys another layer owns), under scores so large that single
    keys decide: prompts that end just before, at and just after page borders and chunk edges, decoded across the next
    ones.  (tests/test_goridra_cpu.py shows that a chunk one position off moves most positions by ten tolerances.)"""
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


def test_finished_chunks_give_their_pages_back(models):
    """While a sequence decodes, the owner's group holds the pages of the largest chunk among its readers' and its own,
    no more; a pool that could not hold the whole sequences serves them."""
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
            sizes = [g.need.window] + [n for _, n in g.need.also]
            first = min(t // n * n for n in sizes) // 64
            held = np.nonzero(g.tables[slot] >= 0)[0].tolist()
            assert held == list(range(first, t // 64 + 1)), (t, g.need)
    eng.free(slot)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_readers_follow_their_owner(models, tmp_path, dtype):
    """The owner's key projection scaled between two models: a reader's output moves with it, as the plain model's."""
    from oracle_engine_b200.weights.safetensors_io import ModelFiles, write_safetensors
    folder, plain = models["G1"]
    other = tmp_path / "other"
    other.mkdir()
    (other / "config.json").write_text((pg.Path(folder) / "config.json").read_text())
    files = ModelFiles(folder)
    tensors = {n: files.read(n).clone() for n in files.names()}
    files.close()
    tensors["l0.mix.k"] = tensors["l0.mix.k"] * -2
    tensors["l0.mix.v"] = tensors["l0.mix.v"] * 0.5
    write_safetensors(other / "model.safetensors", tensors)
    moved = pg.PlainGoridra(other)
    toks = helpers.random_tokens(90, plain.cfg["vocab"], 4)
    apart = (plain.logits(toks) - moved.logits(toks)).pow(2).mean().sqrt() / plain.logits(toks).pow(2).mean().sqrt()
    assert apart.item() > 3 * TOL[dtype]
    for d, p in ((folder, plain), (str(other), moved)):
        eng = _engine(d, dtype)
        got = _run(eng, tmp_path / f"{dtype}{d[-5:]}", helpers.tail_steps([toks], 30), [toks])
        _compare(got, p, [toks], TOL[dtype], f"readers {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_real_sizes(tmp_path, dtype):
    """Heads of 128, of 64, and of 64 keys with 128 values at a width of 1,024, experts of 256, 128 and 100: in bfloat16
    the prompts go through the tensor-core products with the joined input and the tensor-memory attention, decoding
    through the one-launch kernel and the one that splits the keys."""
    folder = gm.write(tmp_path / "m", gm.REAL, 31, std=0.03, router_scale=2.0)
    plain = pg.PlainGoridra(folder)
    lens = [333, 70, 200, 530]
    requests = [helpers.random_tokens(n, 1000, 800 + i) for i, n in enumerate(lens)]
    eng = _engine(folder, dtype, max_tokens=2048)
    if dtype == "bfloat16":
        assert [b.joined.weight is not None for b in eng.model.layers] == [True] * 4
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


@pytest.mark.parametrize("seed", [21, 22, 23, 24, 25, 26, 27, 28])
def test_configurations_drawn_at_random(tmp_path, seed):
    """Any number of layers, sizes that are and are not multiples of 16, optional parts present or absent, readers of any
    earlier owner: whole prompts, a prompt and 34 single tokens, and a ragged batch, in both precisions."""
    raw = gm.random_config(random.Random(seed))
    folder = gm.write(tmp_path / "m", raw, seed, std=0.06, router_scale=3.0)
    plain = pg.PlainGoridra(folder)
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
    another left reads nothing of it."""
    folder, plain = models["G1"]
    lens = [70, 40, 90, 66, 5, 120]
    requests = [helpers.random_tokens(n, plain.cfg["vocab"], 500 + i) for i, n in enumerate(lens)]
    eng = _engine(folder, dtype, max_tokens=256, n_slots=2)
    steps = helpers.batched_steps(requests, [max(1, n - 8) for n in lens], 2)
    got = _run(eng, tmp_path / "t", steps, requests)
    _compare(got, plain, requests, TOL[dtype], f"reuse {dtype}")
    assert eng.cache.slots.n_free == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["G2", "G3"])
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
    folder, plain = models["G1"]
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
    assert [int(t) for t in r.stdout.split()] == pg.generate(plain, prompt, 6)
