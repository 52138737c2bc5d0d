"""The Mavinex design without a GPU: its config.json reader, its model description, the rotary tables, random model folders
and the plain model's own mechanisms, each against a closed form; and how far mistakes planted in the plain model move it."""
import copy
import json
import math
import random

import numpy as np
import pytest
import torch

import helpers
import mavinex_models as mm
import plain_mavinex as pm


def _model(raw, max_positions=512):
    from oracle_engine_b200.config.mavinex import MavinexConfig
    from oracle_engine_b200.engine.runtime import Runtime
    from oracle_engine_b200.models.mavinex import build_spec
    from oracle_engine_b200.parts.model import DecoderModel
    return DecoderModel(build_spec(MavinexConfig.from_dict(raw), max_positions), Runtime(torch.float32, torch.device("cpu")))


def test_config_round_trip_and_refusals():
    from oracle_engine_b200.config.base import ConfigError
    from oracle_engine_b200.config.mavinex import MavinexConfig
    raws = [raw for raw, _ in mm.ALL.values()] + [mm.REAL] + [mm.random_config(random.Random(s)) for s in range(20)]
    for raw in raws:
        cfg = MavinexConfig.from_dict(raw)
        assert MavinexConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
        assert cfg.vocab == raw["vocab"] and cfg.width == raw["width"] and cfg.norm_eps == raw["norm"]["eps"]
        assert cfg.postln_alpha == raw["postln_alpha"] and cfg.embedding_scale == raw["embedding"]["scale"]
        assert [cfg.owner(i) for i in range(len(cfg.layers))] == [pm.owner(raw, i) for i in range(len(raw["layers"]))]
    noted = dict(copy.deepcopy(mm.M1), seed=3, name="a note")          # a file's own notes at the top level are not read
    assert MavinexConfig.from_dict(noted) == MavinexConfig.from_dict(mm.M1)
    bare = copy.deepcopy(mm.M2)                                        # absent and null mean the same
    for L in bare["layers"]:
        for part in (L["mixer"], L["mixer"].get("left", {})):
            for key in ("mask", "rot"):
                if key in part and part[key] is None:
                    del part[key]
        if L["mlp"] is None:
            del L["mlp"]
    del bare["embedding"]
    bare["layers"][0]["weights_of"] = None
    del bare["layers"][4]["mixer"]["rot_dim"]
    bare["layers"][4]["mixer"]["rot"] = {"dims": 0, "base": 10.0}      # nothing is turned
    assert MavinexConfig.from_dict(bare) == MavinexConfig.from_dict(mm.M2)

    def refused(match, change):
        bad = copy.deepcopy(mm.M1)
        change(bad)
        with pytest.raises(ConfigError, match=match):
            MavinexConfig.from_dict(bad)

    L = lambda c, i: c["layers"][i]                                     # noqa: E731
    refused("layers", lambda c: c.pop("layers"))
    refused("vocab", lambda c: c.pop("vocab"))
    refused("postln_alpha", lambda c: c.pop("postln_alpha"))
    refused("norm", lambda c: c["norm"].update(groups=2))
    refused("embedding", lambda c: c["embedding"].update(bigram={}))
    refused("type", lambda c: L(c, 3).update(type="gla"))
    refused("keys this design", lambda c: L(c, 3)["mixer"]["left"].update(sink=True))
    refused("keys this design", lambda c: L(c, 3)["mixer"]["right"].update(heads=2))
    refused("keys this design", lambda c: L(c, 3)["mixer"].update(middle={}))
    refused("keys this design", lambda c: L(c, 1)["mixer"].update(q_rank=4))
    refused("keys this design", lambda c: L(c, 0)["mlp"]["router"].update(groups=None))
    refused("keys this design", lambda c: L(c, 1)["mixer"]["rot"]["scaling"].update(low=1.0))
    refused("keys this design", lambda c: L(c, 0)["mixer"]["left"]["rot"]["scaling"].update(fast=1.0))
    refused("kv_heads", lambda c: L(c, 3)["mixer"]["left"].update(kv_heads=3))
    refused("inner", lambda c: L(c, 3)["mixer"]["right"].pop("inner"))
    refused("size", lambda c: L(c, 3)["mixer"]["left"]["mask"].update(size=0))
    refused("even", lambda c: L(c, 1)["mixer"]["rot"].update(dims=18))
    refused("above 1", lambda c: L(c, 1)["mixer"]["rot"].update(base=1.0))
    refused("kind", lambda c: L(c, 0)["mlp"].update(kind="dense"))
    refused("exceeds", lambda c: L(c, 0)["mlp"]["router"].update(top=7))
    refused("weights_of", lambda c: L(c, 2).update(weights_of=7))
    refused("leads back", lambda c: L(c, 3).update(weights_of=6))
    refused("differs from layer 0", lambda c: c["layers"].append(mm.shares(mm.parallel(
        4, 2, 32, 48, 0.5, 40, L(c, 0)["mixer"]["left"]["rot"], 64, 8, 8, 4, L(c, 0)["mlp"]), 0)))
    refused("differs from layer 1", lambda c: c["layers"].append(mm.shares(L(c, 0), 1)))


def test_model_description():
    from oracle_engine_b200.parts.spec import CacheNeed, StateNeed
    m = _model(mm.M1)
    names = {d.name: d.shape for d in m.tensors()}
    assert names["l0.mix.left.q"] == (128, 96) and names["l0.mix.left.q.norm"] == (128,) and names["l0.mix.left.g"] == (192, 96)
    assert names["l0.mix.right.in"] == (128, 96) and names["l0.mix.right.x"] == (24, 64) and names["l0.mix.right.conv"] == (64, 4)
    assert names["l1.mix.q"] == (192, 96) and names["l1.mix.dkv"] == (80, 96) and names["l1.mix.g"] == (4, 96)
    assert names["l1.mix.sink"] == (4,) and names["l0.mlp.router.b"] == (6,) and names["head"] == (300, 96)
    assert not any(n.startswith(("l2.", "l4.", "l5.", "l6.", "l3.mlp", "l3.norm2")) for n in names)
    # a layer on another's weights is one more entry of the schedule, with a cache and a state of its own
    assert [e.layer for e in m.schedule] == [0, 1, 0, 2, 1, 0, 2] and len(m.layers) == 3
    kv, lat = CacheNeed("window", (("k", (2, 32)), ("v", (2, 48))), 40), CacheNeed("window", (("latent", (80,)),), 24)
    small = CacheNeed("window", (("k", (2, 16)), ("v", (2, 16))), 70)
    assert m.cache_needs() == [kv, lat, kv, small, lat, kv, small]
    states = m.state_needs()
    assert states[0] == states[2] == {"right.S": StateNeed((64, 8), torch.float32), "right.conv": StateNeed((3, 64), torch.float32)}
    assert states[1] == {} and states[3]["right.conv"].shape == (2, 48)
    assert m.stages() == [(True, 0, 9)]
    assert [n.kind for n in _model(mm.M2).cache_needs()] == ["window", "window", "full", "full", "window"]
    # roofline figures: a query sees its window, the state is read and written
    left, right = (b[1] for b in m.layers[0].mixer.branches)
    assert left.cache_bytes_per_query(39) == 39 * 2 * 80 * 4 and left.cache_bytes_per_query(500) == 40 * 2 * 80 * 4
    assert right.cache_bytes_per_query(7) == 2 * 4 * 64 * (8 + 3)
    assert m.layers[1].mixer.cache_bytes_per_query(100) == 24 * 80 * 4


@pytest.mark.parametrize("rot", [mm.rot(16, 10000.0), mm.rot(40, 300000.0, mm.wave(6.0, 1.0, 5.0, 700)),
                                 mm.rot(10, 1000.0, mm.wave(2.0, 1.0, 2.0, 40)), mm.rot(24, 20000.0, mm.yarn(6.0, 2000, 24.0, 2.0)),
                                 mm.rot(6, 50000.0, mm.yarn(40.0, 4096, 32.0, 1.0)), mm.rot(64, 10.0, mm.yarn(3.0, 9, 1.0, 1.0))])
def test_rotary_tables_are_the_plain_models(rot):
    """Frequencies, both rescalings and the magnitude; a pair at position 0 is the magnitude and nothing else."""
    raw = mm.config(10, 64, 1e-5, 1.0, 1.0, [mm.latent(1, 8, rot["dims"], 8, 8, 1.0, None, rot)
                                              if rot["scaling"] and "fast" in rot["scaling"] else
                                              mm.parallel(1, 1, rot["dims"], 8, 1.0, None, rot, 8, 1, 1, 1)])
    (table,) = _model(raw, 300).positions.values()
    cos, sin = table.tables()
    f, mag = pm.frequencies(rot["dims"], rot["base"], rot["scaling"])
    ang = torch.arange(300, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    assert cos.shape == (300, rot["dims"] // 2)
    assert (cos - mag * torch.cos(ang)).abs().max() < 2e-7 and (sin - mag * torch.sin(ang)).abs().max() < 2e-7
    assert torch.allclose(cos[0], torch.full_like(cos[0], mag))


def test_frequencies_in_closed_form():
    # by wavelength: above high turns in `original` positions kept, below low divided, in between a mixture
    f, m = pm.frequencies(8, 10000.0, mm.wave(8.0, 1.0, 4.0, 628.3185307179587))
    turns = [100.0, 10.0, 1.0, 0.1]                       # 100 positions per unit of angle
    assert m == 1.0 and f[:2] == [1.0, 0.1] and abs(f[2] - 0.01 / 8) < 1e-15 and abs(f[3] - 0.001 / 8) < 1e-16, turns
    f, _ = pm.frequencies(8, 10000.0, mm.wave(8.0, 1.0, 4.0, 2 * 628.3185307179587))
    s = (2.0 - 1.0) / 3.0
    assert abs(f[2] - ((1 - s) * 0.01 / 8 + s * 0.01)) < 1e-15
    # YaRN: ramp from 0 (kept) at the pair with `fast` turns to 1 (divided) at the one with `slow`; with base 10000 and 8
    # dimensions the pair with t turns in 2 pi 100 positions is 2 - log10(t)
    f, m = pm.frequencies(8, 10000.0, mm.yarn(4.0, 2 * math.pi * 100, 100.0, 0.1))
    plain = [1.0, 0.1, 0.01, 0.001]
    assert abs(m - (0.1 * math.log(4.0) + 1)) < 1e-15
    assert all(abs(f[i] - (plain[i] / 4 * i / 3 + plain[i] * (1 - i / 3))) < 1e-15 for i in range(4))
    # floor and ceiling, and a ramp that starts below 0
    f, _ = pm.frequencies(8, 10000.0, mm.yarn(4.0, 2 * math.pi * 100, 3000.0, 3.0))
    assert all(abs(f[i] - plain[i] * (1 - 0.75 * min(i / 2, 1))) < 1e-15 for i in range(4))
    # both ends on one pair: a step
    f, _ = pm.frequencies(8, 10000.0, mm.yarn(4.0, 2 * math.pi * 100, 10.0, 10.0))
    assert all(abs(f[i] - plain[i] * (1.0 if i <= 1 else 0.25)) < 1e-15 for i in range(4))


def test_plain_mechanisms_in_closed_form():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)        # noqa: E731
    # the turn: halves and interleaved pairs as complex products
    x, pos = r(5, 2, 10), torch.tensor([0, 1, 7, 100, 3])
    rt = mm.rot(6, 100.0, mm.yarn(2.0, 50, 4.0, 1.0))
    f, m = pm.frequencies(6, 100.0, rt["scaling"])
    ph = m * torch.exp(1j * pos[:, None, None] * torch.tensor(f, dtype=torch.float64))
    z = torch.complex(x[..., :3], x[..., 3:6]) * ph
    y = pm.turn(x, pos, rt, True)
    assert torch.allclose(y[..., :3], z.real) and torch.allclose(y[..., 3:6], z.imag) and torch.equal(y[..., 6:], x[..., 6:])
    z = torch.complex(x[..., 0:6:2], x[..., 1:6:2]) * ph
    y = pm.turn(x, pos, rt, False)
    assert torch.allclose(y[..., 0:6:2], z.real) and torch.allclose(y[..., 1:6:2], z.imag) and torch.equal(y[..., 6:], x[..., 6:])
    # a window of n: itself and the n - 1 before it
    assert pm.visible(6, 3).sum(1).tolist() == [1, 2, 3, 3, 3, 3] and pm.visible(6, None).sum().item() == 21
    # a sink takes its share and gives nothing
    s = torch.tensor([[0.0, 1.0], [50.0, 0.0]], dtype=torch.float64)
    p = pm.softmax_with_sink(s, torch.tensor(2.0, dtype=torch.float64))
    d = 1 + math.e + math.e ** 2
    assert torch.allclose(p[0], torch.tensor([1 / d, math.e / d], dtype=torch.float64)) and abs(p[1, 0].item() - 1) < 1e-15
    assert pm.softmax_with_sink(s, torch.tensor(400.0, dtype=torch.float64)).sum().item() < 1e-100
    # the recurrence unrolled: S after t tokens is the sum of the inputs, each times the decays behind it
    T, C, N = 6, 3, 2
    u, dt, A, b, c = r(T, C), r(T, C).abs(), -r(C, N).abs(), r(T, N), r(T, N)
    got = pm.scan(u, dt, A, b, c)
    for t in range(T):
        want = torch.zeros(C, dtype=torch.float64)
        for j in range(t + 1):
            want += (torch.exp(A * dt[j + 1:t + 1].sum(0)[:, None]) * (dt[j] * u[j])[:, None] * b[j] * c[t]).sum(1)
        assert torch.allclose(got[t], want)
    # the convolution: the last tap is the current token's, zeros before the start
    k, bias = r(C, 3), r(C)
    y = pm.causal_conv(u, k, bias)
    assert torch.allclose(y[0], u[0] * k[:, 2] + bias) and torch.allclose(y[4], u[2] * k[:, 0] + u[3] * k[:, 1] + u[4] * k[:, 2] + bias)
    # the choice and its weights
    wt, gap = pm.route(torch.tensor([[1.0, 3.0, 2.0, -1.0]], dtype=torch.float64), 2)
    assert torch.allclose(wt[0], torch.tensor([0, math.e / (1 + math.e), 1 / (1 + math.e), 0], dtype=torch.float64)) and gap.item() == 1.0
    # a norm whose weight is kept around zero, of a sum: alpha scales the stream alone
    cfg = mm.config(4, 2, 0.5, 3.0, 2.0, [mm.latent(1, 1, 0, 1, 1, 1.0, None, None)])
    w = {"embed": torch.tensor([[1.0, 0.5]] * 4), "head": torch.eye(4)[:, :2], "final.norm": torch.zeros(2), "l0.norm1": torch.tensor([0.0, 1.0]),
         "l0.mix.q": torch.zeros(1, 2), "l0.mix.dkv": torch.zeros(1, 2), "l0.mix.dkv.norm": torch.ones(1), "l0.mix.uk": torch.zeros(1, 1),
         "l0.mix.uv": torch.zeros(1, 1), "l0.mix.g": torch.zeros(1, 2), "l0.mix.o": torch.zeros(2, 1), "l0.mix.sink": torch.zeros(1)}
    _, kept = pm.forward(cfg, {n: t.double() for n, t in w.items()}, [1], keep_layers=True)
    want = torch.tensor([6.0, 3.0], dtype=torch.float64) / math.sqrt(22.5 + 0.5) * torch.tensor([1.0, 2.0], dtype=torch.float64)
    assert torch.allclose(kept[0, 0], want)


def _moved(folder, tokens, monkeypatch, name, fake, cfg_change=None):
    """Per position: how far the logits of the plain model move under a planted mistake, relative to their size."""
    plain = pm.PlainMavinex(folder)
    want = plain.logits(tokens).numpy()
    with monkeypatch.context() as mp:
        if name:
            mp.setattr(pm, name, fake)
        if cfg_change:
            cfg_change(plain.cfg)
        got = plain.logits(tokens).numpy()
    return np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean())


def test_mistakes_show(tmp_path, monkeypatch):
    """Mistakes planted in the plain model move positions by many tolerances of the GPU comparisons (float32: 1e-4; peaked
    models in bfloat16: 0.1): what those compare can tell the design from its neighbours."""
    sharp = mm.write(tmp_path / "sharp", mm.SHARP, 6)
    toks = helpers.random_tokens(330, 200, 77)
    for d in (-1, 1):                                     # a window one position off, either way
        def off(c, d=d):
            for L in c["layers"]:
                m = L["mixer"].get("left", L["mixer"])
                m["mask"]["size"] += d
        err = _moved(sharp, toks, monkeypatch, None, None, off)
        assert (err[152:] > 1e-3).mean() > 0.9 and (err[152:] > 0.1).mean() > 0.2, d
        assert err[:30].max() < 1e-12
    m1 = mm.write(tmp_path / "m1", mm.M1, 3)
    toks = helpers.random_tokens(150, 300, 5)
    err = _moved(m1, toks, monkeypatch, "softmax_with_sink", lambda s, sink=None: torch.softmax(s, -1))
    assert (err > 1e-3).mean() > 0.9
    scan = pm.scan

    def lost(u, dt, A, b, c):                             # the state is lost at token 64
        return torch.cat([scan(u[:64], dt[:64], A, b[:64], c[:64]), scan(u[64:], dt[64:], A, b[64:], c[64:])])
    err = _moved(m1, toks, monkeypatch, "scan", lost)
    assert err[:64].max() < 1e-12 and (err[64:80] > 0.02).all() and (err[64:] > 1e-3).mean() > 0.6
    conv, route = pm.causal_conv, pm.route

    def cut(x, k, b):                                     # the convolution's inputs are lost at token 64
        return torch.cat([conv(x[:64], k, b), conv(x[64:], k, b)])
    err = _moved(m1, toks, monkeypatch, "causal_conv", cut)
    assert err[:64].max() < 1e-12 and err[64:67].min() > 0.02
    err = _moved(m1, toks, monkeypatch, "route", lambda z, top: route(z - z.new_tensor([0.5] + [0.0] * (z.shape[1] - 1)), top))
    assert (err > 1e-3).mean() > 0.5
    err = _moved(m1, toks, monkeypatch, None, None, lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=8.5))
    assert (err[5:] > 3e-4).mean() > 0.9


def test_random_model_folder_loads(tmp_path):
    from oracle_engine_b200.config.base import load_config
    from oracle_engine_b200.weights.loader import check_tensors
    from oracle_engine_b200.weights.safetensors_io import ModelFiles, WeightError
    for name, (raw, seed) in mm.ALL.items():
        folder = mm.write(tmp_path / name, raw, seed)
        cfg, arch = load_config(folder)
        assert arch.name == "Mavinex"
        files = ModelFiles(folder)
        model = _model(raw)
        have = {n: (files.info(n).dtype, tuple(files.info(n).shape)) for n in files.names()}
        check_tensors(have, model.tensors(), model.spec.ignored_tensors)
        short = {n: i for n, i in have.items() if n != "l0.mix.right.A_log"}
        with pytest.raises(WeightError, match="A_log"):
            check_tensors(short, model.tensors(), model.spec.ignored_tensors)
        files.close()
        logits = pm.PlainMavinex(folder).logits(helpers.random_tokens(20, raw["vocab"], 1))
        assert torch.isfinite(logits).all() and logits.std() > 0.05
