"""The Goridra design without a GPU: its config.json reader, its model description, the cache of chunks, random model
folders and the plain model's own mechanisms, each against a closed form."""
import copy
import json
import math
import random

import pytest
import torch

import goridra_models as gm
import plain_goridra as pg


def _model(raw, max_positions=512):
    from oracle_engine_b200.config.goridra import GoridraConfig
    from oracle_engine_b200.engine.runtime import Runtime
    from oracle_engine_b200.models.goridra import build_spec
    from oracle_engine_b200.parts.model import DecoderModel
    return DecoderModel(build_spec(GoridraConfig.from_dict(raw), max_positions), Runtime(torch.float32, torch.device("cpu")))


def test_config_round_trip_and_refusals():
    from oracle_engine_b200.config.base import ConfigError
    from oracle_engine_b200.config.goridra import GoridraConfig
    raws = [raw for raw, _ in gm.ALL.values()] + [gm.REAL] + [gm.random_config(random.Random(s)) for s in range(20)]
    for raw in raws:
        cfg = GoridraConfig.from_dict(raw)
        assert GoridraConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
        assert cfg.vocab == raw["vocab"] and cfg.width == raw["width"] and cfg.norm_eps == raw["norm"]["eps"]
        assert cfg.logit_softcap == raw.get("logit_softcap")
    noted = dict(copy.deepcopy(gm.G1), seed=3, name="a note")          # a file's own notes at the top level are not read
    assert GoridraConfig.from_dict(noted) == GoridraConfig.from_dict(gm.G1)
    bare = copy.deepcopy(gm.G2)                                        # absent and null mean the same
    for L in bare["layers"]:
        for key in ("mask", "rot"):
            if L["mixer"][key] is None:
                del L["mixer"][key]
        if L["mlp"] is None:
            del L["mlp"]
    bare["logit_softcap"] = None
    bare["layers"][4]["mixer"]["kv_from"] = None
    bare["layers"][1]["mlp"]["router"]["groups"] = None
    bare["layers"][4]["mixer"]["rot"] = {"dims": 0, "base": 10.0}      # nothing is turned
    assert GoridraConfig.from_dict(bare) == GoridraConfig.from_dict(gm.G2)

    def refused(match, change):
        bad = copy.deepcopy(gm.G1)
        change(bad)
        with pytest.raises(ConfigError, match=match):
            GoridraConfig.from_dict(bad)

    L = lambda c, i: c["layers"][i]                                     # noqa: E731
    refused("layers", lambda c: c.pop("layers"))
    refused("vocab", lambda c: c.pop("vocab"))
    refused("norm", lambda c: c["norm"].update(groups=2))
    refused("logit_softcap", lambda c: c.update(logit_softcap=-1.0))
    refused("type", lambda c: L(c, 0).update(type="gla"))
    refused("keys this design", lambda c: L(c, 0)["mixer"].update(sink=True))
    refused("keys this design", lambda c: L(c, 0)["mixer"]["mask"].update(kind="window"))
    refused("keys this design", lambda c: L(c, 0)["mixer"]["rot"].update(scaling={}))
    refused("keys this design", lambda c: L(c, 0)["mlp"].update(shared={"ff": 3}))
    refused("keys this design", lambda c: L(c, 0)["mlp"]["router"].update(bias=True))
    refused("multiple of kv_heads", lambda c: L(c, 0)["mixer"].update(kv_heads=3))
    refused("size", lambda c: L(c, 0)["mixer"]["mask"].update(size=0))
    refused("even", lambda c: L(c, 0)["mixer"]["rot"].update(dims=34))
    refused("kind", lambda c: L(c, 1)["mlp"].update(kind="swiglu"))
    refused("equal groups", lambda c: L(c, 0)["mlp"]["router"].update(groups={"count": 4, "keep": 2}))
    refused("equal groups", lambda c: L(c, 0)["mlp"]["router"].update(groups={"count": 3, "keep": 4}))
    refused("exceeds the 2 experts", lambda c: L(c, 0)["mlp"]["router"].update(groups={"count": 3, "keep": 1}, top=3))
    refused("kv_from", lambda c: L(c, 1)["mixer"].update(kv_from=1))    # itself
    refused("kv_from", lambda c: L(c, 3)["mixer"].update(kv_from=1))    # a layer that reads another's
    refused("kv_from", lambda c: L(c, 3)["mixer"].update(kv_from=2))    # other heads
    refused("kv_from", lambda c: L(c, 1)["mixer"]["rot"].update(base=3.0))


def test_model_description():
    from oracle_engine_b200.parts.spec import CacheNeed
    m = _model(gm.G1)
    names = {d.name: d.shape for d in m.tensors()}
    assert "l0.mix.k" in names and "l1.mix.k" not in names and "l3.mix.v" not in names and "l1.mix.q" in names
    assert names["l0.mlp.e5.up"] == (40, 96) and names["l0.mlp.e5.down"] == (96, 40) and names["l0.mlp.router"] == (6, 96)
    assert names["l1.mlp.up"] == (56, 96) and names["final.norm.b"] == (96,) and "head" not in names
    assert not any(n.startswith("l2.mlp") for n in names)
    # the owner keeps what its readers still see: chunks of its own size and of theirs
    assert m.cache_needs() == [CacheNeed("chunk", (("kv", (2, 2, 32)),), 40, (("chunk", 9), ("chunk", 72))), None,
                               CacheNeed("chunk", (("kv", (2, 1, 16)),), 7, (("chunk", 64),)), None, None]
    assert m.stages() == [(True, 0, 7)] and not any(m.state_needs())
    # equal rotations share one table
    assert len(m.positions) == 2
    full = copy.deepcopy(gm.G1)
    full["layers"][1]["mixer"]["mask"] = None
    assert _model(full).cache_needs()[0].kind == "full"
    # sizes of keys and values that differ, or are odd, lie in two tensors
    needs = _model(gm.G2).cache_needs()
    assert [None if n is None else n.tensors for n in needs] == [
        (("k", (5, 20)), ("v", (5, 12))), (("k", (1, 34)), ("v", (1, 6))), None, (("k", (2, 7)), ("v", (2, 7))),
        (("k", (1, 18)), ("v", (1, 10)))]
    assert [n.kind for n in needs if n] == ["chunk", "chunk", "chunk", "full"]
    # roofline figures: a query sees its own chunk up to itself
    mixer = m.layers[0].mixer
    assert mixer.cache_bytes_per_query(40) == 40 * 2 * 2 * 32 * 4 and mixer.cache_bytes_per_query(41) == 2 * 2 * 32 * 4
    # (a layer that projects no keys: its rows are q and o only)
    assert m.layers[1].mixer.flops(0, 1) == 2.0 * 96 * 2 * 4 * 32 + 4.0 * 4 * 32


def test_visible_pairs_counts_the_mask():
    from oracle_engine_b200.parts.spec import mask_span, visible_keys, visible_pairs
    for span in (0, 5, 64, -1, -7, -64):
        for start, count in ((0, 1), (0, 70), (63, 2), (6, 1), (10, 130)):
            seen = 0
            for t in range(start, start + count):
                one = sum(1 for j in range(t + 1) if (span == 0 or (span > 0 and j > t - span) or
                                                      (span < 0 and j // -span == t // -span)))
                assert one == visible_keys(span, t + 1)
                seen += one
            assert visible_pairs(span, start, count) == seen, (span, start, count)
    assert mask_span(None, 9) == -9 and mask_span(4, 0) == 4 and mask_span(None, None) == 0
    with pytest.raises(ValueError):
        mask_span(4, 9)


def test_chunk_group_gives_finished_chunks_back():
    """Under random traffic: every page that a query of a step may read, by the owner's mask or a reader's, is mapped, no
    older one is, and nothing is lost."""
    from oracle_engine_b200.cache.kv_cache import KVCache, pages_for
    from oracle_engine_b200.cache.slots import CacheFull
    from oracle_engine_b200.csrc.ops import PAGE
    from oracle_engine_b200.parts.spec import CacheNeed
    T = (("kv", (2, 1, 16)),)
    plain, joint = CacheNeed("chunk", T, 100), CacheNeed("chunk", T, 100).joined(CacheNeed("chunk", T, 130))
    assert joint == CacheNeed("chunk", T, 100, (("chunk", 130),)) and joint.joined(plain) == joint
    assert plain.joined(CacheNeed("full", T)) == CacheNeed("full", T)
    assert plain.joined(CacheNeed("window", T, 3)).first_position(205) == 200
    assert plain.joined(CacheNeed("window", T, 30)).first_position(205) == 176
    assert [joint.first_position(p) for p in (0, 99, 100, 129, 130, 199, 200, 259, 260)] == \
        [0, 0, 0, 0, 100, 100, 130, 130, 200]
    rng = random.Random(1)
    c = KVCache([plain, joint], max_tokens=2048, max_seq_len=900, allocate=False, window_pool_tokens=1024)
    assert [g.pool.n for g in c.groups] == [16, 16]
    live = {}
    for _ in range(1500):
        r = rng.random()
        if r < 0.3 and c.slots.n_free:
            live[c.alloc_slot()] = 0
        elif r < 0.45 and live:
            s = rng.choice(list(live))
            c.free_slot(s)
            del live[s]
        elif live:
            s = rng.choice(list(live))
            n = live[s] + rng.choice([1, 1, 1, 17, 64, 130])
            try:
                c.reserve(s, n)
            except CacheFull:
                continue
            for g, sizes in zip(c.groups, ((100,), (100, 130))):
                first = min(live[s] // k * k for k in sizes)
                assert (g.tables[s][first // PAGE:pages_for(n)] >= 0).all() and (g.tables[s][:first // PAGE] < 0).all()
            c.commit(s, n)
            live[s] = n
        c.check()
    for s in list(live):
        c.free_slot(s)
    c.check()
    assert all(g.pool.n_free == g.pool.n for g in c.groups)


def test_a_partial_rotation_by_reordered_heads():
    """Rotary.head_order: rotating whole heads by halves in that order scores as turning the first `dims` dimensions."""
    from oracle_engine_b200.engine.runtime import Runtime
    from oracle_engine_b200.parts.positions import Rotary
    rt = Runtime(torch.float32, torch.device("cpu"))
    torch.manual_seed(0)
    for hd, dims in ((16, 8), (64, 24), (10, 2), (12, 0), (32, 32)):
        rot = Rotary({"head_dim": hd, "dims": dims, "theta": 100.0, "max_positions": 20}, "", rt)
        cos, sin = (t.double() for t in rot.tables())
        assert cos.shape == (20, hd // 2) and (cos[:, dims // 2:] == 1).all() and (sin[:, dims // 2:] == 0).all()
        order = rot.head_order()
        assert (order is None) == (dims == hd) and (order is None or sorted(order) == list(range(hd)))
        q, k, pos = torch.randn(20, 1, hd).double(), torch.randn(20, 1, hd).double(), torch.arange(20)
        want = pg.turn_halves(q, pos, dims, 100.0)[:, 0] @ pg.turn_halves(k, pos, dims, 100.0)[:, 0].T

        def whole(x):
            x = x[:, 0, order] if order is not None else x[:, 0]
            a, b = x[:, :hd // 2], x[:, hd // 2:]
            return torch.cat([a * cos - b * sin, b * cos + a * sin], 1)
        assert (whole(q) @ whole(k).T - want).abs().max().item() < 1e-5


def test_random_folder_loads_in_the_plain_model(tmp_path):
    for name, (raw, seed) in gm.ALL.items():
        plain = pg.PlainGoridra(gm.write(tmp_path / name, raw, seed))
        lg = plain.logits([1, 2, 3, 4, 5])
        assert lg.shape == (5, raw["vocab"]) and torch.isfinite(lg).all()
        declared = {d.name: tuple(d.shape) for d in _model(raw).tensors()}
        assert declared == {n: tuple(t.shape) for n, t in plain.w.items()}
        cap = raw.get("logit_softcap")
        if cap:                                                       # the cap bites
            flat = pg.forward({k: v for k, v in plain.cfg.items() if k != "logit_softcap"}, plain.w, [1, 2, 3, 4, 5])
            assert lg.abs().max().item() < cap and (flat - lg).abs().max().item() > 0.05 * cap
            assert (cap * torch.tanh(flat / cap) - lg).abs().max().item() < 1e-12


# ------------------------------------------------------------------ the plain model's mechanisms, in closed forms

def test_plain_layer_norm():
    torch.manual_seed(1)
    x, w, b = torch.randn(3, 10).double() * 4 + 2, torch.randn(10).double(), torch.randn(10).double()
    y = (pg.layer_norm(x, w, b, 0.0) - b) / w
    assert y.mean(-1).abs().max().item() < 1e-12 and ((y * y).mean(-1) - 1).abs().max().item() < 1e-12
    assert torch.equal(pg.layer_norm(torch.full((1, 10), 7.0).double(), w, b, 1e-5)[0], b)          # no deviation: the bias
    small = pg.layer_norm(x * 1e-4, w, b, 1e-3)                        # eps inside the root: it wins over a small variance
    assert (small - ((x - x.mean(-1, keepdim=True)) * 1e-4 / math.sqrt(1e-3) * w + b)).abs().max().item() < 1e-3


def test_plain_gelu():
    z = torch.tensor([0.0, 1.0, -1.0, 8.0, -8.0]).double()
    phi1 = 0.8413447460685429                                         # the normal distribution function at one
    assert torch.allclose(pg.gelu(z), torch.tensor([0.0, phi1, phi1 - 1.0, 8.0, 0.0]).double(), atol=1e-12)


def test_plain_mask_and_attention():
    for size in (1, 3, 4, None):
        seen = pg.visible(9, size)
        for i in range(9):
            first = 0 if size is None else i - i % size
            assert seen[i].tolist() == [first <= j <= i for j in range(9)]
    # equal scores: the mean of the values of the own chunk up to the query
    T, D = 10, 6
    torch.manual_seed(2)
    h = torch.randn(T, D).double()
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 1.0, "mask": {"size": 4}, "rot": {"dims": 2, "base": 10.0}}
    w = {"q": torch.zeros(8, D).double(), "k": torch.randn(4, D).double(), "v": torch.randn(3, D).double(),
         "o": torch.eye(6).double()}
    kv = pg.keys_values(h, w, "", m)
    out = pg.attention(h, kv, w, "", m)
    for t in range(T):
        want = kv[1][t - t % 4:t + 1, 0].mean(0)
        assert torch.allclose(out[t], torch.cat([want, want]), atol=1e-12)
    # a reader with another mask, over the same keys and values
    out = pg.attention(h, kv, w, "", dict(m, mask={"size": 3}))
    assert torch.allclose(out[5, :3], kv[1][3:6, 0].mean(0), atol=1e-12)
    # turned queries and keys score by the distance alone; the dimensions behind `dims` do not turn
    q = torch.randn(1, 1, 4).double().expand(T, 1, 4)
    turned = pg.turn_halves(q, torch.arange(T), 2, 10.0)
    dots = turned[:, 0] @ turned[:, 0].T
    assert torch.allclose(dots[3, 1], dots[8, 6]) and torch.equal(turned[..., 2:], q[..., 2:])
    assert not torch.allclose(dots[3, 1], dots[3, 2])


def test_plain_routing():
    z = torch.log(torch.tensor([[0.30, 0.015, 0.16, 0.15, 0.02, 0.29, 0.03, 0.04]], dtype=torch.float64))
    w, gap = pg.route(z, {"experts": 8, "top": 2})
    assert torch.allclose(w[0, [0, 5]], torch.tensor([0.30, 0.29], dtype=torch.float64) / 0.59) and (w > 0).sum() == 2
    assert abs(gap.item() - math.log(0.29 / 0.16)) < 1e-9
    # pairs: the runs' scores are 0.30, 0.16, 0.29, 0.04; two stay, and 0.16 cannot be chosen although it is third best
    w, gap = pg.route(z, {"experts": 8, "top": 3, "groups": {"count": 4, "keep": 2}})
    assert torch.nonzero(w[0]).flatten().tolist() == [0, 4, 5] and abs(w.sum().item() - 1.0) < 1e-12
    assert abs(gap.item() - math.log(0.02 / 0.015)) < 1e-9              # the closest call is the last expert's
    w, gap = pg.route(z, {"experts": 8, "top": 4, "groups": {"count": 4, "keep": 2}})
    assert torch.nonzero(w[0]).flatten().tolist() == [0, 1, 4, 5]
    assert abs(gap.item() - math.log(0.29 / 0.16)) < 1e-9              # ... here the last run's


def test_plain_experts_and_the_parallel_layer():
    torch.manual_seed(3)
    D = 5
    h = torch.randn(2, D).double()
    w = {"router": torch.zeros(2, D).double(), "e0.up": torch.randn(3, D).double(), "e0.down": torch.randn(D, 3).double(),
         "e1.up": torch.randn(3, D).double(), "e1.down": torch.randn(D, 3).double()}
    w["router"][1] = 50.0 * h[0]                                      # token 0 goes to expert 1 alone
    out = pg.moe(h[:1], w, "", gm.moe(2, 1, 3))
    assert torch.allclose(out[0], w["e1.down"] @ torch.relu(w["e1.up"] @ h[0]) ** 2, atol=1e-12)
    # one layer: both sublayers read the same normed stream, and the stream keeps both outputs
    cfg = gm.config(7, D, 1e-5, [gm.layer(gm.attention(1, 1, 2, 2, 1.0, 3), gm.dense(4))])
    W = {"embed": torch.randn(7, D).double(), "l0.norm1": torch.randn(D).double(), "l0.norm1.b": torch.randn(D).double(),
         "final.norm": torch.ones(D).double(), "final.norm.b": torch.zeros(D).double()}
    for n, s in (("q", (2, D)), ("k", (2, D)), ("v", (2, D)), ("o", (D, 2))):
        W["l0.mix." + n] = torch.randn(s).double()
    W["l0.mlp.up"], W["l0.mlp.down"] = torch.randn(4, D).double(), torch.randn(D, 4).double()
    logits, layers = pg.forward(cfg, W, [4], keep_layers=True)
    x = W["embed"][4]
    n = pg.layer_norm(x, W["l0.norm1"], W["l0.norm1.b"], 1e-5)
    want = x + W["l0.mix.o"] @ (W["l0.mix.v"] @ n) + W["l0.mlp.down"] @ pg.gelu(W["l0.mlp.up"] @ n)
    assert torch.allclose(layers[0, 0], want, atol=1e-12)
    assert torch.allclose(logits[0], W["embed"] @ pg.layer_norm(want, torch.ones(D).double(), torch.zeros(D).double(), 1e-5))


def test_plain_sharp_model_shows_a_chunk_one_off(tmp_path):
    """In the model with peaked scores a chunk edge one position off moves most positions behind the first edge by many
    tolerances (the GPU tests hold the kernels to one)."""
    plain = pg.PlainGoridra(gm.write(tmp_path / "s", gm.SHARP, gm.ALL["SHARP"][1]))
    toks = torch.randint(0, 200, (330,), generator=torch.Generator().manual_seed(77)).tolist()
    a = plain.logits(toks)
    for step in (1, -1):
        off = copy.deepcopy(plain.cfg)
        for L in off["layers"]:
            L["mixer"]["mask"]["size"] += step
        moved = ((a - pg.forward(off, plain.w, toks)).pow(2).mean(-1).sqrt() / a.pow(2).mean().sqrt())[110:]
        assert (moved > 1e-3).float().mean().item() > 0.8, step
