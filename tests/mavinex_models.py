"""Small Mavinex configurations for the tests, and a writer of model folders with weights that make faults show: router
logits lie well apart and their bias is of their size, sinks are of the size of the scores, the convolution's taps and the
step sizes make the scan's state remember dozens of tokens."""
from pathlib import Path


def rot(dims, base, scaling=None):
    return {"dims": dims, "base": base, "scaling": scaling}


def wave(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def parallel(heads, kv_heads, dim, vdim, scale, window, turn, inner, state, dt_rank, conv, mlp=None):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                               "mask": None if window is None else {"size": window}, "rot": turn},
                      "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window, turn, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "mask": None if window is None else {"size": window}, "rot": turn}}


def shares(layer, j):
    return dict(layer, weights_of=j)


def config(vocab, width, eps, alpha, emb, layers):
    return {"architecture": "Mavinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": emb}, "layers": layers}


# Sizes that the tensor-core kernels take; both kinds of layer, each with a second layer on its weights (one of them on a
# layer that already borrows), layers without a feed-forward, an eps that shows.
_A = parallel(4, 2, 32, 48, 0.25, 40, rot(16, 10000.0, wave(4.0, 1.0, 4.0, 64)), 64, 8, 8, 4, moe(6, 2, 40))
_B = latent(4, 32, 16, 32, 64, 0.2, 24, rot(16, 500.0, yarn(8.0, 64, 8.0, 1.0)), moe(5, 2, 24))
_C = parallel(2, 2, 16, 16, 0.3, 70, rot(16, 77.0), 48, 16, 5, 3)
M1 = config(300, 96, 1e-3, 1.7, 9.0, [_A, _B, shares(_A, 0), _C, shares(_B, 1), shares(_A, 2), shares(_C, 3)])
# No multiples of 8 anywhere; values longer and shorter than keys; one state, one rank, one tap, one channel tile; windows
# of one position and of a page, none at all; no rotation; a base whose scaling ramp lies between two dimensions.
M2 = config(257, 100, 3e-6, 0.6, 1.0, [
    parallel(5, 5, 20, 12, 0.22, 64, rot(10, 1000.0, wave(2.0, 1.0, 2.0, 40)), 50, 1, 1, 1, moe(3, 3, 20)),
    latent(3, 10, 6, 7, 20, 0.3, 1, rot(6, 50000.0, yarn(40.0, 4096, 32.0, 1.0))),
    parallel(3, 1, 7, 9, 0.4, None, None, 37, 5, 3, 7, moe(12, 1, 12)),
    latent(1, 9, 4, 30, 33, 0.4, None, rot(2, 100.0), moe(4, 2, 10)),
    latent(2, 8, 0, 8, 16, 0.3, 33, None)])
# More experts than a warp has lanes, a group of queries wider than the kernels' usual, many states per channel, a rank of
# its inner size, a latent longer than the tensor-core kernel takes.
M3 = config(150, 64, 1e-5, 2.5, 8.0, [
    parallel(20, 1, 32, 32, 0.2, 45, rot(32, 500.0), 32, 200, 32, 2, moe(80, 3, 8)),
    latent(20, 16, 32, 16, 272, 0.15, 50, rot(32, 10000.0, yarn(4.0, 256, 16.0, 2.0)), moe(33, 2, 8)),
    parallel(2, 1, 64, 64, 0.125, 150, rot(48, 50000.0), 256, 64, 24, 5)])
# Peaked attention: large scales, so that one key decides a query's output; windows that end inside a page, at a page's edge
# and beyond two pages; little else in the layers.
SHARP = config(200, 64, 1e-5, 1.0, 4.0, [
    parallel(4, 2, 16, 16, 2.5, 100, rot(8, 10000.0), 16, 4, 4, 4),
    latent(2, 16, 16, 32, 32, 4.0, 64, rot(16, 1000.0, yarn(2.0, 128, 8.0, 1.0))),
    latent(4, 16, 16, 16, 32, 4.0, 33, rot(16, 1000.0)),
    parallel(2, 2, 32, 48, 2.0, 150, rot(32, 1000.0), 16, 4, 4, 4)])
# sizes of real models at a width of 1,024
_RP = parallel(8, 2, 128, 128, 0.09, 256, rot(128, 10000.0, wave(8.0, 1.0, 4.0, 1024)), 2048, 16, 64, 4, moe(8, 2, 256))
_RL = latent(8, 128, 64, 128, 192, 0.072, 200, rot(64, 10000.0, yarn(8.0, 512, 32.0, 1.0)), moe(16, 4, 128))
REAL = config(1000, 1024, 1e-6, 2.0, 32.0, [_RP, _RL, shares(_RP, 0)])

ALL = {"M1": (M1, 3), "M2": (M2, 4), "M3": (M3, 5), "SHARP": (SHARP, 6)}


def random_config(rng):
    """A configuration drawn from `rng` (random.Random): 2 to 6 layers, sizes that are and are not multiples of 16, every
    optional part present or absent, layers on any earlier layer's weights."""
    layers = []
    for i in range(rng.randint(2, 6)):
        if layers and rng.random() < 0.3:
            j = rng.randrange(len(layers))
            layers.append(shares({k: v for k, v in layers[j].items() if k != "weights_of"}, j))
            continue
        experts = rng.choice([1, 3, 5, 8, 12])
        mlp = None if rng.random() < 0.25 else moe(experts, rng.randint(1, min(4, experts)), rng.choice([32, 64, 50, 72]))
        window = rng.choice([None, 1, 17, 64, 96, 140, 200])
        base = rng.choice([10000.0, 300000.0, 500.0])
        if rng.random() < 0.5:
            heads = rng.choice([2, 4, 6, 8])
            kv = rng.choice([k for k in (1, 2, 4, 8) if heads % k == 0])
            dim, vdim = rng.choice([32, 48, 64, 96, 40, 128]), rng.choice([32, 48, 96, 64, 24])
            dims = rng.choice([d for d in (0, 8, 16, 24, 32, dim) if d <= dim])
            scaling = rng.choice([None, wave(rng.choice([2.0, 8.0]), 1.0, rng.choice([2.0, 4.0]), rng.choice([64, 700]))])
            layers.append(parallel(heads, kv, dim, vdim, dim ** -0.5, window, rot(dims, base, scaling) if dims else None,
                                   rng.choice([64, 128, 100, 256]), rng.choice([4, 8, 16, 32, 10]), rng.choice([3, 8, 12, 16]),
                                   rng.choice([2, 3, 4, 6]), mlp))
        else:
            rd = rng.choice([0, 8, 16, 32, 32])
            scaling = rng.choice([None, yarn(rng.choice([2.0, 8.0]), rng.choice([128, 2000]), 32.0, 1.0)])
            dim = rng.choice([16, 32, 64, 40])
            layers.append(latent(rng.choice([1, 2, 4, 5]), dim, rd, rng.choice([16, 32, 64, 24]), rng.choice([32, 64, 128, 50]),
                                 (dim + rd) ** -0.5, window, rot(rd, base, scaling) if rd else None, mlp))
    return config(rng.choice([256, 500, 1000]), rng.choice([128, 192, 256, 320, 200]), rng.choice([1e-5, 1e-6]),
                  rng.choice([0.8, 1.0, 2.5]), rng.choice([1.0, 12.0]), layers)


def write(folder, raw, seed, std=0.1, router_scale=6.0, moe_out=0.25):
    """A model folder of seeded random weights, adjusted as the top of this file says.  moe_out scales the experts' down
    projections: in bfloat16 a router now and then chooses another expert than exact arithmetic does (two logits a rounding
    apart); with a part of the output the other choice still shows at its own position, which a comparison in bfloat16
    leaves out, and hardly at the later ones."""
    from oracle_engine_b200.config.mavinex import MavinexConfig
    from oracle_engine_b200.weights.random_init import write_model_folder
    from oracle_engine_b200.weights.safetensors_io import ModelFiles, write_safetensors
    folder = Path(folder)
    write_model_folder(folder, MavinexConfig.from_dict(raw), seed=seed, std=std)
    files = ModelFiles(folder)
    tensors = {}
    for n in files.names():
        t = files.read(n).clone()
        f = t.float()
        unit = f / std                            # standard normal values
        if n.endswith(".router"):
            f = f * router_scale * min(1.0, 10.0 / raw["width"] ** 0.5)
        elif n.endswith(".router.b") or n.endswith(".sink") or n.endswith(".conv.b"):
            f = unit
        elif ".mlp.e" in n and n.endswith(".down"):
            f = f * moe_out
        elif n.endswith(".conv"):
            f = unit * 0.5
        elif n.endswith(".dt.b"):
            f = unit * 0.7 - 2.5                  # step sizes of 0.02 to 0.3
        elif n.endswith(".A_log"):
            f = unit * 0.7 - 0.7                  # decays of 0.9 to 0.999 a token
        tensors[n] = f.to(t.dtype)
    files.close()
    write_safetensors(folder / "model.safetensors", tensors)
    return str(folder)
