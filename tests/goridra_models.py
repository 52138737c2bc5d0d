"""Small Goridra configurations for the tests, and a writer of model folders with weights that make faults show: router
weights are scaled up so that the experts' scores lie well apart, norm biases are of the size of the values they are added
to, and caps on the logits lie inside the logits' spread."""
from pathlib import Path


def attention(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
         "mask": None if chunk is None else {"size": chunk},
         "rot": None if rot is None else {"dims": rot[0], "base": rot[1]}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def config(vocab, width, eps, layers, cap=None):
    c = {"architecture": "Goridra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap is not None:
        c["logit_softcap"] = cap
    return c


# One even head size for keys and values: the one cache tensor.  Two owners of keys; readers of the first with a chunk
# larger than its own, with one smaller, and with none, so that its pages must outlive its own chunks; an eps that shows;
# layers without feed-forward; a reader between them that reads over another owner.
G1 = config(300, 96, 1e-3, [
    layer(attention(4, 2, 32, 32, 0.25, 40, (16, 10000.0)), moe(6, 2, 40, (3, 2))),
    layer(attention(4, 2, 32, 32, 0.3, 72, (16, 10000.0), 0), dense(56)),
    layer(attention(3, 1, 16, 16, 0.2, 7, (16, 77.0))),
    layer(attention(6, 2, 32, 32, 0.2, 9, (16, 10000.0), 0), moe(4, 4, 16, (2, 2))),
    layer(attention(3, 1, 16, 16, 0.35, 64, (16, 77.0), 2), moe(5, 1, 24))], cap=1.5)
# Key and value sizes that differ both ways (two cache tensors), and one odd size for both; a width and sizes that are no
# multiples of 8; no rotation, no mask, no cap, no groups; chunks of one position and of a page.
G2 = config(257, 100, 3e-6, [
    layer(attention(5, 5, 20, 12, 0.22, 64, (10, 1000.0)), dense(60)),
    layer(attention(2, 1, 34, 6, 0.17, 1, (2, 50000.0)), moe(3, 2, 20)),
    layer(attention(5, 5, 20, 12, 0.3, 50, (10, 1000.0), 0), moe(12, 3, 12, (6, 2))),
    layer(attention(2, 2, 7, 7, 0.4, 33)),
    layer(attention(1, 1, 18, 10, 0.3), dense(30))])
# Heads of 64 (the tensor-memory prompt attention in bfloat16), part of each turned; more experts than a warp has lanes and
# more groups than a word has bits; a group of queries wider than the one-launch decode kernel takes.
G3 = config(150, 64, 1e-5, [
    layer(attention(2, 1, 64, 64, 0.125, 70, (24, 50000.0)), moe(80, 3, 8, (40, 5))),
    layer(attention(2, 1, 64, 64, 0.2, 70, (24, 50000.0), 0), dense(64)),
    layer(attention(20, 1, 32, 32, 0.2, 45, (32, 500.0)), moe(33, 2, 8, (11, 3)))], cap=4.0)
# Peaked attention: large scales, so that one key decides a query's output; chunks that end inside a page, at a page's
# edge and beyond two pages; readers with another chunk than the owner's; little else in the layers.
SHARP = config(200, 64, 1e-5, [
    layer(attention(4, 2, 16, 16, 2.5, 100, (8, 10000.0))),
    layer(attention(2, 2, 32, 48, 2.0, 64, (32, 1000.0))),
    layer(attention(2, 2, 32, 48, 2.0, 33, (32, 1000.0), 1)),
    layer(attention(4, 2, 16, 16, 2.0, 150, (8, 10000.0), 0))])
# sizes of real models at a width of 1,024: the tensor-core products (with the joined input), the tensor-memory attention
REAL = config(1000, 1024, 1e-6, [
    layer(attention(8, 2, 128, 128, 0.09, 256, (64, 10000.0)), dense(2048)),
    layer(attention(8, 2, 128, 128, 0.09, 256, (64, 10000.0), 0), moe(8, 2, 256, (4, 2))),
    layer(attention(16, 4, 64, 128, 0.125, 100, (64, 500000.0)), moe(16, 4, 128, (4, 3))),
    layer(attention(16, 4, 64, 64, 0.125, None, (32, 500000.0)), moe(16, 4, 100, (8, 4)))], cap=10.0)

ALL = {"G1": (G1, 3), "G2": (G2, 4), "G3": (G3, 5), "SHARP": (SHARP, 6)}


def random_config(rng):
    """A configuration drawn from `rng` (random.Random): 2 to 6 layers, sizes that are and are not multiples of 16, every
    optional part present or absent, readers of any earlier owner's keys."""
    layers = []
    for i in range(rng.randint(2, 6)):
        kind = rng.choice(["dense", "moe", "moe", None])
        if kind == "dense":
            mlp = dense(rng.choice([64, 96, 200, 333]))
        elif kind == "moe":
            count = rng.choice([1, 2, 4])
            experts = count * rng.choice([2, 3, 5])
            keep = rng.randint(1, count)
            top = rng.randint(1, min(4, keep * (experts // count)))
            mlp = moe(experts, top, rng.choice([32, 64, 96, 50]), rng.choice([None, (count, keep), (count, keep)]))
        else:
            mlp = None
        owners = [j for j, L in enumerate(layers) if L["mixer"].get("kv_from") is None]
        chunk = rng.choice([None, 1, 17, 64, 96, 128, 200])
        if owners and rng.random() < 0.45:
            m = dict(layers[rng.choice(owners)]["mixer"])
            src = next(j for j in owners if layers[j]["mixer"] == m)
            mixer = attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"] * rng.choice([1.0, 1.5]), chunk,
                              None if m["rot"] is None else (m["rot"]["dims"], m["rot"]["base"]), src)
        else:
            heads = rng.choice([2, 4, 6, 8])
            kv = rng.choice([k for k in (1, 2, 4, 8) if heads % k == 0])
            dim = rng.choice([32, 48, 64, 96, 128, 40])
            vdim = dim if rng.random() < 0.6 else rng.choice([32, 48, 64, 24])
            dims = rng.choice([d for d in (0, 8, 16, 24, 32, dim) if d <= dim])
            mixer = attention(heads, kv, dim, vdim, dim ** -0.5, chunk,
                              None if not dims else (dims, rng.choice([10000.0, 50000.0, 500.0])))
        layers.append(layer(mixer, mlp))
    return config(rng.choice([256, 512, 1000]), rng.choice([128, 192, 256, 320, 200]), rng.choice([1e-5, 1e-6]), layers,
                  cap=rng.choice([None, 2.0, 30.0]))


def write(folder, raw, seed, std=0.1, router_scale=6.0, moe_out=0.25):
    """A model folder of seeded random weights, adjusted as the top of this file says.  moe_out scales the experts'
    down projections: in bfloat16 a router now and then chooses another expert than exact arithmetic does (two scores
    a rounding apart); with a quarter of the output the other choice still shows at its own position, which a
    comparison in bfloat16 leaves out, and hardly at the later ones."""
    from oracle_engine_b200.config.goridra import GoridraConfig
    from oracle_engine_b200.weights.random_init import write_model_folder
    from oracle_engine_b200.weights.safetensors_io import ModelFiles, write_safetensors
    folder = Path(folder)
    write_model_folder(folder, GoridraConfig.from_dict(raw), seed=seed, std=std)
    files = ModelFiles(folder)
    tensors = {}
    for n in files.names():
        t = files.read(n).clone()
        f = t.float()
        if n.endswith(".router"):
            f = f * router_scale                  # scores well apart: few choices hang on a rounding
        elif ".mlp.e" in n and n.endswith(".down"):
            f = f * moe_out
        elif n.endswith(".b"):
            f = f * (0.3 / std)                   # a norm's bias: leaving it out shows
        elif n == "embed":
            f = f * (0.3 / std)                   # logits of a few units: a cap on them shows
        tensors[n] = f.to(t.dtype)
    files.close()
    write_safetensors(folder / "model.safetensors", tensors)
    return str(folder)
