"""A plain, slow Goridra: one function per mechanism, float64 on the CPU.

It shares no code with the package: it reads config.json and the safetensors file by itself
(through torch only) and follows the equations below literally.

Notation.  x_t is the residual stream at token t (width D), p its position in its sequence.
    embedding   x_t = E[tok_t]
    norm        N(x; w, b) = (x - mean x) / sqrt(mean((x - mean x)^2) + eps) * w + b
    layer       h = N_1(x);   x <- x + (M(h) + F(h))                   (F only if the layer has one)

Mixer "attention" (H query heads over G key heads, key size d, value size dv):
    q = Wq h, k = Wk h, v = Wv h; the first `dims` dimensions of every head of q and k turned by the position, i paired
    with i + dims/2, angle p * base^(-2i/dims).  A layer with `kv_from` j has neither Wk nor Wv: it takes the turned
    keys and the values of layer j.
    s_j = scale * q . k_j for j <= t with floor(j / size) = floor(t / size);   p = softmax(s);   M = Wo concat_h sum_j p_j v_j

Feed-forward "dense":  Wdown g(Wup h), g(z) = z * (1 + erf(z / sqrt 2)) / 2
Feed-forward "moe":    s = softmax(Wr h) over all experts; the experts stand in `count` equal runs, a run's score is its
    largest s, the `keep` best runs stay; the `top` largest s among their experts choose; the weights are the chosen s over
    (their sum + 1e-20); expert: Wdown max(Wup h, 0)^2

Logits: z = E N_final(x), then c * tanh(z / c) with the cap c.
"""
import json
import math
import struct
from pathlib import Path

import torch

F64 = torch.float64


def read_safetensors(path):
    raw = Path(path).read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    out = {}
    for name, info in head.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        buf = bytearray(raw[8 + n + lo: 8 + n + hi])
        t = torch.frombuffer(buf, dtype=kinds[info["dtype"]]).reshape(info["shape"])
        out[name] = t.to(F64) if t.is_floating_point() else t.clone()
    return out


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def gelu(z):
    return z * 0.5 * (1.0 + torch.erf(z / math.sqrt(2.0)))


def turn_halves(x, pos, dims, base):
    """x [T, heads, n]; the first `dims` dimensions turned by the position, i paired with i + dims/2; pos [T]."""
    half = dims // 2
    if half == 0:
        return x
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    ang = pos.to(F64)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], -1)


def visible(T, size):
    """[T, T] booleans: query i sees key j; size None: every j up to i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size:
        seen = seen & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))
    return seen


def keys_values(h, w, pre, m):
    """The turned keys [T, G, d] and the values [T, G, dv] of a layer with projections of its own."""
    T = h.shape[0]
    k = (h @ w[pre + "k"].T).view(T, m["kv_heads"], m["dim"])
    v = (h @ w[pre + "v"].T).view(T, m["kv_heads"], m["vdim"])
    rot = m.get("rot")
    return (turn_halves(k, torch.arange(T), rot["dims"], rot["base"]) if rot else k), v


def attention(h, kv, w, pre, m):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k, v = kv
    q = (h @ w[pre + "q"].T).view(T, H, d)
    rot = m.get("rot")
    if rot:
        q = turn_halves(q, torch.arange(T), rot["dims"], rot["base"])
    seen = visible(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        out[:, hh] = torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, g]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


def dense(h, w, pre):
    return gelu(h @ w[pre + "up"].T) @ w[pre + "down"].T


def route(z, router):
    """Router logits [T, E] -> (weights [T, E], zero where not chosen; the margin [T] of the closest call: how far, as a
    difference of logits, the last expert or run that was taken lies above the first that was not)."""
    T, E = z.shape
    top = router["top"]
    s = torch.softmax(z, -1)
    gap = torch.full((T,), math.inf, dtype=F64)
    score, zc = s.clone(), z.clone()
    groups = router.get("groups")
    if groups:
        n, keep = groups["count"], groups["keep"]
        best, zbest = s.view(T, n, E // n).max(-1).values, z.view(T, n, E // n).max(-1).values
        kept = torch.zeros(T, n, dtype=torch.bool)
        kept.scatter_(1, torch.topk(best, keep, dim=-1).indices, True)
        if keep < n:
            ranked = torch.sort(zbest, dim=-1, descending=True).values
            gap = torch.minimum(gap, ranked[:, keep - 1] - ranked[:, keep])
        out_of_reach = ~kept.repeat_interleave(E // n, dim=1)
        score, zc = score.masked_fill(out_of_reach, -1.0), zc.masked_fill(out_of_reach, -math.inf)
    chosen = torch.topk(score, top, dim=-1).indices
    if top < E:
        ranked = torch.sort(zc, dim=-1, descending=True).values
        gap = torch.minimum(gap, ranked[:, top - 1] - ranked[:, top])
    wt = torch.zeros(T, E, dtype=F64).scatter_(1, chosen, s.gather(1, chosen))
    return wt / (wt.sum(-1, keepdim=True) + 1e-20), gap


def moe(h, w, pre, mlp, gaps=None):
    wt, gap = route(h @ w[pre + "router"].T, mlp["router"])
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros(h.shape[0], w[pre + "e0.down"].shape[0], dtype=F64)
    for e in range(mlp["router"]["experts"]):
        rows = torch.nonzero(wt[:, e]).flatten()
        if rows.numel():
            a = torch.relu(h[rows] @ w[f"{pre}e{e}.up"].T) ** 2
            out[rows] += wt[rows, e:e + 1] * (a @ w[f"{pre}e{e}.down"].T)
    return out


def forward(cfg, w, tokens, keep_layers=False, gaps=None):
    """Logits [T, vocab] of one sequence from its first token (and the stream after every layer)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kept, stored = [], {}
    for i, L in enumerate(cfg["layers"]):
        if L["type"] != "attention":
            raise ValueError(L["type"])
        pre, m = f"l{i}.", L["mixer"]
        h = layer_norm(x, w[pre + "norm1"], w[pre + "norm1.b"], eps)
        if m.get("kv_from") is None:
            stored[i] = keys_values(h, w, pre + "mix.", m)
        add = attention(h, stored[i if m.get("kv_from") is None else m["kv_from"]], w, pre + "mix.", m)
        mlp = L.get("mlp")
        if mlp:
            add = add + (dense(h, w, pre + "mlp.") if mlp["kind"] == "dense" else moe(h, w, pre + "mlp.", mlp, gaps))
        x = x + add
        kept.append(x.clone())
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(kept)) if keep_layers else logits


def load(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


class PlainGoridra:
    def __init__(self, folder):
        self.cfg, self.w = load(folder)

    def logits(self, tokens):
        return forward(self.cfg, self.w, tokens)

    def layers(self, tokens):
        """The stream after every layer, [layers, T, D]."""
        return forward(self.cfg, self.w, tokens, keep_layers=True)[1]

    def close_calls(self, tokens, margin):
        """The positions at which some router's choice hangs on less than `margin` of a logit: arithmetic of fewer bits
        may choose otherwise there, and no comparison at reduced precision should rest on them."""
        gaps = []
        forward(self.cfg, self.w, tokens, gaps=gaps)
        if not gaps:
            return set()
        return set(torch.nonzero(torch.stack(gaps).min(0).values < margin).flatten().tolist())


def generate(plain, prompt, n_new):
    """Greedy continuation, the whole sequence recomputed for every token."""
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(plain.logits(toks)[-1].argmax()))
    return toks[len(prompt):]
