"""A plain, slow Mavinex: one function per mechanism, float64 on the CPU.

It shares no code with the package: it reads config.json and the safetensors file by itself
(through torch only) and follows the equations below literally.

Notation.  x_t is the residual stream at token t (width D), p its position in its sequence, R(u) = u / sqrt(mean(u^2) + eps).
    embedding   x_t = s E[tok_t]
    norm        N(x; w) = R(x) * (1 + w)
    layer       x <- N_1(a x + M(x));   x <- N_2(a x + F(x))               (the second only if the layer has an F)
    a layer with `weights_of` j computes with layer j's tensors; keys, values and states are its own

Mixer "parallel":  M = (R(A(x)) * w_left + R(B(x)) * w_right) / 2
    A, attention (H query heads over G key heads, key size d, value size dv): q = R(Wq x) * wq, k = R(Wk x) * wk, the norms
        over ALL rows of a projection, v = Wv x; pairs (2i, 2i + 1) of the first `dims` dimensions of every head of q and k
        turned by p f_i; s_j = scale q . k_j for t - size < j <= t; A = Wo (concat_h sum_j softmax(s)_j v_j * sigmoid(Wg x))
    B, selective scan over C channels with N states each: [u0 | z] = Win x; u = silu(conv(u0) + cb), causal, per channel;
        [r | b | c] = Wx u; dt = softplus(Wdt r + db); S[c, n] <- exp(-dt_c e^(Alog[c, n])) S[c, n] + dt_c u_c b_n;
        y_c = sum_n S[c, n] c_n + D_c u_c; B = Wo (y * silu(z))
Mixer "latent_attention": q = Wq x, per head [d without position | r turned]; [l | kr] = Wdkv x, l <- R(l) * wl;
    k_h = [Wuk_h l | turned kr], v_h = Wuv_h l; the turned part pairs i with i + r/2, angle p f_i, cosine and sine times m;
    s_j = scale q . k_j for t - size < j <= t; weights exp(s_j) / (exp(sink_h) + sum exp(s_j));
    M = Wo concat_h (o_h sigmoid(Wg x)_h)
Frequencies f_i = base^(-2i/dims), rescaled by wavelength (low / high) in the first attention and by YaRN in the second.
Feed-forward "moe": z = Wr x + br; the `top` largest z choose, weights = softmax over them; expert Wdown(silu(Wgate x) * Wup x)
Logits: head N_final(x).
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


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def frequencies(dims, base, scaling):
    """(f_i, the factor of cosine and sine) for i < dims / 2, in double precision."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, orig = scaling["factor"], scaling["original"]
    if "low" in scaling:
        out = []
        for v in f:
            wave = 2 * math.pi / v
            if wave < orig / scaling["high"]:
                out.append(v)
            elif wave > orig / scaling["low"]:
                out.append(v / factor)
            else:
                s = (orig / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                out.append((1 - s) * v / factor + s * v)
        return out, 1.0

    def turns(t):              # the dimension whose wave makes t turns in `orig` positions
        return dims * math.log(orig / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
    return [v / factor * r + v * (1 - r) for v, r in zip(f, ramp)], 0.1 * math.log(factor) + 1.0


def turn(x, pos, rot, halves):
    """x [T, heads, n] with its first rot.dims dimensions turned by the positions pos [T]: i paired with i + dims/2
    (halves) or 2i with 2i + 1."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    f, m = frequencies(dims, rot["base"], rot.get("scaling"))
    ang = pos.to(F64)[:, None] * torch.tensor(f, dtype=F64)[None, :]
    c, s = (m * torch.cos(ang))[:, None, :], (m * torch.sin(ang))[:, None, :]
    a, b = (x[..., :dims // 2], x[..., dims // 2:dims]) if halves else (x[..., 0:dims:2], x[..., 1:dims:2])
    u, v = a * c - b * s, b * c + a * s
    turned = torch.cat([u, v], -1) if halves else torch.stack([u, v], -1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], -1)


def visible(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i - j < size) if size else seen


def softmax_with_sink(s, sink=None):
    """softmax over the last axis; `sink`: one more score in the denominator, without a key."""
    if sink is None:
        return torch.softmax(s, -1)
    top = torch.maximum(s.max(-1, keepdim=True).values, torch.as_tensor(sink, dtype=F64))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention(h, w, pre, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (rms(h @ w[pre + "q"].T, eps) * w[pre + "q.norm"]).view(T, H, d)
    k = (rms(h @ w[pre + "k"].T, eps) * w[pre + "k.norm"]).view(T, G, d)
    v = (h @ w[pre + "v"].T).view(T, G, dv)
    q, k = turn(q, pos, m.get("rot"), False), turn(k, pos, m.get("rot"), False)
    seen = visible(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        out[:, hh] = softmax_with_sink(s.masked_fill(~seen, -math.inf)) @ v[:, g]
    return (out.reshape(T, H * dv) * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K], the last column the current token's; zeros before the start."""
    K = taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(K)) + bias


def scan(u, dt, A, b, c):
    """The recurrence alone: u, dt [T, C], A [C, N], b, c [T, N] -> sum_n S[c, n] c_n per token [T, C]."""
    S = torch.zeros_like(A)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * u[t])[:, None] * b[t][None, :]
        out[t] = S @ c[t]
    return out


def selective_scan(h, w, pre, m):
    C, N, r = m["inner"], m["state"], m["dt_rank"]
    both = h @ w[pre + "in"].T
    u = silu(causal_conv(both[:, :C], w[pre + "conv"], w[pre + "conv.b"]))
    thin = u @ w[pre + "x"].T
    dt = torch.nn.functional.softplus(thin[:, :r] @ w[pre + "dt"].T + w[pre + "dt.b"], threshold=50.0)
    y = scan(u, dt, -torch.exp(w[pre + "A_log"]), thin[:, r:r + N], thin[:, r + N:r + 2 * N]) + w[pre + "D"] * u
    return (y * silu(both[:, C:])) @ w[pre + "o"].T


def parallel(h, w, pre, m, eps):
    a, b = attention(h, w, pre + "left.", m["left"], eps), selective_scan(h, w, pre + "right.", m["right"])
    return 0.5 * (rms(a, eps) * w[pre + "left.out"] + rms(b, eps) * w[pre + "right.out"])


def latent_attention(h, w, pre, m, eps):
    T = h.shape[0]
    H, d, dv, r, rd = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["rot_dim"]
    pos = torch.arange(T)
    q = (h @ w[pre + "q"].T).view(T, H, d + rd)
    down = h @ w[pre + "dkv"].T
    lat = rms(down[:, :r], eps) * w[pre + "dkv.norm"]
    k_plain, v = (lat @ w[pre + "uk"].T).view(T, H, d), (lat @ w[pre + "uv"].T).view(T, H, dv)
    q_turned = turn(q[..., d:], pos, m.get("rot"), True)
    k_turned = turn(down[:, None, r:], pos, m.get("rot"), True)[:, 0]
    gate = torch.sigmoid(h @ w[pre + "g"].T)
    seen = visible(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        s = (q[:, hh, :d] @ k_plain[:, hh].T + q_turned[:, hh] @ k_turned.T) * m["scale"]
        p = softmax_with_sink(s.masked_fill(~seen, -math.inf), w[pre + "sink"][hh])
        out[:, hh] = (p @ v[:, hh]) * gate[:, hh:hh + 1]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


def route(z, top):
    """Logits [T, E] -> (weights [T, E], zero where not chosen; the margin [T] between the last one chosen and the next)."""
    ranked = torch.sort(z, dim=-1, descending=True)
    gap = ranked.values[:, top - 1] - ranked.values[:, top] if top < z.shape[1] else torch.full((z.shape[0],), math.inf, dtype=F64)
    wt = torch.zeros_like(z).scatter_(1, ranked.indices[:, :top], torch.softmax(ranked.values[:, :top], -1))
    return wt, gap


def moe(h, w, pre, mlp, gaps=None):
    wt, gap = route(h @ w[pre + "router"].T + w[pre + "router.b"], mlp["router"]["top"])
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows = torch.nonzero(wt[:, e]).flatten()
        if rows.numel():
            a = silu(h[rows] @ w[f"{pre}e{e}.gate"].T) * (h[rows] @ w[f"{pre}e{e}.up"].T)
            out[rows] += wt[rows, e:e + 1] * (a @ w[f"{pre}e{e}.down"].T)
    return out


def owner(cfg, i):
    """The layer whose tensors layer i computes with."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, tokens, keep_layers=False, gaps=None):
    """Logits [T, vocab] of one sequence from its first token (and the stream after every layer)."""
    eps, a = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    kept = []
    for i, L in enumerate(cfg["layers"]):
        pre, m = f"l{owner(cfg, i)}.", L["mixer"]
        y = {"parallel": parallel, "latent_attention": latent_attention}[L["type"]](x, w, pre + "mix.", m, eps)
        x = rms(a * x + y, eps) * (1 + w[pre + "norm1"])
        if L.get("mlp"):
            x = rms(a * x + moe(x, w, pre + "mlp.", L["mlp"], gaps), eps) * (1 + w[pre + "norm2"])
        kept.append(x.clone())
    logits = (rms(x, eps) * (1 + w["final.norm"])) @ w["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


def load(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


class PlainMavinex:
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
