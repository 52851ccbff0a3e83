"""TEST INFRASTRUCTURE ONLY -- plain float64 restatement of the `Tiradra` design, one function per mechanism, written
from the equations; shares no code with the product path (llm_decoder.hybrid and the CUDA kernels).  Slow on purpose:
keys and values are built for every head, every sequence is recomputed from its first token.

Notation: a sequence is X [tokens, width]; position i counts from 0; n(x; w) = x / sqrt(mean(x^2) + eps) * (1 + w).

    X0          = E[token] + B[(previous token * a + token * b) mod buckets]      (B's last row for the first token)
    layer       X <- X + mixer(n(X; w1)) + ff(n(X; w2))                           (both read the same X)
    block pass  t = 0, 1, ...:  X <- X + (X0 if t > 0) + step_t, then the block's layers
    logits      cap * tanh(head n(X; w_final) / cap)
"""
import math

import torch

F = torch.float64


# ------------------------------------------------------------------------------------------------------- small functions
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm1p(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_row(prev, tok, a, b, buckets):
    """Row of the pair table; prev is None for a sequence's first token."""
    return buckets if prev is None else (prev * a + tok * b) % buckets


def embed(W, emb, tokens):
    rows = []
    bg = emb["bigram"]
    for i, tok in enumerate(tokens):
        r = bigram_row(tokens[i - 1] if i else None, tok, bg["mul_prev"], bg["mul_cur"], bg["buckets"])
        rows.append(W["embed"][tok] + W["bigram"][r])
    return torch.stack(rows)


def stretched_frequencies(dims, base, sc):
    """Angle per position of every pair, and the factor on cos and sin.  Fast pairs keep their frequency, slow ones are
    divided by the factor, with a linear ramp over the pair index in between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0

    def turns(t):
        return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns(sc["fast"])), 0), min(math.ceil(turns(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def turn_neighbours(x, pos, rot):
    """One head vector at position pos: entries 2i and 2i + 1 of x[:dims] turn with each other."""
    f, mult = stretched_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    y = x.clone()
    for i, fi in enumerate(f):
        c, s = math.cos(pos * fi) * mult, math.sin(pos * fi) * mult
        u, v = x[2 * i], x[2 * i + 1]
        y[2 * i] = u * c - v * s
        y[2 * i + 1] = v * c + u * s
    return y


def turn_all(x, rot):
    """x [tokens, heads, dim]: every head vector turned by its token's position."""
    dims = rot["dims"]
    if dims == 0:
        return x
    f, mult = stretched_frequencies(dims, rot["base"], rot.get("scaling"))
    ang = torch.arange(x.shape[0], dtype=F)[:, None] * torch.tensor(f, dtype=F)
    c, s = torch.cos(ang)[:, None] * mult, torch.sin(ang)[:, None] * mult
    y = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * c - v * s
    y[..., 1:dims:2] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------------------------ mechanisms
def short_convolution(u, w):
    """u [T, channels], w [channels, taps]: y_t = sum_j w_j u_(t - taps + 1 + j), nothing before the first token."""
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] += w[:, j] * u[t - taps + 1 + j]
    return y


def softmax_attention(q, k, v, scale, sink=None):
    """Causal softmax, one query at a time; q, k [T, H, d], v [T, H, e].  sink [H]: a logit per head that takes its share
    of the weights and gives nothing back."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        for i in range(T):
            s = [float(q[i, h] @ k[j, h]) * scale for j in range(i + 1)]
            m = max(s + ([float(sink[h])] if sink is not None else []))
            w = [math.exp(z - m) for z in s]
            total = sum(w) + (math.exp(float(sink[h]) - m) if sink is not None else 0.0)
            for j in range(i + 1):
                out[i, h] += w[j] / total * v[j, h]
    return out


def softmax_attention_matrix(q, k, v, scale, sink=None):
    """The same numbers with one weight matrix per head (for long sequences)."""
    T, H, _ = q.shape
    vis = torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T * scale).masked_fill(~vis, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[h].expand(T, 1)], 1)
        out[:, h] = torch.softmax(s, -1)[:, :T] @ v[:, h]
    return out


FORM = "matrix"


def attend(*args):
    return (softmax_attention if FORM == "loop" else softmax_attention_matrix)(*args)


def attention_mixer(h, W, p, c, eps):
    """Grouped heads; biased projections through a short convolution; turned, then divided by their root mean square."""
    T, H, G, d, e = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (short_convolution(h @ W[p + n].T + W[p + n + ".b"], W[p + n + ".conv"]) for n in "qkv")
    q = rms(turn_all(q.reshape(T, H, d), c["rot"]), eps)
    k = rms(turn_all(k.reshape(T, G, d), c["rot"]), eps)
    v = v.reshape(T, G, e)
    group = [hh // (H // G) for hh in range(H)]
    return attend(q, k[:, group], v[:, group], c["scale"]).reshape(T, H * e) @ W[p + "o"].T


def latent_mixer(h, W, p, c, eps):
    """Per-head keys and values built from a normed latent, next to one turned key part that all heads share; a sink per
    head; the heads' outputs gated element by element."""
    T, H, d, r, kr, e = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"], c["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, d + r)
    down = h @ W[p + "dkv"].T
    lat = rms(down[:, :kr], eps) * W[p + "dkv.norm"]
    shared = turn_all(down[:, None, kr:], c["rot"]).expand(T, H, r)
    k = torch.cat([(lat @ W[p + "uk"].T).reshape(T, H, d), shared], -1)
    v = (lat @ W[p + "uv"].T).reshape(T, H, e)
    q = torch.cat([q[..., :d], turn_all(q[..., d:], c["rot"])], -1)
    o = attend(q, k, v, c["scale"], W[p + "sink"]).reshape(T, H * e)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def dense_ff(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


MIXER = {"attention": attention_mixer, "latent_attention": latent_mixer}


def layer_order(config):
    """[(layer, pass number where the layer is the first of a pass, else None)]."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(config, weights, tokens, layers_out=None):
    """Logits [tokens, vocab] in float64; layers_out (a list) gets the residual after every layer run."""
    W = {n: t.to(F) for n, t in weights.items()}
    eps, cap = config["norm"]["eps"], config.get("logit_softcap")
    x0 = embed(W, config["embedding"], list(tokens))
    x = x0.clone()
    for i, t in layer_order(config):
        lc, p = config["layers"][i], f"l{i}."
        if t is not None:
            x = (x + x0 if t else x) + W["loop.step"][t]
        y = MIXER[lc["type"]](norm1p(x, W[p + "norm1"], eps), W, p + "mix.", lc["mixer"], eps)
        if lc.get("mlp"):
            y = y + dense_ff(norm1p(x, W[p + "norm2"], eps), W, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    logits = norm1p(x, W["final.norm"], eps) @ W["head"].T
    return cap * torch.tanh(logits / cap) if cap else logits


# ------------------------------------------------------------------------------- configurations and weights of the tests
def scaling(factor=4.0, original=64, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=None, taps=4, rot_dims=None, base=10000.0, sc="default", scale=None, ff=48):
    vdim = dim if vdim is None else vdim
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps,
                      "rot": {"dims": dim if rot_dims is None else rot_dims, "base": base, "scaling": scaling() if sc == "default" else sc},
                      "scale": 0.5 if scale is None else scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent_layer(heads=3, dim=12, rot_dim=8, vdim=20, kv_rank=16, base=10000.0, sc="default", scale=None, ff=48):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "rot": {"dims": rot_dim, "base": base, "scaling": scaling(2.5, 128, 16.0, 0.5) if sc == "default" else sc},
                      "scale": (dim + rot_dim) ** -0.5 if scale is None else scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def make_config(layers, width=48, vocab=71, eps=1e-5, loop=None, buckets=89, mul_prev=31, mul_cur=5, cap=20.0):
    return {"architecture": "Tiradra", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "loop": loop,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "logit_softcap": cap}


def random_weights(config, seed=0):
    g = torch.Generator().manual_seed(seed)
    Wd = config["width"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * s / math.sqrt(i)).to(torch.bfloat16)

    def vec(n, std, mean=0.0):
        return (torch.randn(n, generator=g) * std + mean).to(torch.bfloat16)

    W = {"embed": torch.randn(config["vocab"], Wd, generator=g).to(torch.bfloat16),
         "bigram": torch.randn(config["embedding"]["bigram"]["buckets"] + 1, Wd, generator=g).to(torch.bfloat16),
         "head": mat(config["vocab"], Wd, 4.0), "final.norm": vec(Wd, 0.2)}
    if config.get("loop"):
        W["loop.step"] = torch.randn(config["loop"]["times"], Wd, generator=g).mul(0.7).to(torch.bfloat16)
    for i, lc in enumerate(config["layers"]):
        p, m, c = f"l{i}.", f"l{i}.mix.", lc["mixer"]
        H = c["heads"]
        W[p + "norm1"] = vec(Wd, 0.2)
        if lc["type"] == "attention":
            G, d, e, taps = c["kv_heads"], c["dim"], c["vdim"], c["conv"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
                W[m + n], W[m + n + ".b"] = mat(rows, Wd), vec(rows, 0.5)
                W[m + n + ".conv"] = torch.randn(rows, taps, generator=g).mul(0.6).to(torch.bfloat16)
        else:
            d, r, e, kr = c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
            W[m + "q"], W[m + "dkv"], W[m + "dkv.norm"] = mat(H * (d + r), Wd, 1.5), mat(kr + r, Wd), vec(kr, 0.3, 1.0)
            W[m + "uk"], W[m + "uv"], W[m + "g"] = mat(H * d, kr, 1.5), mat(H * e, kr), mat(H * e, Wd)
            W[m + "sink"] = vec(H, 1.0, 1.0)
        W[m + "o"] = mat(Wd, H * e)
        if lc.get("mlp"):
            ff = lc["mlp"]["ff"]
            W[p + "norm2"] = vec(Wd, 0.2)
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = mat(ff, Wd), mat(ff, Wd), mat(Wd, ff)
    return W
