"""TEST INFRASTRUCTURE ONLY -- plain float64 restatement of the `Namudra` design, one function per mechanism, written
from the equations; shares no code with the product path (llm_decoder.hybrid and the CUDA kernels).  Slow on purpose:
keys and values are built for every head, the recurrence walks token by token, every sequence is recomputed from its
first token.

Notation: a sequence is X [streams, tokens, width]; position i counts from 0.

    norm(x; w)      = x / sqrt(mean(x^2) + eps) * (1 + w)
    sublayer q      u = sum_s a[s] X_s;  y = f(norm(u; w_q));  X_t <- sum_s M[s, t] X_s + b[t] y      (a, M, b of sublayer q)
    layer           the mixer's sublayer, then the feed-forward's (none where the layer has no feed-forward)
    looped block    layers [start, stop) run `times` times in a row
    logits          head norm(sum_s X_s; w_final)
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


def silu(z):
    return z * sigmoid(z)


def turn_halves(x, pos, dims, base):
    """One head vector at position pos: entry i of the first half of x[:dims] turns with entry i of the second half."""
    y = x.clone()
    half = dims // 2
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[i], x[i + half]
        y[i] = u * math.cos(a) - v * math.sin(a)
        y[i + half] = v * math.cos(a) + u * math.sin(a)
    return y


def turn_all(x, dims, base):
    """x [tokens, heads, dim]: every head vector turned by its token's position."""
    if dims == 0:
        return x
    T, half = x.shape[0], dims // 2
    ang = torch.arange(T, dtype=F)[:, None] * torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def sees_window(i, j, size):
    return 0 <= i - j < size


# ------------------------------------------------------------------------------------------------------------ mechanisms
def sigmoid_attention(q, k, v, per, scale, head_bias, size):
    """q [T, H, d]; k, v [T, G, d]; query head h reads key/value head h // per.  One query, one key at a time: the weight
    of a visible key is sigmoid(score + bias of the head), and nothing divides the sum."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        for i in range(T):
            for j in range(T):
                if sees_window(i, j, size):
                    out[i, h] += sigmoid((q[i, h] @ k[j, h // per]) * scale + head_bias[h]) * v[j, h // per]
    return out


def sigmoid_attention_matrix(q, k, v, per, scale, head_bias, size):
    """The same numbers with one weight matrix per head (for long sequences)."""
    T, H, _ = q.shape
    d = torch.arange(T)[:, None] - torch.arange(T)[None]
    vis = (d >= 0) & (d < size)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        out[:, h] = (sigmoid(q[:, h] @ k[:, h // per].T * scale + head_bias[h]) * vis) @ v[:, h // per]
    return out


def softmax_attention(q, k, v, scale):
    """Causal softmax, one query at a time; q, k [T, H, d], v [T, H, e]."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        for i in range(T):
            s = k[:i + 1, h] @ q[i, h] * scale
            w = torch.exp(s - s.max())
            out[i, h] = (w / w.sum()) @ v[:i + 1, h]
    return out


def softmax_attention_matrix(q, k, v, scale):
    T, H, _ = q.shape
    vis = torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        out[:, h] = torch.softmax((q[:, h] @ k[:, h].T * scale).masked_fill(~vis, -math.inf), -1) @ v[:, h]
    return out


def retain(q, k, v, decay):
    """S <- decay_h S + k v^T, o = S^T q per head, token by token; q, k [T, H, d], v [T, H, e]."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        S = torch.zeros(d, v.shape[-1], dtype=F)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


FORM = "matrix"


def window_mixer(h, W, p, c, eps):
    """Windowed sigmoid attention on per-head normed queries and keys; the values are the keys before their norm; the
    heads' outputs are gated element by element."""
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q = (h @ W[p + "q"].T).reshape(T, H, d)
    k = (h @ W[p + "k"].T).reshape(T, G, d)
    v = k
    q, k = rms(q, eps) * W[p + "q.norm"], rms(k, eps) * W[p + "k.norm"]
    att = sigmoid_attention if FORM == "loop" else sigmoid_attention_matrix
    o = att(q, k, v, H // G, c["scale"], W[p + "pb"], c["mask"]["size"])
    return (o.reshape(T, H * d) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def latent_mixer(h, W, p, c, eps):
    """Queries through a normed latent; per-head keys and values built from the normed latent of the key side, next to one
    turned key part that all heads share; causal softmax."""
    T, H, d, r, kr = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    q = (rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T
    q = q.reshape(T, H, d + r)
    down = h @ W[p + "dkv"].T
    lat = rms(down[:, :kr], eps) * W[p + "dkv.norm"]
    dims, base = c["rot"]["dims"], c["rot"]["base"]
    shared = turn_all(down[:, None, kr:], dims, base).expand(T, H, r)
    k = torch.cat([(lat @ W[p + "uk"].T).reshape(T, H, d), shared], -1)
    v = (lat @ W[p + "uv"].T).reshape(T, H, c["vdim"])
    q = torch.cat([q[..., :d], turn_all(q[..., d:], dims, base)], -1)
    att = softmax_attention if FORM == "loop" else softmax_attention_matrix
    return att(q, k, v, c["scale"]).reshape(T, H * c["vdim"]) @ W[p + "o"].T


def retention_mixer(h, W, p, c, eps):
    """Linear attention with a constant decay per head on turned queries and keys, keys scaled by dim^(-1/2); the heads'
    outputs are divided by their root mean square and gated by silu."""
    T, H, d, e = h.shape[0], c["heads"], c["dim"], c["vdim"]
    dims, base = c["rot"]["dims"], c["rot"]["base"]
    q = turn_all((h @ W[p + "q"].T).reshape(T, H, d), dims, base)
    k = turn_all((h @ W[p + "k"].T).reshape(T, H, d), dims, base) * d ** -0.5
    v = (h @ W[p + "v"].T).reshape(T, H, e)
    o = rms(retain(q, k, v, c["decay"]), eps).reshape(T, H * e)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def dense_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


MIXER = {"attention": window_mixer, "latent_attention": latent_mixer, "retention": retention_mixer}


def sublayer(X, W, p, f):
    """u = sum_s in[s] X_s, y = f(u), then every stream t from the old ones: sum_s mix[s, t] X_s + out[t] y."""
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + W[p + "in"][s] * X[s]
    y = f(u)
    new = []
    for t in range(X.shape[0]):
        new.append(sum(W[p + "mix"][s, t] * X[s] for s in range(X.shape[0])) + W[p + "out"][t] * y)
    return torch.stack(new)


def layer_order(config):
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(config, weights, tokens, layers_out=None):
    """Logits [tokens, vocab] in float64; layers_out (a list) gets the sum of the streams after every layer run."""
    W = {n: t.to(F) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    X = torch.stack([x] * config["streams"])
    for i in layer_order(config):
        lc, p = config["layers"][i], f"l{i}."
        X = sublayer(X, W, p + "hc1.", lambda u: MIXER[lc["type"]](norm1p(u, W[p + "norm1"], eps), W, p + "mix.", lc["mixer"], eps))
        if lc.get("mlp"):
            X = sublayer(X, W, p + "hc2.", lambda u: dense_ff(norm1p(u, W[p + "norm2"], eps), W, p + "mlp."))
        if layers_out is not None:
            layers_out.append(X.sum(0))
    return norm1p(X.sum(0), W["final.norm"], eps) @ W["head"].T


# ------------------------------------------------------------------------------- configurations and weights of the tests
def window_layer(heads=4, kv_heads=2, dim=16, size=9, scale=None, ff=48):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": size},
                                           "scale": dim ** -0.5 if scale is None else scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent_layer(heads=3, dim=12, rot_dim=8, vdim=20, q_rank=24, kv_rank=16, base=10000.0, scale=None, ff=48):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "rot": {"dims": rot_dim, "base": base}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def retention_layer(heads=2, dim=16, vdim=12, rot_dims=16, base=10000.0, decay=None, ff=None):
    decay = [1.0 - 2.0 ** -(3 + h) for h in range(heads)] if decay is None else decay
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot_dims, "base": base},
                                           "decay": decay},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def make_config(layers, width=48, vocab=71, streams=2, eps=1e-5, loop=None):
    return {"architecture": "Namudra", "layers": layers, "width": width, "vocab": vocab, "streams": streams,
            "norm": {"eps": eps}, "loop": loop}


def random_weights(config, seed=0):
    g = torch.Generator().manual_seed(seed)
    Wd, S = config["width"], config["streams"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * s / math.sqrt(i)).to(torch.bfloat16)

    def vec(n, std, mean=0.0):
        return (torch.randn(n, generator=g) * std + mean).to(torch.bfloat16)

    W = {"embed": torch.randn(config["vocab"], Wd, generator=g).to(torch.bfloat16), "head": mat(config["vocab"], Wd),
         "final.norm": vec(Wd, 0.2)}
    for i, lc in enumerate(config["layers"]):
        p, m = f"l{i}.", f"l{i}.mix."
        c, H = lc["mixer"], lc["mixer"]["heads"]
        W[p + "norm1"] = vec(Wd, 0.2)
        for q in (1, 2) if lc.get("mlp") else (1,):
            W[p + f"hc{q}.in"] = vec(S, 0.4, 1.0 / S)
            W[p + f"hc{q}.out"] = vec(S, 0.4, 1.0)
            W[p + f"hc{q}.mix"] = (torch.eye(S) * 0.7 + torch.randn(S, S, generator=g) * 0.2).to(torch.bfloat16)
        if lc["type"] == "attention":
            G, d = c["kv_heads"], c["dim"]
            W[m + "q"], W[m + "k"], W[m + "g"], W[m + "o"] = mat(H * d, Wd), mat(G * d, Wd), mat(H * d, Wd), mat(Wd, H * d)
            W[m + "q.norm"], W[m + "k.norm"], W[m + "pb"] = vec(d, 0.3, 1.5), vec(d, 0.3, 1.5), vec(H, 0.5, -1.0)
        elif lc["type"] == "latent_attention":
            d, r, e, qr, kr = c["dim"], c["rot_dim"], c["vdim"], c["q_rank"], c["kv_rank"]
            W[m + "dq"], W[m + "dq.norm"], W[m + "uq"] = mat(qr, Wd), vec(qr, 0.3, 1.5), mat(H * (d + r), qr)
            W[m + "dkv"], W[m + "dkv.norm"] = mat(kr + r, Wd), vec(kr, 0.3, 1.0)
            W[m + "uk"], W[m + "uv"], W[m + "o"] = mat(H * d, kr), mat(H * e, kr), mat(Wd, H * e)
        else:
            d, e = c["dim"], c["vdim"]
            W[m + "q"], W[m + "v"] = mat(H * d, Wd), mat(H * e, Wd)
            # keys that lean towards the queries: a token meets its own key with a score well above zero, so the norm of a
            # head (no weight, small eps) does not blow up the rounding of a nearly empty state
            W[m + "k"] = (0.8 * W[m + "q"].float() + mat(H * d, Wd, 0.6).float()).to(torch.bfloat16)
            W[m + "g"], W[m + "o"] = mat(H * e, Wd), mat(Wd, H * e)
        if lc.get("mlp"):
            ff = lc["mlp"]["ff"]
            W[p + "norm2"] = vec(Wd, 0.2)
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = mat(ff, Wd), mat(ff, Wd), mat(Wd, ff)
    return W
