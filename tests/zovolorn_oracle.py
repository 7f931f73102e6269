"""Plain, slow restatement of the Zovolorn design in float64 torch ops, one function per mechanism.  It shares no code with the
product path: tests build small random checkpoints with `random_model` and compare the framework against this.

Notation: x residual stream [T, W].  Every sublayer f reads c(x), the stream plus a short causal convolution of it over time, and
hands its result back through a norm in groups of channels: x <- x + gn(f(c(x)), w).
"""
import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


# ---- norms, convolution, activations -------------------------------------------------------------------------------
def unit_rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def grouped_norm(x, w, groups, eps):
    """Every one of `groups` equal runs of neighbouring channels is divided by its own root mean square."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return unit_rms(parts, eps).reshape(x.shape) * w


def causal_conv(x, w):
    """x [T, C], w [C, taps]: out_t = sum_j w[:, j] x_(t - taps + 1 + j), zeros before the first token."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.nn.functional.softplus(z, beta=1.0, threshold=200.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


# ---- embedding -----------------------------------------------------------------------------------------------------
def pair_rows(tokens, buckets, mul_prev, mul_cur):
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def embed(cfg, W, tokens):
    e = cfg["embedding"]
    x = W["embed"][torch.tensor(tokens)] * e["scale"]
    bg = e.get("bigram")
    if bg:
        x = x + W["bigram"][torch.tensor(pair_rows(tokens, bg["buckets"], bg["mul_prev"], bg["mul_cur"]))]
    return x


# ---- attention -----------------------------------------------------------------------------------------------------
def rotate_pairs(t, pos, dims, base):
    """t [T, heads, dim]: channels 2i and 2i + 1 (below `dims`) turn by pos * base^(-2i / dims)."""
    out = t.clone()
    for i in range(dims // 2):
        a = pos.to(F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = t[..., 2 * i], t[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def distance_bucket(n, n_buckets, far):
    """One bucket per distance up to half of the buckets, then buckets that widen in proportion to the distance until `far`."""
    half = n_buckets // 2
    if n < half:
        return n
    if far <= half:
        return n_buckets - 1
    # the largest e with (n / half)^m >= (far / half)^e, m = buckets of the widening part, in whole numbers
    m, e = n_buckets - half, 0
    while e < m and n ** m * half ** (e + 1) >= far ** (e + 1) * half ** m:
        e += 1
    return min(n_buckets - 1, half + e)


def softmax_attention(q, k, v, pos_q, pos_k, scale, sink=None, temp=None, rel=None, bias_max=0, chunk=0):
    """q [Tq, H, D], k [Tk, G, D], v [Tk, G, V] -> [Tq, H, V].  score = scale * q . k (times temp[h], plus the distance bucket's
    number rel[bucket, h]); keys of later positions, and of other chunks of `chunk` positions, are not seen; `sink` [H] adds
    exp(sink[h]) to the denominator."""
    Tq, H, _ = q.shape
    rep = H // k.shape[1]
    d = pos_q[:, None] - pos_k[None, :]
    seen = d >= 0
    if chunk:
        seen = seen & (pos_q[:, None] // chunk == pos_k[None, :] // chunk)
    bucket = None
    if rel is not None:
        of = torch.tensor([distance_bucket(n, rel.shape[0], bias_max) for n in range(int(d.max()) + 1)])
        bucket = of[d.clamp(min=0)]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].T * scale
        if temp is not None:
            s = s * temp[h]
        if rel is not None:
            s = s + rel[bucket, h]
        s = s.masked_fill(~seen, -float("inf"))
        m = s.max(-1, keepdim=True).values
        if sink is not None:
            m = torch.clamp(m, min=float(sink[h]))
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - m)
        out.append(e / den @ v[:, h // rep])
    return torch.stack(out, 1)


def attention_mixer(W, p, h, c, eps, pos):
    H, D, V = c["heads"], c["dim"], c["vdim"]
    G, T = c.get("kv_heads", H), h.shape[0]
    q = unit_rms(h @ W[p + "q"].T, eps, W[p + "q.norm"]).view(T, H, D)
    k = unit_rms(h @ W[p + "k"].T, eps, W[p + "k.norm"]).view(T, G, D)
    v = (h @ W[p + "v"].T).view(T, G, V)
    q, k = (rotate_pairs(t, pos, c["rot"]["dims"], c["rot"]["base"]) for t in (q, k))
    o = softmax_attention(q, k, v, pos, pos, c["scale"], sink=W[p + "sink"])
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ W[p + "o"].T


def chunked_branch(W, p, h, c, eps, pos):
    H, D = c["heads"], c["dim"]
    G, T = c.get("kv_heads", H), h.shape[0]
    q = unit_rms((h @ W[p + "q"].T).view(T, H, D), eps, W[p + "q.norm"])
    plain = (h @ W[p + "k"].T).view(T, G, D)
    k = unit_rms(plain, eps, W[p + "k.norm"])
    o = softmax_attention(q, k, plain, pos, pos, c["scale"], temp=W[p + "temp"], rel=W[p + "rel"], bias_max=c["bias_max"], chunk=c["mask"]["size"])
    return o.reshape(T, H * D) @ W[p + "o"].T


# ---- gated delta rule ------------------------------------------------------------------------------------------------
def log_decay(z, a_log, dim):
    """z [T, H * dim] -> log of the decay per head and key channel, [T, H, dim]."""
    return -torch.exp(a_log)[None, :, None] * softplus(z).view(z.shape[0], -1, dim)


def delta_recurrence(q, k, v, ld, beta, state=None):
    """q, k [T, H, D], v [T, H, V], ld [T, H, D], beta [T, H]: the state forgets per key channel, then is corrected towards v at k."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        S = torch.exp(ld[t])[:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def delta_branch(W, p, h, c, eps):
    H, D, V = c["heads"], c["dim"], c["vdim"]
    G, T = c.get("kv_heads", H), h.shape[0]
    q, k, v = (silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    rep = H // G
    q = (unit_vector(q.view(T, G, D)) * D ** -0.5).repeat_interleave(rep, 1)
    k = unit_vector(k.view(T, G, D)).repeat_interleave(rep, 1)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    ld = log_decay((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"], W[p + "A_log"], D)
    o, _ = delta_recurrence(q, k, v.view(T, H, V), ld, beta)
    o = unit_rms(o, eps, W[p + "norm"]).reshape(T, H * V) * torch.sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    return o @ W[p + "o"].T


def parallel_mixer(W, p, h, c, eps, pos):
    return c["left_scale"] * chunked_branch(W, p + "left.", h, c["left"], eps, pos) + c["right_scale"] * delta_branch(W, p + "right.", h, c["right"], eps)


# ---- feed-forward and output -----------------------------------------------------------------------------------------
def dense_ff(W, p, h):
    a = gelu_tanh(h @ W[p + "gate"].T + W[p + "gate.b"]) * (h @ W[p + "up"].T + W[p + "up.b"])
    return a @ W[p + "down"].T + W[p + "down.b"]


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


# ---- the model -------------------------------------------------------------------------------------------------------
def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence run whole."""
    tokens = [int(t) for t in tokens]
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    pos = torch.arange(len(tokens))
    x = embed(cfg, W, tokens)
    for i, L in enumerate(cfg["layers"]):
        p, c = f"l{i}.", L["mixer"]
        h = x + causal_conv(x, W[p + "canon1"])
        y = attention_mixer(W, p + "mix.", h, c, eps, pos) if L["type"] == "attention" else parallel_mixer(W, p + "mix.", h, c, eps, pos)
        x = x + grouped_norm(y, W[p + "norm1"], groups, eps)
        if L.get("mlp") is not None:
            h = x + causal_conv(x, W[p + "canon2"])
            x = x + grouped_norm(dense_ff(W, p + "mlp.", h), W[p + "norm2"], groups, eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return soft_cap(grouped_norm(x, W["final.norm"], groups, eps) @ W["embed"].T, cfg["logit_softcap"])


def greedy(cfg, W, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]


# ---- small random checkpoints ----------------------------------------------------------------------------------------
def attention_layer(heads=4, kv_heads=2, dim=12, vdim=10, rot_dims=8, base=300.0, scale=None, ff=40):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims},
                                           "scale": scale if scale is not None else dim ** -0.5},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel_layer(heads=4, kv_heads=2, dim=8, chunk=9, bias_max=14, scale=None, left_scale=0.7, right_scale=1.2, r_heads=4, r_kv_heads=2, r_dim=8,
                   r_vdim=12, conv=4, ff=40, buckets=8, rank=5, g_rank=3):
    """`buckets`, `rank` and `g_rank` only show in the tensors' shapes: they travel under a key the framework does not read."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else dim ** -0.5, "bias_max": bias_max,
            "mask": {"size": chunk}}
    right = {"heads": r_heads, "kv_heads": r_kv_heads, "dim": r_dim, "vdim": r_vdim, "conv": conv}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": left_scale, "right": right, "right_scale": right_scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None, "_shape": (buckets, rank, g_rank)}


def make_config(layers, width=32, vocab=53, embed_scale=1.7, eps=1e-5, groups=4, taps=3, cap=20.0, buckets=37, mul_prev=11, mul_cur=5):
    return {"architecture": "Zovolorn", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps}, "logit_softcap": cap, "layers": layers}


def random_model(cfg, seed=0):
    """float64 weights for `cfg`, every one exactly representable in bfloat16: a checkpoint written in bfloat16 holds the same numbers."""
    g = torch.Generator().manual_seed(seed)
    width, taps, W = cfg["width"], cfg["canon"]["taps"], {}

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(tuple(shape), generator=g, dtype=F64) * std + mean).to(torch.bfloat16).to(F64)

    lin = lambda o, i: rnd(o, i, std=i ** -0.5)
    W["embed"], W["bigram"] = rnd(cfg["vocab"], width), rnd(cfg["embedding"]["bigram"]["buckets"] + 1, width)
    for i, L in enumerate(cfg["layers"]):
        p, c = f"l{i}.", L["mixer"]
        W[p + "norm1"], W[p + "canon1"] = rnd(width, std=0.2, mean=1.0), rnd(width, taps, std=0.4)
        if L["type"] == "attention":
            m, H, D, V = p + "mix.", c["heads"], c["dim"], c["vdim"]
            G = c.get("kv_heads", H)
            W[m + "q"], W[m + "k"], W[m + "v"] = lin(H * D, width), lin(G * D, width), lin(G * V, width)
            W[m + "q.norm"], W[m + "k.norm"] = rnd(H * D, std=0.3, mean=1.5), rnd(G * D, std=0.3, mean=1.5)
            W[m + "sink"], W[m + "g"], W[m + "o"] = rnd(H), lin(H, width) * 2, lin(width, H * V)
        else:
            buckets, rank, g_rank = L["_shape"]
            m, a = p + "mix.left.", c["left"]
            H, D = a["heads"], a["dim"]
            G = a.get("kv_heads", H)
            W[m + "q"], W[m + "k"], W[m + "o"] = lin(H * D, width), lin(G * D, width), lin(width, H * D)
            W[m + "q.norm"], W[m + "k.norm"] = rnd(D, std=0.3, mean=1.3), rnd(D, std=0.3, mean=1.3)
            W[m + "rel"], W[m + "temp"] = rnd(buckets, H), rnd(H, std=0.3, mean=1.2)
            m, a = p + "mix.right.", c["right"]
            H, D, V = a["heads"], a["dim"], a["vdim"]
            G = a.get("kv_heads", H)
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                W[m + n], W[m + n + ".conv"] = lin(rows, width), rnd(rows, a["conv"], std=0.5)
            W[m + "b"], W[m + "A_log"], W[m + "dt_bias"] = lin(H, width), rnd(H, std=0.5, mean=-1.5), rnd(H * D)
            W[m + "a1"], W[m + "a2"] = lin(rank, width), lin(H * D, rank) * 0.5
            W[m + "g1"], W[m + "g2"], W[m + "norm"], W[m + "o"] = lin(g_rank, width), lin(H * V, g_rank), rnd(V, std=0.3, mean=1.0), lin(width, H * V)
        if L.get("mlp") is not None:
            ff = L["mlp"]["ff"]
            W[p + "norm2"], W[p + "canon2"] = rnd(width, std=0.2, mean=1.0), rnd(width, taps, std=0.4)
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = lin(ff, width), lin(ff, width), lin(width, ff)
            W[p + "mlp.gate.b"], W[p + "mlp.up.b"], W[p + "mlp.down.b"] = rnd(ff, std=0.3), rnd(ff, std=0.3), rnd(width, std=0.3)
    W["final.norm"] = rnd(width, std=0.2, mean=1.0)
    return W
