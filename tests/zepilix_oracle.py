"""Plain, slow restatement of the Zepilix design in float64 torch ops, one function per mechanism.  It shares no code with the product
path: tests build small random checkpoints with `random_model` and compare the framework against this.

Notation: x residual stream [T, W].  A layer adds its mixer and its feed-forward, both of normed copies of the SAME x, then a gated
projection of a second, per-layer token embedding; a span of layers may run several times.
"""
import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


# ---- norms, convolution, activations -------------------------------------------------------------------------------
def unit_rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def stream_norm(x, w, eps):
    """The layers' norm: the stored weight is what is added to one."""
    return unit_rms(x, eps) * (1.0 + w)


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.nn.functional.softplus(z, beta=1.0, threshold=200.0)


def causal_conv(x, w):
    """x [T, C], w [C, taps]: out_t = sum_j w[:, j] x_(t - taps + 1 + j), zeros before the first token."""
    T, taps = x.shape[0], w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(w[:, j] * pad[j:j + T] for j in range(taps))


def rotate_pairs(t, pos, dims, base):
    """t [T, heads, dim]: channels 2i and 2i + 1 (below `dims`) turn by pos * base^(-2i / dims)."""
    out = t.clone()
    for i in range(dims // 2):
        a = pos.to(F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = t[..., 2 * i], t[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---- attention -----------------------------------------------------------------------------------------------------
def softmax_attention(q, k, v, pos_q, pos_k, scale, window=0):
    """q [Tq, H, D], k [Tk, G, D], v [Tk, G, V] -> [Tq, H, V]; later keys are not seen, nor (window > 0) keys `window` or more back."""
    rep = q.shape[1] // k.shape[1]
    d = pos_q[:, None] - pos_k[None, :]
    hidden = d < 0
    if window:
        hidden = hidden | (d >= window)
    out = []
    for h in range(q.shape[1]):
        s = (q[:, h] @ k[:, h // rep].T * scale).masked_fill(hidden, -float("inf"))
        out.append(torch.softmax(s, -1) @ v[:, h // rep])
    return torch.stack(out, 1)


def attention_mixer(W, p, h, c, eps, pos):
    """Values are the keys as projected; the unit-RMS norm of a query or key head comes after its rotation."""
    H, D, T = c["heads"], c["dim"], h.shape[0]
    G, rot = c["kv_heads"], c["rot"]
    q, k = (h @ W[p + "q"].T).view(T, H, D), (h @ W[p + "k"].T).view(T, G, D)
    qn, kn = (unit_rms(rotate_pairs(t, pos, rot["dims"], rot["base"]), eps) for t in (q, k))
    return softmax_attention(qn, kn, k, pos, pos, c["scale"]).reshape(T, H * D) @ W[p + "o"].T


def latent_attention_mixer(W, p, h, c, eps, pos):
    H, D, R, V, C, T = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"], h.shape[0]
    rot = c["rot"]
    q = (unit_rms(h @ W[p + "dq"].T, eps, W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, D + R)
    down = h @ W[p + "dkv"].T
    lat = unit_rms(down[:, :C], eps, W[p + "dkv.norm"])
    turn = lambda t: rotate_pairs(t, pos, rot["dims"], rot["base"])
    k_rot = turn(down[:, C:].view(T, 1, R)).expand(T, H, R)
    q = torch.cat([q[..., :D], turn(q[..., D:])], -1)
    k = torch.cat([(lat @ W[p + "uk"].T).view(T, H, D), k_rot], -1)
    v = (lat @ W[p + "uv"].T).view(T, H, V)
    return softmax_attention(q, k, v, pos, pos, c["scale"], window=c["mask"]["size"]).reshape(T, H * V) @ W[p + "o"].T


# ---- gated delta rule ------------------------------------------------------------------------------------------------
def log_decay(z, a_log, dt_bias):
    """z [T, H] -> log of every head's decay, [T, H]."""
    return -torch.exp(a_log) * softplus(z + dt_bias)


def delta_recurrence(q, k, v, ld, beta, state=None):
    """q, k [T, H, D], v [T, H, V], ld [T, H], beta [T, H]: the state forgets, then is corrected towards v at k, then is read at q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        S = torch.exp(ld[t])[:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def delta_mixer(W, p, h, c, eps):
    H, G, D, V, T = c["heads"], c["kv_heads"], c["dim"], c["vdim"], h.shape[0]
    q, k, v = (silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = (unit_vector(q.view(T, G, D)) * D ** -0.5).repeat_interleave(H // G, 1)
    k = unit_vector(k.view(T, G, D)).repeat_interleave(H // G, 1)
    ld = log_decay(h @ W[p + "a"].T, W[p + "A_log"], W[p + "dt_bias"])
    o, _ = delta_recurrence(q, k, v.view(T, H, V), ld, torch.sigmoid(h @ W[p + "b"].T))
    return (unit_rms(o, eps, W[p + "norm"]).reshape(T, H * V) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---- feed-forward, token side input ------------------------------------------------------------------------------------
def dense_ff(W, p, h):
    a = silu(h @ W[p + "gate"].T + W[p + "gate.b"]) * (h @ W[p + "up"].T + W[p + "up.b"])
    return a @ W[p + "down"].T + W[p + "down.b"]


def side_input(x, e, gate, proj, w, eps):
    """What a layer adds from its part e [T, dim] of the tokens' second embedding."""
    return unit_rms((gelu_tanh(x @ gate.T) * e) @ proj.T, eps, w)


# ---- the model -------------------------------------------------------------------------------------------------------
def run_order(cfg):
    """(layer, number of the pass that begins with it, or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence run whole."""
    ids = torch.tensor([int(t) for t in tokens])
    eps, pos = cfg["norm"]["eps"], torch.arange(len(ids))
    x = x0 = W["embed"][ids]
    for i, begins in run_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        c, m = L["mixer"], p + "mix."
        if begins is not None:
            x = x + (x0 if begins > 0 else 0.0) + W["loop.step"][begins]
        h = stream_norm(x, W[p + "norm1"], eps)
        if L["type"] == "delta":
            y = delta_mixer(W, m, h, c, eps)
        else:
            y = (attention_mixer if L["type"] == "attention" else latent_attention_mixer)(W, m, h, c, eps, pos)
        if L.get("mlp") is not None:
            y = y + dense_ff(W, p + "mlp.", stream_norm(x, W[p + "norm2"], eps))
        x = x + y
        if cfg.get("token_side"):
            d = cfg["token_side"]["dim"]
            x = x + side_input(x, W["side.embed"][ids, i * d:(i + 1) * d], W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return stream_norm(x, W["final.norm"], eps) @ W["embed"].T


def greedy(cfg, W, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]


# ---- small random checkpoints ----------------------------------------------------------------------------------------
def delta_layer(heads=4, kv_heads=2, dim=8, vdim=12, conv=4, ff=40):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention_layer(heads=4, kv_heads=2, dim=12, rot_dims=8, base=300.0, scale=0.4, ff=40):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": {"base": base, "dims": rot_dims}, "scale": scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent_layer(heads=3, dim=8, rot_dim=6, vdim=10, kv_rank=14, q_rank=9, base=500.0, scale=0.35, window=11, ff=40):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                  "rot": {"base": base, "dims": rot_dim}, "scale": scale, "mask": {"size": window}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def make_config(layers, width=32, vocab=53, eps=1e-5, side=6, loop=None):
    cfg = {"architecture": "Zepilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side:
        cfg["token_side"] = {"dim": side}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def random_model(cfg, seed=0):
    """float64 weights for `cfg`, every one exactly representable in bfloat16: a checkpoint written in bfloat16 holds the same numbers."""
    g = torch.Generator().manual_seed(seed)
    width, W = cfg["width"], {}

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(tuple(shape), generator=g, dtype=F64) * std + mean).to(torch.bfloat16).to(F64)

    lin = lambda o, i: rnd(o, i, std=i ** -0.5)
    W["embed"] = rnd(cfg["vocab"], width)
    if cfg.get("loop"):
        W["loop.step"] = rnd(cfg["loop"]["times"], width, std=0.5)
    d = (cfg.get("token_side") or {}).get("dim", 0)
    if d:
        W["side.embed"] = rnd(cfg["vocab"], d * len(cfg["layers"]))
    for i, L in enumerate(cfg["layers"]):
        p, c = f"l{i}.", L["mixer"]
        m = p + "mix."
        W[p + "norm1"] = rnd(width, std=0.3)
        if L["type"] == "delta":
            H, G, D, V = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                W[m + n], W[m + n + ".conv"] = lin(rows, width), rnd(rows, c["conv"], std=0.5)
            W[m + "b"], W[m + "a"], W[m + "A_log"], W[m + "dt_bias"] = lin(H, width), lin(H, width), rnd(H, std=0.5, mean=-1.5), rnd(H)
            W[m + "g"], W[m + "norm"], W[m + "o"] = lin(H * V, width), rnd(V, std=0.3, mean=1.0), lin(width, H * V)
        elif L["type"] == "attention":
            H, G, D = c["heads"], c["kv_heads"], c["dim"]
            W[m + "q"], W[m + "k"], W[m + "o"] = lin(H * D, width), lin(G * D, width), lin(width, H * D)
        else:
            H, D, R, V, C, Q = (c[n] for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            W[m + "dq"], W[m + "dq.norm"], W[m + "uq"] = lin(Q, width), rnd(Q, std=0.3, mean=1.2), lin(H * (D + R), Q)
            W[m + "dkv"], W[m + "dkv.norm"] = lin(C + R, width), rnd(C, std=0.3, mean=1.2)
            W[m + "uk"], W[m + "uv"], W[m + "o"] = lin(H * D, C), lin(H * V, C), lin(width, H * V)
        if L.get("mlp") is not None:
            ff = L["mlp"]["ff"]
            W[p + "norm2"] = rnd(width, std=0.3)
            for n, o, i_ in (("gate", ff, width), ("up", ff, width), ("down", width, ff)):
                W[p + "mlp." + n], W[p + "mlp." + n + ".b"] = lin(o, i_), rnd(o, std=0.3)
        if d:
            W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"] = lin(d, width), lin(width, d), rnd(width, std=0.2, mean=0.6)
    W["final.norm"] = rnd(width, std=0.3)
    return W
