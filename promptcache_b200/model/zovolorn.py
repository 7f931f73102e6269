"""Zovolorn: a decoder-only model of full attention layers and layers that run chunked attention beside a gated delta rule, with norms
on the sublayers' RESULTS only and a short causal convolution in front of every sublayer.

    embedding     token row times a scale + a row of a hashed (previous token, token) table          (`pcs_embed_bigram`)
    every layer   x += gn(mixer(c1(x)), w1);  x += gn(ff(c2(x)), w2)   with gn an RMS norm in equal groups of channels and
                  c(x) = x + a causal convolution of x over time; the residual sum and the next sublayer's convolution are one
                  launch, and the stream alternates between two buffers because a token's convolution needs its predecessors'
                  new rows                                                                             (`pcs_group_norm_conv`)
    attention     grouped heads; q and k normed over the WHOLE projection, then the leading coordinates turn by position in
                  neighbouring pairs (`pcs_rope_kv_prep`); a learned sink term per head; a sigmoid gate per head (`pcs_attn`)
    parallel      two mixers on the same input, added with two constants:
                  left   attention whose values are the keys before their norm; head norms, no rotation, scores times a number per
                         head plus a learned bias per bucket of the distance (tabulated by distance at load); a token sees its own
                         chunk of positions only                                          (`pcs_rope_kv_prep`, `pcs_attn`)
                  right  the gated delta rule: q, k, v through a short convolution with silu, q and k unit vectors, a decay per key
                         channel, a step size per head, per-head norm and a low-rank sigmoid gate
                                          (`pcs_short_conv`, `pcs_gla_decay`, `pcs_delta_scan` / `pcs_delta_chunk_*`, `pcs_head_norm_gate`;
                         decoding takes the inputs in one launch, `pcs_delta_inputs`)
                  both write their columns of ONE matrix, already times their constants, so one product with the two output
                  projections side by side adds them in 32-bit
    feed-forward  W_down(gelu(W_gate h + b) * (W_up h + b)) + b with the tanh form of gelu                    (`pcs_glu_mul`)
    output        grouped norm, the embedding table as the head, logits capped by cap * tanh(z / cap)        (`pcs_soft_cap`)

K/V rows, delta states and the convolutions' last inputs live in the slot pool; the previous token is part of a sequence's handle.
Sizes, the order of layers and every constant that can differ between models come from config.json; tensors are named l<i>.norm1,
l<i>.canon1, l<i>.mix.q, l<i>.mix.left.rel, l<i>.mix.right.q.conv, l<i>.mlp.gate, ... in the checkpoint.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import torch

from .. import _native_seq as nsq
from .. import weights as wio
from ._seqbase import SlotPoolCausalLM
from ._state import ConvTailSpec, DecayStateSpec, KVSpec

UNIT_VECTOR_EPS = 1e-6     # added under the root of the delta rule's unit vectors
ROW_ALIGN = 8              # fused projections are padded with zero rows to a multiple of this


def distance_bucket(n: int, n_buckets: int, far: int) -> int:
    """Bucket of a distance n >= 0: one bucket per distance below half of the buckets, then buckets of equal width in ln n that reach
    the last one at `far`."""
    half = n_buckets // 2
    if n < half:
        return n
    if half < 1 or far <= half:
        return n_buckets - 1
    # (the nudge keeps a distance that sits exactly on a border on its upper side whatever the logarithms' last bits are)
    return min(n_buckets - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (n_buckets - half) + 1e-9))


def distance_bias_table(rel: torch.Tensor, far: int, max_distance: Optional[int] = None) -> torch.Tensor:
    """float32 [heads, L] with column n the bias at distance n, from rel [buckets, heads]; distances of L and more have the last column's.
    `max_distance`: the largest distance any query sees (a chunk's size minus one), if bounded."""
    last = far if far > rel.shape[0] // 2 else rel.shape[0]     # from here on every distance is in the last bucket
    if max_distance is not None:
        last = min(last, max(max_distance, 0))
    idx = torch.tensor([distance_bucket(n, rel.shape[0], far) for n in range(last + 1)], device=rel.device)
    return rel.float()[idx].t().contiguous()


class ZovolornConfig:
    """config.json of the design: {"architecture", "vocab", "width", "embedding": {"scale", "bigram": {"buckets", "mul_prev", "mul_cur"}},
    "norm": {"eps", "groups"}, "canon": {"taps"}, "logit_softcap", "layers": [{"type": "attention" | "parallel", "mixer": {...},
    "mlp": {"kind": "dense", "ff"} | null}]}."""

    def __init__(self, d: dict):
        self.raw = d
        self.architecture = d.get("architecture", "Zovolorn")
        self.vocab_size = int(d["vocab"])
        self.width = int(d["width"])
        emb = d.get("embedding") or {}
        self.embedding_scale = float(emb.get("scale", 1.0))
        self.bigram = emb.get("bigram")
        self.eps = float(d["norm"]["eps"])
        self.groups = int(d["norm"].get("groups", 1))
        if self.groups < 1 or self.width % self.groups:
            raise ValueError(f"{self.groups} norm groups do not divide the width {self.width}")
        self.taps = int((d.get("canon") or {}).get("taps", 0))
        self.softcap = float(d.get("logit_softcap") or 0.0)
        self.layers = []
        for i, layer in enumerate(d["layers"]):
            kind = layer["type"]
            if kind not in ("attention", "parallel"):
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            self.layers.append({"type": kind, "mixer": dict(layer["mixer"]), "mlp": dict(mlp) if mlp is not None else None})
        self.num_hidden_layers = len(self.layers)

    @classmethod
    def from_dir(cls, path: str) -> "ZovolornConfig":
        with open(os.path.join(path, "config.json")) as fh:
            return cls(json.load(fh))


def _grouped(i: int, c: dict):
    H = int(c["heads"])
    G = int(c.get("kv_heads", H))
    if H % G:
        raise ValueError(f"layer {i}: {H} heads do not divide into {G} key/value heads")
    return H, G, int(c["dim"]), int(c["vdim"])


class ZovolornForCausalLM(SlotPoolCausalLM):
    def __init__(self, config: ZovolornConfig, tensors: Dict[str, torch.Tensor], device="cuda", dtype=torch.bfloat16,
                 max_tokens: Optional[int] = None):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Zovolorn computes in bfloat16 or float32")
        self.config, self.compute_dtype = config, dtype
        self.vocab_size, self.width, self.eps = config.vocab_size, config.width, config.eps
        dev = torch.device(device)

        def raw(name):
            if name not in tensors:
                raise KeyError(f"the checkpoint has no tensor {name!r}")
            return tensors[name]

        def get(name):
            return raw(name).to(dev, dtype).contiguous()

        def f32(name):
            return raw(name).to(dev, torch.float32).reshape(-1).contiguous()

        def taps_first(name):   # [channels, taps] -> [taps, channels]: a tap's weights of neighbouring channels are one load
            return get(name).t().contiguous()

        def input_conv(name):
            if not config.taps:
                return None
            w = taps_first(name)
            if w.shape[0] != config.taps:
                raise ValueError(f"{name} has {w.shape[0]} taps in the checkpoint, {config.taps} in the configuration")
            return w

        def fuse(*parts):
            """Rows of several projections of the same input as one matrix, padded with zero rows, and every part's first row."""
            offs, n = [], 0
            for p in parts:
                offs.append(n)
                n += p.shape[0]
            pad = -n % ROW_ALIGN
            if pad:
                parts = parts + (torch.zeros(pad, parts[0].shape[1], dtype=dtype, device=dev),)
            return torch.cat(parts, 0).contiguous(), offs

        self.embed, self.final_norm = get("embed"), get("final.norm")
        self.pair_table = get("bigram") if config.bigram else None
        if config.bigram and self.pair_table.shape[0] != int(config.bigram["buckets"]) + 1:
            raise ValueError("the bigram table must have buckets + 1 rows")
        self.blocks: List[dict] = []
        for i, layer in enumerate(config.layers):
            p, m = f"l{i}.", layer["mixer"]
            blk = {"type": layer["type"], "norm1": get(p + "norm1"), "canon1": input_conv(p + "canon1")}
            if layer["type"] == "attention":
                H, G, D, V = _grouped(i, m)
                rot = m.get("rot") or {}
                rd = int(rot.get("dims", 0))
                if rd % 2 or rd > D:
                    raise ValueError(f"layer {i}: {rd} rotated coordinates do not fit a head of {D}")
                w_in, offs = fuse(get(p + "mix.q"), get(p + "mix.k"), get(p + "mix.v"), get(p + "mix.g"))
                freqs = [float(rot.get("base", 10000.0)) ** (-2.0 * j / rd) for j in range(rd // 2)]
                blk.update(heads=H, kv_heads=G, dim=D, vdim=V, scale=float(m.get("scale", D ** -0.5)), rot_dims=rd,
                           freqs=torch.tensor(freqs, dtype=torch.float64, device=dev) if rd else None, w_in=w_in, offs=offs,
                           q_norm=get(p + "mix.q.norm"), k_norm=get(p + "mix.k.norm"), sink=f32(p + "mix.sink"), w_o=get(p + "mix.o"), spec=[KVSpec(G, D, V)])
            else:
                a, r, pl, pr = m["left"], m["right"], p + "mix.left.", p + "mix.right."
                H, G, D, V = _grouped(i, a)
                if V != D:
                    raise ValueError(f"layer {i}: values that are the keys have the keys' size ({D}, not {V})")
                Hr, Gr, Dr, Vr = _grouped(i, r)
                chunk = int((a.get("mask") or {}).get("size", 0))
                w_in, offs = fuse(get(pl + "q"), get(pl + "k"), get(pr + "q"), get(pr + "k"), get(pr + "v"), get(pr + "g1"), get(pr + "a1"), get(pr + "b"))
                conv = torch.cat([taps_first(pr + n + ".conv") for n in ("q", "k", "v")], 1).contiguous()
                if int(r.get("conv", conv.shape[0])) != conv.shape[0]:
                    raise ValueError(f"layer {i}: the short convolution has {conv.shape[0]} taps in the checkpoint, {r['conv']} in the configuration")
                rel = raw(pl + "rel").to(dev)
                if rel.shape[1] != H:
                    raise ValueError(f"layer {i}: the distance bias has {rel.shape[1]} heads, not {H}")
                blk.update(heads=H, kv_heads=G, dim=D, scale=float(a.get("scale", D ** -0.5)), chunk=chunk, w_in=w_in, q_norm=get(pl + "q.norm"),
                           k_norm=get(pl + "k.norm"), temp=f32(pl + "temp"), bias=distance_bias_table(rel, int(a["bias_max"]), chunk - 1 if chunk > 0 else None),
                           offs=(offs[0], offs[1], offs[1]), r_heads=Hr, r_kv_heads=Gr, r_dim=Dr, r_vdim=Vr, conv=conv, conv_off=offs[2],
                           g1=(offs[5], offs[6]), a1=(offs[6], offs[7]), b=(offs[7], offs[7] + Hr), w_g2=get(pr + "g2"), w_a2=get(pr + "a2"), dt_bias=f32(pr + "dt_bias"),
                           rate=torch.exp(f32(pr + "A_log")), r_norm=get(pr + "norm"), left_scale=float(m["left_scale"]), right_scale=float(m["right_scale"]),
                           # one product adds the two branches: their results side by side, their output projections side by side
                           w_o=torch.cat([get(pl + "o"), get(pr + "o")], 1).contiguous(),
                           spec=[KVSpec(G, D, D), DecayStateSpec(Hr, Dr, Vr)] + ([ConvTailSpec(conv.shape[0], conv.shape[1], "conv_tail")] if conv.shape[0] > 1 else []))
            f = layer["mlp"]
            blk["mlp"] = f is not None
            tails = ["tail1"]
            if f is not None:
                tails.append("tail2")
                gate, up = get(p + "mlp.gate"), get(p + "mlp.up")
                blk.update(norm2=get(p + "norm2"), canon2=input_conv(p + "canon2"), ff=gate.shape[0],
                           w_gu=torch.cat([gate, up], 0).contiguous(), b_gu=torch.cat([get(p + "mlp.gate.b"), get(p + "mlp.up.b")]).contiguous(),
                           w_down=get(p + "mlp.down"), b_down=get(p + "mlp.down.b"))
            if config.taps > 1:
                blk["spec"] += [ConvTailSpec(config.taps, self.width, n) for n in tails]
            self.blocks.append(blk)
        # bfloat16 products accumulate in 32-bit all the way (no reduced-precision split-K sums); float32 stays true float32
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cudnn.allow_tf32 = False
        self.attn_impl = 0
        self.scan_impl = 0     # delta rule: 0 by step, 1 / 2 token by token, 3 in chunks
        self._init_runtime(dev, max_tokens)

    def state_specs(self):
        return [tuple(b["spec"]) for b in self.blocks]

    @classmethod
    def from_pretrained(cls, path: str, device="cuda", dtype=torch.bfloat16, max_tokens: Optional[int] = None, **_):
        """`path`: a folder with config.json and model.safetensors."""
        cfg = ZovolornConfig.from_dir(path)
        tensors = wio.load_file(os.path.join(path, "model.safetensors"), device=device)
        return cls(cfg, tensors, device=device, dtype=dtype, max_tokens=max_tokens)

    # ---- the mixers ---------------------------------------------------------------------------------------------
    def _attention(self, h, blk, st, batch):
        T, dt, dev = h.shape[0], self.compute_dtype, self._device
        H, G, D, V, offs = blk["heads"], blk["kv_heads"], blk["dim"], blk["vdim"], blk["offs"]
        proj = nsq.linear(h, blk["w_in"])                 # q | k | v | head gates
        q = torch.empty(T, H * D, dtype=dt, device=dev)
        nsq.rope_kv_prep(proj, offs[:3], H, G, D, V, blk["freqs"], blk["rot_dims"], True, False, self.eps, q, st["k"], st["v"], batch,
                         q_norm_w=blk["q_norm"], k_norm_w=blk["k_norm"], norm_whole=True)
        mixed = torch.empty(T, H * V, dtype=dt, device=dev)
        # few tokens (decoding): the keys are split over more blocks; the bound is the pool's capacity, so that a replayed graph
        # stays valid while the sequences grow
        ws = nsq.attn_workspace(T, H, V, dev) if T <= 16 else None
        nsq.attention(q, st["k"], st["v"], mixed, H, blk["scale"], None, None, True, batch, impl=self.attn_impl, max_keys=self.pool.cap, workspace=ws,
                      sink_logit=blk["sink"], head_gate=proj[:, offs[3]:offs[3] + H])
        return nsq.linear(mixed, blk["w_o"])

    def _parallel(self, h, blk, st, batch):
        T, dt, dev = h.shape[0], self.compute_dtype, self._device
        H, G, D, Hr, Gr, Dr, Vr = (blk[k] for k in ("heads", "kv_heads", "dim", "r_heads", "r_kv_heads", "r_dim", "r_vdim"))
        proj = nsq.linear(h, blk["w_in"])                 # left q | k, right q | k | v | gate | decay | step size (low-rank inputs)
        mixed = torch.empty(T, H * D + Hr * Vr, dtype=dt, device=dev)
        q = torch.empty(T, H * D, dtype=dt, device=dev)
        # the value rows are the key columns as projected: the norm only touches the key rows
        nsq.rope_kv_prep(proj, blk["offs"], H, G, D, D, None, 0, True, False, self.eps, q, st["k"], st["v"], batch, q_norm_w=blk["q_norm"], k_norm_w=blk["k_norm"])
        seen = min(self.pool.cap, blk["chunk"]) if blk["chunk"] > 0 else self.pool.cap
        ws = nsq.attn_workspace(T, H, D, dev) if T <= 16 else None
        nsq.attention(q, st["k"], st["v"], mixed[:, :H * D], H, blk["scale"], None, None, False, batch, impl=self.attn_impl, max_keys=seen, workspace=ws,
                      head_scale=blk["temp"], bias_table=blk["bias"], chunk=blk["chunk"], out_scale=blk["left_scale"])
        qk, v, decay, gate = nsq.delta_inputs(proj, blk["conv_off"], Gr, Hr, Dr, Vr, blk["conv"], st.get("conv_tail"), Dr ** -0.5, UNIT_VECTOR_EPS, blk["a1"],
                                              blk["w_a2"], blk["dt_bias"], blk["rate"], blk["g1"], blk["w_g2"], batch,
                                              expo=not nsq.delta_takes_chunks(batch, Dr, self.scan_impl))
        nsq.delta_scan(qk, v, decay, proj[:, slice(*blk["b"])], Gr, st["s"], blk["r_norm"], gate, mixed[:, H * D:], self.eps, batch, out_scale=blk["right_scale"],
                       impl=self.scan_impl)
        return nsq.linear(mixed, blk["w_o"])

    def _feed_forward(self, h, blk):
        gu = nsq.linear(h, blk["w_gu"], blk["b_gu"])
        return nsq.linear(nsq.glu_mul(gu, blk["ff"], (nsq.GLU_GELU_TANH, 0.0, 0.0)), blk["w_down"], blk["b_down"])

    # ---- the layers over one batch ------------------------------------------------------------------------------
    def _layers(self, ids: torch.Tensor, batch, rows: Optional[torch.Tensor]) -> torch.Tensor:
        T, W, dt, dev, eps, groups = ids.shape[0], self.width, self.compute_dtype, self._device, self.eps, self.config.groups
        x, other = torch.empty(T, W, dtype=torch.float32, device=dev), torch.empty(T, W, dtype=torch.float32, device=dev)   # the 32-bit stream, old and new
        h = torch.empty(T, W, dtype=dt, device=dev)                # the next sublayer's input
        if self.pair_table is not None:
            bg = self.config.bigram
            nsq.embed_bigram(self.embed, self.pair_table, ids, batch.prev_ids, x, int(bg["buckets"]), int(bg["mul_prev"]), int(bg["mul_cur"]), scale=self.config.embedding_scale)
        else:
            nsq.embed(self.embed, ids, x, self.config.embedding_scale)
        pending = None             # the latest sublayer's result and its norm weight, not yet added to the stream

        def boundary(conv, tail):
            """Add the pending result and form the next sublayer's input."""
            nonlocal x, other
            if conv is None:       # no convolution in this model: the input is the stream itself
                if pending is not None:
                    nsq.group_norm_conv(x, groups, eps, dt, x_out=x, y=pending[0], w=pending[1])
                h.copy_(x)
                return
            nsq.group_norm_conv(x, groups, eps, dt, x_out=other if pending is not None else None, y=pending[0] if pending is not None else None,
                                w=pending[1] if pending is not None else None, conv_w=conv, tail=tail, h_out=h, batch=batch)
            if pending is not None:
                x, other = other, x

        for i, blk in enumerate(self.blocks):
            st = self.pool.layers[i]
            boundary(blk["canon1"], st.get("tail1"))
            if self.layer_trace is not None and i:
                self.layer_trace.append(x.clone())
            y = self._attention(h, blk, st, batch) if blk["type"] == "attention" else self._parallel(h, blk, st, batch)
            pending = (y, blk["norm1"])
            if blk["mlp"]:
                boundary(blk["canon2"], st.get("tail2"))
                pending = (self._feed_forward(h, blk), blk["norm2"])
        y, w = pending if pending is not None else (None, None)
        if self.layer_trace is not None and y is not None:
            nsq.group_norm_conv(x, groups, eps, dt, x_out=other, y=y, w=w)
            self.layer_trace.append(other.clone())
        if rows is None or rows.numel() == 0:
            return torch.zeros(0, self.vocab_size, dtype=torch.float32, device=dev)
        hw = torch.empty(rows.numel(), W, dtype=dt, device=dev)
        nsq.group_norm_conv(x, groups, eps, dt, y=y, w=w, next_w=self.final_norm, h_out=hw, rows=rows)   # only the wanted rows go on
        return nsq.soft_cap(nsq.linear(hw, self.embed), self.config.softcap)
