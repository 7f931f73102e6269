"""Zepilix: a decoder-only model of gated-delta-rule layers, full attention and latent attention under a sliding window, whose layers run
their mixer and their feed-forward SIDE BY SIDE on the same stream and then take a gated row of a second, per-layer token embedding; a
span of layers may run several times in a row.

    embedding     token row                                                                                   (`pcs_embed`)
    every layer   x += mixer(n(x, w1)) + ff(n(x, w2)) with n(x, w) = rms(x) * (1 + w): weights are stored around zero and the 1 is added in 32-bit
    side input    e = this layer's part of the token's row in a second table; g = gelu(W_gate x) * e; x += rms(W_proj g) * w
                  (prompts: two products around `pcs_side_gate`, the sums and both norms of the next layer in `pcs_add_layer_norm`;
                  a few tokens: all of it is one launch, `pcs_side_boundary`)
    loop          layers [start, stop) run `times` times in a row on the same weights; every RUN of a layer owns a state.  Before a pass
                  but the first the embedding output joins the stream again, and every pass adds a vector of its own: both ride
                  in the launch that forms the pass's first norms
    delta         the gated delta rule with ONE decay per head, formed in 32-bit inside the recurrence; q, k, v through a short convolution with
                  silu, q and k unit vectors; per-head norm and a silu gate
                                                            (`pcs_short_conv`, `pcs_delta_scan` / `pcs_delta_chunk_*`, `pcs_head_norm_gate`)
    attention     grouped heads whose values are the keys as projected; rotation of neighbouring pairs, queries and keys of unit root mean
                  square (a turn keeps a head's root mean square, so the norm is taken before it)             (`pcs_rope_kv_prep`, `pcs_attn`)
    latent_attention   as in model/_latent.py: neighbouring pairs turn, a sliding window, no gate
    feed-forward  W_down(silu(W_gate h + b) * (W_up h + b)) + b                                               (`pcs_glu_mul`)
    output        the norm, then the embedding table as the head

Sizes, the order of layers and every constant that can differ between models come from config.json; tensors are named l<i>.norm1,
l<i>.mix.q.conv, l<i>.mlp.gate.b, l<i>.side.proj, loop.step, ... in the checkpoint.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List, Optional

import torch

from .. import _native_seq as nsq
from .. import weights as wio
from ._latent import latent_attention, load_latent
from ._seqbase import SlotPoolCausalLM
from ._state import ConvTailSpec, DecayStateSpec, KVSpec
from .tevilix import divided_frequencies, layer_runs
from .zovolorn import UNIT_VECTOR_EPS

NORM_WEIGHT_OFFSET = 1.0   # the layers' norm weights are stored around zero
ROW_ALIGN = 8              # fused projections are padded with zero rows to a multiple of this
BRANCH_MAX_TOKENS = 64     # steps of at most this many tokens run mixer and feed-forward side by side on the device too
MIXERS = ("delta", "attention", "latent_attention")


class ZepilixConfig:
    """config.json of the design: {"architecture", "vocab", "width", "norm": {"eps"}, "token_side": {"dim"}, "loop": {"start", "stop", "times"},
    "layers": [{"type": "delta" | "attention" | "latent_attention", "mixer": {...}, "mlp": {"kind": "dense", "ff"} | null}]}."""

    def __init__(self, d: dict):
        self.raw = d
        self.architecture = d.get("architecture", "Zepilix")
        self.vocab_size = int(d["vocab"])
        self.width = int(d["width"])
        self.eps = float(d["norm"]["eps"])
        self.side_dim = int((d.get("token_side") or {}).get("dim", 0))
        self.layers = []
        for i, layer in enumerate(d["layers"]):
            kind = layer["type"]
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            self.layers.append({"type": kind, "mixer": dict(layer["mixer"]), "mlp": dict(mlp) if mlp is not None else None})
        self.num_hidden_layers = len(self.layers)
        self.loop = dict(d["loop"]) if d.get("loop") else None
        self.runs = layer_runs(len(self.layers), self.loop)
        # run index -> number of the pass that begins with it
        self.passes: Dict[int, int] = {}
        if self.loop:
            a = int(self.loop.get("start", 0))
            span = int(self.loop.get("stop", 0)) - a
            if span > 0:
                self.passes = {a + t * span: t for t in range(int(self.loop.get("times", 1)))}

    @classmethod
    def from_dir(cls, path: str) -> "ZepilixConfig":
        with open(os.path.join(path, "config.json")) as fh:
            return cls(json.load(fh))


def _rotation(i: int, rot: dict, dim: int):
    rd = int(rot.get("dims", 0))
    if rd % 2 or rd > dim:
        raise ValueError(f"layer {i}: {rd} rotated coordinates do not fit {dim}")
    return rd, divided_frequencies(rd, float(rot.get("base", 10000.0)))


class ZepilixForCausalLM(SlotPoolCausalLM):
    def __init__(self, config: ZepilixConfig, tensors: Dict[str, torch.Tensor], device="cuda", dtype=torch.bfloat16,
                 max_tokens: Optional[int] = None):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Zepilix computes in bfloat16 or float32")
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
        self.loop_step = get("loop.step") if config.passes else None
        if config.passes and tuple(self.loop_step.shape) != (len(config.passes), self.width):
            raise ValueError(f"loop.step must be [times, width] = [{len(config.passes)}, {self.width}]")
        S = config.side_dim
        self.side_table = get("side.embed") if S else None
        if S and self.side_table.shape[1] != S * len(config.layers):
            raise ValueError(f"side.embed has {self.side_table.shape[1]} columns, not {S} for each of {len(config.layers)} layers")
        self.blocks: List[dict] = []
        for i, layer in enumerate(config.layers):
            p, m = f"l{i}.", layer["mixer"]
            blk = {"type": layer["type"], "norm1": get(p + "norm1")}
            if layer["type"] == "latent_attention":
                R, rot = int(m["rot_dim"]), m.get("rot") or {}
                freqs = _rotation(i, dict(rot, dims=R), R)[1]
                blk.update(load_latent(get, p + "mix.", f"layer {i}", m, freqs, interleaved=True, window=int((m.get("mask") or {}).get("size", 0)), device=dev))
            else:
                H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
                G = int(m.get("kv_heads", H))
                if H % G:
                    raise ValueError(f"layer {i}: {H} heads do not divide into {G} key/value heads")
                if layer["type"] == "attention":
                    if V != D:
                        raise ValueError(f"layer {i}: values that are the keys have the keys' size ({D}, not {V})")
                    rd, freqs = _rotation(i, m.get("rot") or {}, D)
                    w_in, offs = fuse(get(p + "mix.q"), get(p + "mix.k"))
                    blk.update(heads=H, kv_heads=G, dim=D, scale=float(m["scale"]), rot_dims=rd, offs=offs, w_in=w_in, w_o=get(p + "mix.o"),
                               freqs=torch.tensor(freqs, dtype=torch.float64, device=dev) if rd else None, unit=torch.ones(D, dtype=dtype, device=dev), spec=KVSpec(G, D, D))
                else:
                    w_in, offs = fuse(*(get(p + "mix." + n) for n in ("q", "k", "v", "g", "b", "a")))
                    conv = torch.cat([get(p + f"mix.{n}.conv").t() for n in ("q", "k", "v")], 1).contiguous()   # [taps, channels]
                    if int(m.get("conv", conv.shape[0])) != conv.shape[0]:
                        raise ValueError(f"layer {i}: the short convolution has {conv.shape[0]} taps in the checkpoint, {m['conv']} in the configuration")
                    blk.update(heads=H, kv_heads=G, dim=D, vdim=V, w_in=w_in, conv=conv, gate=(offs[3], offs[4]), b=(offs[4], offs[4] + H), a=(offs[5], offs[5] + H),
                               dt_bias=f32(p + "mix.dt_bias"), rate=torch.exp(f32(p + "mix.A_log")), mix_norm=get(p + "mix.norm"), w_o=get(p + "mix.o"),
                               spec=(DecayStateSpec(H, D, V),) + ((ConvTailSpec(conv.shape[0], conv.shape[1], "conv_tail"),) if conv.shape[0] > 1 else ()))
            blk["mlp"] = layer["mlp"] is not None
            if blk["mlp"]:
                gate, up = get(p + "mlp.gate"), get(p + "mlp.up")
                blk.update(norm2=get(p + "norm2"), ff=gate.shape[0], w_gu=torch.cat([gate, up], 0).contiguous(),
                           b_gu=torch.cat([get(p + "mlp.gate.b"), get(p + "mlp.up.b")]).contiguous(), w_down=get(p + "mlp.down"), b_down=get(p + "mlp.down.b"))
            if S:
                blk.update(side_gate=get(p + "side.gate"), side_proj=get(p + "side.proj"), side_norm=get(p + "side.norm"), side_col=i * S)
            self.blocks.append(blk)
        self.runs, self.passes = list(config.runs), dict(config.passes)
        # bfloat16 products accumulate in 32-bit all the way (no reduced-precision split-K sums); float32 stays true float32
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cudnn.allow_tf32 = False
        self.attn_impl = 0
        self.scan_impl = 0           # delta rule: 0 by step, 1 / 2 token by token, 3 in chunks
        self.latent_form = None      # None: by step (prompts expanded, decoding in the latent space); "expanded" / "latent" force one
        self.expand_min_len = 16     # steps whose longest entry brings at least this many tokens attend over expanded keys
        self.fused_side = None       # a layer's end in one launch: None: for a few tokens; True / False force it
        self.branches = None         # mixer and feed-forward on two streams: None: for a few tokens; True / False force it
        self._branch_stream = None
        self._init_runtime(dev, max_tokens)
        if not all(b.get("latent_ok", True) for b in self.blocks):
            self.use_cuda_graphs = False   # the expanded form describes the step's context on the host: it is not recorded

    def state_specs(self):
        """One state per layer RUN: a layer inside the loop keeps as many as it has passes."""
        return [self.blocks[i]["spec"] for i in self.runs]

    @classmethod
    def from_pretrained(cls, path: str, device="cuda", dtype=torch.bfloat16, max_tokens: Optional[int] = None, **_):
        """`path`: a folder with config.json and model.safetensors."""
        cfg = ZepilixConfig.from_dir(path)
        tensors = wio.load_file(os.path.join(path, "model.safetensors"), device=device)
        return cls(cfg, tensors, device=device, dtype=dtype, max_tokens=max_tokens)

    # ---- the sublayers ------------------------------------------------------------------------------------------
    def _delta(self, h, blk, st, batch):
        T, dt, dev = h.shape[0], self.compute_dtype, self._device
        H, G, D, V = blk["heads"], blk["kv_heads"], blk["dim"], blk["vdim"]
        proj = nsq.linear(h, blk["w_in"])                 # q | k | v | gate | step sizes | decays
        qk, v = nsq.short_conv(proj, 0, G, D, H * V, blk["conv"], st.get("conv_tail"), D ** -0.5, UNIT_VECTOR_EPS, batch)
        mixed = torch.empty(T, H * V, dtype=dt, device=dev)
        nsq.delta_scan(qk, v, None, proj[:, slice(*blk["b"])], G, st["s"], blk["mix_norm"], proj[:, slice(*blk["gate"])], mixed, self.eps, batch, impl=self.scan_impl,
                       head_decay=(proj[:, slice(*blk["a"])], blk["dt_bias"], blk["rate"]), gate_silu=True)
        return nsq.linear(mixed, blk["w_o"])

    def _attention(self, h, blk, st, batch):
        T, dt, dev = h.shape[0], self.compute_dtype, self._device
        H, G, D, offs = blk["heads"], blk["kv_heads"], blk["dim"], blk["offs"]
        proj = nsq.linear(h, blk["w_in"])                 # q | k; the value rows are the key columns as projected
        q = torch.empty(T, H * D, dtype=dt, device=dev)
        nsq.rope_kv_prep(proj, (offs[0], offs[1], offs[1]), H, G, D, D, blk["freqs"], blk["rot_dims"], True, False, self.eps, q, st["k"], st["v"], batch,
                         q_norm_w=blk["unit"], k_norm_w=blk["unit"])
        mixed = torch.empty(T, H * D, dtype=dt, device=dev)
        # few tokens (decoding): the keys are split over more blocks; the bound is the pool's capacity, so that a replayed graph
        # stays valid while the sequences grow
        ws = nsq.attn_workspace(T, H, D, dev) if T <= 16 else None
        nsq.attention(q, st["k"], st["v"], mixed, H, blk["scale"], None, None, False, batch, impl=self.attn_impl, max_keys=self.pool.cap, workspace=ws)
        return nsq.linear(mixed, blk["w_o"])

    def _mixer(self, h, blk, st, batch, step):
        if blk["type"] == "delta":
            return self._delta(h, blk, st, batch)
        if blk["type"] == "attention":
            return self._attention(h, blk, st, batch)
        mixed = latent_attention(h, blk, st["ckv"], batch, step, self.eps, self.pool.cap, form=self.latent_form, expand_min_len=self.expand_min_len, impl=self.attn_impl)
        return nsq.linear(mixed, blk["w_o"])

    def _feed_forward(self, h, blk):
        gu = nsq.linear(h, blk["w_gu"], blk["b_gu"])
        return nsq.linear(nsq.glu_mul(gu, blk["ff"]), blk["w_down"], blk["b_down"])

    # ---- the layers over one batch ------------------------------------------------------------------------------
    def _layers(self, ids: torch.Tensor, batch, rows: Optional[torch.Tensor]) -> torch.Tensor:
        T, W, dt, dev, eps, off = ids.shape[0], self.width, self.compute_dtype, self._device, self.eps, NORM_WEIGHT_OFFSET
        x = torch.empty(T, W, dtype=torch.float32, device=dev)     # the residual stream, 32-bit, updated in place
        h1 = torch.empty(T, W, dtype=dt, device=dev)               # the mixer's input of the next layer run
        h2 = torch.empty(T, W, dtype=dt, device=dev)               # its feed-forward's input
        nsq.embed(self.embed, ids, x, 1.0)
        x0 = None                                                  # the embedding output, kept where a later pass adds it again
        if len(self.passes) > 1:
            x0 = torch.empty(T, W, dtype=torch.float32, device=dev)
            nsq.embed(self.embed, ids, x0, 1.0)
        step: dict = {}

        # every token's logits are asked for (decoding): the last layer's end forms the output norm of all rows
        last = {"norm1": self.final_norm} if batch.wants_all else None

        def entering(r: int) -> list:
            """What joins the stream before run r."""
            t = self.passes.get(r)
            if t is None:
                return []
            return ([(x0, 1.0)] if t > 0 else []) + [(self.loop_step[t].expand(T, W), 1.0)]

        def boundary(r: int, results: list, normed: Optional[torch.Tensor] = None) -> None:
            """Add the results of run r - 1 (the first one through its own norm where `normed` is given) and what enters before run r, and form
            run r's inputs."""
            nxt = self.blocks[self.runs[r]] if r < len(self.runs) else last
            addends = results + entering(r)
            if results and (self.layer_trace is not None or len(addends) > 3):
                nsq.add_rms_norm(x, results, eps, y_norm_w=normed)
                addends, normed = entering(r), None
                if self.layer_trace is not None:
                    self.layer_trace.append(x.clone())
            if nxt is not None or addends:
                nsq.add_rms_norm(x, addends, eps, nxt["norm1"] if nxt else None, h1, nxt.get("norm2") if nxt else None, h2, w_offset=off, y_norm_w=normed)

        def side_end(r: int, blk: dict, ys: list) -> None:
            """A layer's end for a few tokens in one launch: its sublayers' sum, its side input, what enters before run r and run r's inputs."""
            nxt = self.blocks[self.runs[r]] if r < len(self.runs) else last
            t = self.passes.get(r)
            nsq.side_boundary(x, [y for y, _ in ys], ids, self.side_table, blk["side_col"], blk["side_gate"], blk["side_proj"], blk["side_norm"], eps,
                              x0=x0 if t else None, step=self.loop_step[t] if t is not None else None, w1=nxt["norm1"] if nxt else None, h1=h1,
                              w2=nxt.get("norm2") if nxt else None, h2=h2, w_offset=off)

        fused_side = self.fused_side if self.fused_side is not None else T <= nsq.SIDE_BOUNDARY_MAX_TOKENS
        boundary(0, [])
        # the sublayers read the same stream: where a step is bound by its launches the feed-forward runs on a stream of its own
        main, branch = torch.cuda.current_stream(), None
        if self.branches if self.branches is not None else T <= BRANCH_MAX_TOKENS:
            branch = self._branch_stream = self._branch_stream or torch.cuda.Stream(device=dev)
        for r, li in enumerate(self.runs):
            blk, st = self.blocks[li], self.pool.layers[r]
            ff = None
            if blk["mlp"] and branch is not None:
                branch.wait_stream(main)
                with torch.cuda.stream(branch):
                    ff = self._feed_forward(h2, blk)
            ys = [(self._mixer(h1, blk, st, batch, step), 1.0)]
            if ff is not None:
                main.wait_stream(branch)    # the branch starts again only after the launch that reads `ff`, so its memory is free by then
            elif blk["mlp"]:
                ff = self._feed_forward(h2, blk)
            if ff is not None:
                ys.append((ff, 1.0))
            if self.side_table is None:
                boundary(r + 1, ys)
                continue
            if fused_side and self.layer_trace is None:
                side_end(r + 1, blk, ys)
                continue
            xc = torch.empty(T, W, dtype=dt, device=dev)
            nsq.add_rms_norm(x, ys, eps, copy=xc)
            g = nsq.side_gate(nsq.linear(xc, blk["side_gate"]), self.side_table, blk["side_col"], ids)
            boundary(r + 1, [(nsq.linear(g, blk["side_proj"]), 1.0)], blk["side_norm"])
        if rows is None or rows.numel() == 0:
            return torch.zeros(0, self.vocab_size, dtype=torch.float32, device=dev)
        if last is None:
            h1 = torch.empty(rows.numel(), W, dtype=dt, device=dev)
            nsq.add_rms_norm(x, [], eps, self.final_norm, h1, rows=rows, w_offset=off)     # only the wanted rows go on
        return nsq.linear(h1, self.embed).float()
