"""Low-rank (latent) attention as a building block of the slot-pool models.

A token's keys and values of all heads are functions of one normed latent and one rotated key part, and only those are cached
(`LatentKVSpec`).  `load_latent` fuses the checkpoint's tensors, `latent_attention` runs the mixer up to the concatenated heads:

    expanded   (prompts)   per-head keys and values of the step's context go to a dense pool of the step, multi-head attention over it
    latent     (decoding)  the query is carried into the latent space and attends over the cached rows directly

Rotation pairs half a part apart or neighbours, a multiplier on cos and sin, a sliding window, a learned sink and a sigmoid gate per
head are options.  Under a window only the keys that some token of the step sees are expanded.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import _native_seq as nsq
from ._state import LatentKVSpec


def load_latent(get, p: str, what: str, m: dict, freqs: List[float], rot_mult: float = 1.0, interleaved: bool = False, window: int = 0,
                gate: Optional[torch.Tensor] = None, sink: Optional[torch.Tensor] = None, device=None) -> dict:
    """`get(name)`: a tensor of the checkpoint in the compute type; `p`: the mixer's prefix ("l3.mix."); `what`: names the layer in errors."""
    H, D, R, V, C = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    rot = m.get("rot") or {}
    if R and int(rot.get("dims", R)) != R:
        raise ValueError(f"{what}: the rotation covers {rot.get('dims')} dimensions, the rotated part has {R}")
    dq, dkv = get(p + "dq"), get(p + "dkv")
    Q = dq.shape[0]
    if dkv.shape[0] != C + R:
        raise ValueError(f"{what}: the key/value down-projection has {dkv.shape[0]} rows, not kv_rank + rot_dim = {C + R}")
    uk, uv = get(p + "uk"), get(p + "uv")
    parts, rows = [dq, dkv], Q + C + R
    pad = -rows % 8 if gate is None else 0     # rows of whole 16-byte pieces
    if gate is not None:
        parts.append(gate)
    if pad:
        parts.append(torch.zeros(pad, dq.shape[1], dtype=dq.dtype, device=dq.device))
    return dict(heads=H, dim=D, rot_dim=R, vdim=V, kv_rank=C, q_rank=Q, scale=float(m["scale"]), rot_mult=float(rot_mult), interleaved=interleaved, window=int(window),
                freqs=torch.tensor(freqs, dtype=torch.float64, device=device) if R else None,
                # one product of the mixer's input: query latent, key/value latent with the rotated part, head gates
                w_in=torch.cat(parts, 0).contiguous(), offs=(0, Q, Q + C + R), gated=gate is not None,
                cq_norm=get(p + "dq.norm"), ckv_norm=get(p + "dkv.norm"), w_uq=get(p + "uq"),
                w_ukv=torch.cat([uk, uv], 0).contiguous(),             # latents -> plain key parts of all heads, then values
                uk_h=uk.view(H, D, C).contiguous(),                    # per head: carries a query into the latent space
                uv_t=uv.view(H, V, C).transpose(1, 2).contiguous(),    # per head [C, V]: carries a latent result back
                sink=sink, w_o=get(p + "o"), spec=LatentKVSpec(C, R),
                # the latent form's result per head is kv_rank wide: beyond what the decoding kernels hold, only the expanded form runs
                latent_ok=C <= nsq.ATTN_MAX_VDIM)


def _context(batch, step: dict, window: int, device):
    """The step's context tokens (every entry's rows from the first one that some new token sees) as a batch description, the positions
    those begin at (None: all at 0), the new tokens counted from there, and the entries' indices as the dense pool's slots; built once per step and
    window."""
    if "latent_ids" not in step:
        step["latent_ids"] = torch.arange(batch.n_seqs, dtype=torch.int32, device=device)
    lo = [max(0, p0 - window + 1) if window > 0 else 0 for p0 in batch.pos0]
    key = ("latent_ctx", tuple(lo))
    if key not in step:
        if all(p0 == a for p0, a in zip(batch.pos0, lo)):
            ctx = batch
        else:
            ctx = nsq.Batch(batch.slots, lo, [p0 + n - a for p0, n, a in zip(batch.pos0, batch.lens, lo)], device)
        shifted = any(lo)
        new = nsq.Batch(batch.slots, [p0 - a for p0, a in zip(batch.pos0, lo)], batch.lens, device) if shifted else batch
        step[key] = (ctx, ctx.seq_pos0 if shifted else None, new, max(p0 + n - a for p0, n, a in zip(batch.pos0, batch.lens, lo)))
    return step[key] + (step["latent_ids"],)


def latent_attention(h: torch.Tensor, blk: dict, ckv: torch.Tensor, batch, step: dict, eps: float, cap: int, form: Optional[str] = None, expand_min_len: int = 16,
                     impl: int = 0) -> torch.Tensor:
    """[T, H * vdim]: the concatenated heads.  `ckv`: the layer's rows in the slot pool (capacity `cap`); `step`: a dict kept for one step;
    `form` "expanded" / "latent" forces a form (None: steps whose longest entry brings `expand_min_len` tokens expand)."""
    T, dt, dev = h.shape[0], h.dtype, h.device
    H, D, R, V, C, Q = blk["heads"], blk["dim"], blk["rot_dim"], blk["vdim"], blk["kv_rank"], blk["q_rank"]
    window, il, sink = blk["window"], blk["interleaved"], blk["sink"]
    proj = nsq.linear(h, blk["w_in"])
    cq = torch.empty(T, Q, dtype=dt, device=dev)
    nsq.latent_prep(proj, blk["offs"][0], blk["offs"][1], Q, C, R, blk["cq_norm"], blk["ckv_norm"], eps, blk["freqs"], blk["rot_mult"], cq, ckv, batch, interleaved=il)
    q = nsq.linear(cq, blk["w_uq"])                      # [T, H * (D + R)], per head [plain | rotated]
    # a recorded decoding step reads everything that changes from device buffers: only the latent form does
    form = "latent" if torch.cuda.is_current_stream_capturing() else (form or ("expanded" if batch.max_len >= expand_min_len else "latent"))
    if not blk["latent_ok"]:
        form = "expanded"
    mixed = torch.empty(T, H * V, dtype=dt, device=dev)
    if form == "expanded":
        ctx, base, new, most, ids = _context(batch, step, window, dev)
        c_ctx = nsq.latent_gather(ckv, C, ctx)
        kv = nsq.linear(c_ctx, blk["w_ukv"])             # [N, H * D + H * V]
        dense = ((most + 63) // 64) * 64
        kd = torch.empty(batch.n_seqs, H, dense, D + R, dtype=dt, device=dev)
        vd = torch.empty(batch.n_seqs, H, dense, V, dtype=dt, device=dev)
        nsq.latent_expand(kv, ckv, C, R, H, D, V, kd, vd, ctx, seq_base=base)
        nsq.latent_q(q, H, D, R, blk["freqs"], blk["rot_mult"], batch, interleaved=il)
        o = torch.empty(T, H * V, dtype=dt, device=dev) if blk["gated"] else mixed
        nsq.attention(q, kd, vd, o, H, blk["scale"], None, None, sink is not None, new, impl=impl, sink_logit=sink, pool_slot=ids, window=window)
        o3 = o.view(T, H, V)
    else:
        # q'_h = U_k,h^T q_h: [H, T, D] x [H, D, C] into the leading columns of every head; the rotated parts are written beside them
        ql = torch.empty(T, H * (C + R), dtype=dt, device=dev)
        q_lat = ql.view(T, H, C + R)[:, :, :C]
        torch.bmm(q.view(T, H, D + R)[:, :, :D].transpose(0, 1), blk["uk_h"], out=q_lat.transpose(0, 1))
        nsq.latent_q(q, H, D, R, blk["freqs"], blk["rot_mult"], batch, q_lat=q_lat, interleaved=il, out=ql)
        o_lat = torch.empty(T, H * C, dtype=dt, device=dev)
        ws = nsq.attn_workspace(T, H, C, dev) if T <= 32 else None
        nsq.attention(ql, ckv, ckv, o_lat, H, blk["scale"], None, None, sink is not None, batch, impl=impl, max_keys=min(cap, window) if window > 0 else cap,
                      workspace=ws, sink_logit=sink, v_row_stride=C + R, window=window)
        o3 = (torch.empty(T, H, V, dtype=dt, device=dev) if blk["gated"] else mixed.view(T, H, V))
        torch.bmm(o_lat.view(T, H, C).transpose(0, 1), blk["uv_t"], out=o3.transpose(0, 1))
    if blk["gated"]:
        nsq.head_gate(o3, proj[:, blk["offs"][2]:blk["offs"][2] + H], mixed)
    return mixed
