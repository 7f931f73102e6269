"""The Zovolorn design on the GPU against the float64 oracle (tests/zovolorn_oracle.py): each mechanism alone through the kernels'
bindings, then whole models through the step function, the batch engine, the generation engine and bin/trace_run."""
import json
import os
import subprocess

import pytest
import torch

from tests import zovolorn_oracle as O

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16, F64 = torch.float32, torch.bfloat16, torch.float64
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def nsq():
    from promptcache_b200 import _native_seq
    _native_seq.load()
    return _native_seq


def dev(t, dtype=F32):
    return t.to(DEV, dtype).contiguous()


def close(got, want, tol, what=""):
    got, want = got.detach().cpu().to(F64), want.detach().cpu().to(F64)
    assert torch.isfinite(got).all(), f"{what}: not finite"
    err = float((got - want).abs().max() / (want.abs().max() + 1e-30))
    assert err <= tol, f"{what}: relative error {err:.3e} > {tol:.1e}"
    return err


def close_rows(got, want, tol, what="", share=0.9, worst=0.3):
    """bfloat16 runs of whole models: relative rms per row, most rows within `tol`, none beyond `worst`."""
    got, want = got.detach().cpu().to(F64), want.detach().cpu().to(F64)
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    ok = float((err <= tol).double().mean())
    assert ok >= share and float(err.max()) <= worst, f"{what}: {ok:.2f} of the rows within {tol:.1e}, worst {float(err.max()):.3e}"


def write_checkpoint(folder, cfg, W):
    from promptcache_b200 import weights as wio
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(dict(cfg, layers=[{k: v for k, v in L.items() if not k.startswith("_")} for L in cfg["layers"]]), fh)
    wio.save_file({k: v.to(BF16) for k, v in W.items()}, os.path.join(folder, "model.safetensors"))


def load(tmp_path, cfg, W, dtype=F32, name="m"):
    from promptcache_b200.model import load_model
    folder = str(tmp_path / name)
    write_checkpoint(folder, cfg, W)
    return load_model(folder, device=DEV, dtype=dtype)


def tokens(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def batch_of(nsq, slots, pos0, lens, parity=None):
    return nsq.Batch(slots, pos0, lens, torch.device(DEV), parity)


# ---- mechanisms alone ---------------------------------------------------------------------------------------------
def test_embedding_with_scaled_rows_and_pairs(nsq):
    g = torch.Generator().manual_seed(0)
    table, pair = torch.randn(40, 24, generator=g, dtype=F64), torch.randn(12, 24, generator=g, dtype=F64)
    toks = [39, 0, 7, 7, 39]
    prev = torch.tensor([-1] + toks[:-1], device=DEV)
    out = torch.empty(5, 24, device=DEV)
    nsq.embed_bigram(dev(table), dev(pair), torch.tensor(toks, device=DEV), prev, out, 11, 29, 3, scale=2.5)
    want = table[toks] * 2.5 + pair[O.pair_rows(toks, 11, 29, 3)]
    assert O.pair_rows(toks, 11, 29, 3)[0] == 11
    close(out, want, 2e-6, "scaled row + pair row")


@pytest.mark.parametrize("width,groups,taps", [(40, 5, 3), (64, 2, 4), (37, 1, 2), (48, 6, 1), (96, 3, 6), (2304, 9, 3), (4096, 4, 4)])
def test_grouped_norm_sum_and_input_convolution(nsq, width, groups, taps):
    """A sublayer's result joins the stream through the grouped norm and the next input is the NEW stream plus its convolution: whole, in
    portions (down to one token), two entries in a batch, slots with old tails."""
    g = torch.Generator().manual_seed(width + taps)
    eps, R = 1e-4, taps - 1
    for dtype, tol in ((F32, 3e-6), (BF16, 6e-3)):
        rq = lambda *s: torch.randn(*s, generator=g, dtype=F64).to(dtype).to(F64)
        T = 30
        x, y, w, cw = torch.randn(T, width, generator=g, dtype=F64).to(F32).to(F64), rq(T, width) * 2, rq(width), rq(taps, width) * 0.5
        y[:, :width // groups] *= 30.0       # one group of a far larger scale: a norm over the whole width would show
        y = y.to(dtype).to(F64)
        s = x + O.grouped_norm(y, w, groups, eps)
        h = s + O.causal_conv(s, cw.T)
        for impl in (0, 1):
            for cuts in ([30], [1] * 30, [2] * 15, [1, 2, 3, 24], [7, 1, 1, 21]):
                tail = torch.full((3, 2, max(R, 1), width), 5.0, device=DEV)
                xo, ho, p0 = torch.empty(T, width, device=DEV), torch.empty(T, width, device=DEV, dtype=dtype), 0
                for k, n in enumerate(cuts):
                    b = batch_of(nsq, [1], [p0], [n], [k & 1])
                    nsq.group_norm_conv(dev(x[p0:p0 + n]), groups, eps, dtype, x_out=xo[p0:p0 + n], y=dev(y[p0:p0 + n], dtype), w=dev(w, dtype), conv_w=dev(cw, dtype),
                                        tail=tail, h_out=ho[p0:p0 + n], batch=b, impl=impl)
                    p0 += n
                close(xo, s, 3e-6, f"new stream, impl {impl}, portions {cuts[:4]}")
                close(ho, h, tol, f"next input, impl {impl}, portions {cuts[:4]}")
                assert float(tail[0].min()) == 5.0 and float(tail[2].min()) == 5.0
        # an entry that starts beside one that goes on, and no result yet (a model's first layer)
        tail = torch.zeros(4, 2, max(R, 1), width, device=DEV)
        b1 = batch_of(nsq, [3], [0], [11], [0])
        ho = torch.empty(11, width, device=DEV, dtype=dtype)
        nsq.group_norm_conv(dev(x[:11]), groups, eps, dtype, conv_w=dev(cw, dtype), tail=tail, h_out=ho, batch=b1)
        want0 = x + O.causal_conv(x, cw.T)
        close(ho, want0[:11], tol, "without a result")
        cat = torch.cat([x[:5], x[11:]])
        b2 = batch_of(nsq, [0, 3], [0, 11], [5, T - 11], [0, 1])
        ho = torch.empty(cat.shape[0], width, device=DEV, dtype=dtype)
        nsq.group_norm_conv(dev(cat), groups, eps, dtype, conv_w=dev(cw, dtype), tail=tail, h_out=ho, batch=b2)
        close(ho[:5], want0[:5], tol, "the entry that starts")
        close(ho[5:], want0[11:], tol, "the entry that goes on")
        # the model's last norm, at some rows only, with and without a pending result
        rows = torch.tensor([28, 0, 28, 3], dtype=torch.int32, device=DEV)
        for impl in (0, 1):
            hr = torch.empty(4, width, device=DEV, dtype=dtype)
            nsq.group_norm_conv(dev(x), groups, eps, dtype, y=dev(y, dtype), w=dev(w, dtype), next_w=dev(cw[0], dtype), h_out=hr, rows=rows, impl=impl)
            close(hr, O.grouped_norm(s, cw[0], groups, eps)[[28, 0, 28, 3]], tol, f"last norm with the pending result, impl {impl}")
            nsq.group_norm_conv(dev(x), groups, eps, dtype, next_w=dev(cw[0], dtype), h_out=hr, rows=rows, impl=impl)
            close(hr, O.grouped_norm(x, cw[0], groups, eps)[[28, 0, 28, 3]], tol, f"last norm alone, impl {impl}")


def test_long_step_takes_tiles_of_tokens(nsq):
    """Enough rows for the kernel that forms four tokens per block; entries begin inside a tile."""
    g = torch.Generator().manual_seed(3)
    width, groups, taps, lens = 64, 4, 3, [5, 1, 2, 1190, 3]
    T = sum(lens)
    x, y, w, cw = (torch.randn(*s, generator=g, dtype=F64).to(BF16).to(F64) for s in ((T, width), (T, width), (width,), (taps, width)))
    s = x + O.grouped_norm(y, w, groups, 1e-5)
    for dtype, tol in ((F32, 3e-6), (BF16, 6e-3)):
        tail = torch.full((6, 2, taps - 1, width), 5.0, device=DEV)
        b = batch_of(nsq, [5, 0, 2, 4, 1], [0] * 5, lens, [0] * 5)
        xo, ho = torch.empty(T, width, device=DEV), torch.empty(T, width, device=DEV, dtype=dtype)
        nsq.group_norm_conv(dev(x), groups, 1e-5, dtype, x_out=xo, y=dev(y, dtype), w=dev(w, dtype), conv_w=dev(cw, dtype), tail=tail, h_out=ho, batch=b)
        close(xo, s, 3e-6, "new stream")
        o = 0
        for n, slot in zip(lens, (5, 0, 2, 4, 1)):
            part = s[o:o + n]
            close(ho[o:o + n], part + O.causal_conv(part, cw.T), tol, f"entry of {n} tokens")
            kept = torch.cat([torch.full((taps - 1, width), 5.0, dtype=F64), part])[-(taps - 1):]    # rows before the start are never read
            close(tail[slot, 1, max(0, taps - 1 - n):], kept[max(0, taps - 1 - n):], 3e-6, f"tail of the entry of {n} tokens")
            o += n


@pytest.mark.parametrize("dtype,H,G,D,V,rot", [(F32, 4, 2, 12, 8, 8), (F32, 3, 1, 7, 5, 6), (BF16, 6, 2, 32, 16, 32), (BF16, 4, 4, 24, 24, 10), (F32, 2, 2, 8, 12, 0),
                                               (BF16, 2, 1, 16, 8, 4)])
def test_whole_projection_and_head_norms_with_rotation(nsq, dtype, H, G, D, V, rot):
    g = torch.Generator().manual_seed(H * 100 + D)
    lens, pos0, slots, cap = [5, 3], [0, 5000], [2, 0], 5120
    b = batch_of(nsq, slots, pos0, lens)
    pos = torch.tensor(list(range(5)) + list(range(5000, 5003)))
    nq, nk, nv, pad = H * D, G * D, G * V, 8
    proj = (torch.randn(8, pad + nq + nk + nv + 2, generator=g, dtype=F64) * 2).to(dtype).to(F64)
    width = proj.shape[1] + (-proj.shape[1] % 8)
    proj = torch.cat([proj, torch.zeros(8, width - proj.shape[1], dtype=F64)], 1)
    proj[:, pad:pad + D] *= 8.0                       # one head of a larger scale: per-head and whole norms differ
    proj = proj.to(dtype).to(F64)
    q0, k0, v0 = proj[:, pad:pad + nq], proj[:, pad + nq:pad + nq + nk], proj[:, pad + nq + nk:pad + nq + nk + nv]
    wq, wk = (torch.randn(nq, generator=g, dtype=F64) + 1.5).to(dtype).to(F64), (torch.randn(nk, generator=g, dtype=F64) + 1.5).to(dtype).to(F64)
    freqs = torch.tensor([700.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F64, device=DEV) if rot else None
    tol = 3e-6 if dtype == F32 else 6e-3
    for whole in (True, False):
        if whole:
            qn, kn = O.unit_rms(q0, 1e-5, wq).view(8, H, D), O.unit_rms(k0, 1e-5, wk).view(8, G, D)
        else:
            qn, kn = O.unit_rms(q0.view(8, H, D), 1e-5, wq[:D]), O.unit_rms(k0.view(8, G, D), 1e-5, wk[:D])
        qw, kw = O.rotate_pairs(qn, pos, rot, 700.0), O.rotate_pairs(kn, pos, rot, 700.0)
        for impl in (0, 1):
            kp, vp = torch.full((3, G, cap, D), 7.0, device=DEV, dtype=dtype), torch.full((3, G, cap, V), 7.0, device=DEV, dtype=dtype)
            q = torch.empty(8, nq, device=DEV, dtype=dtype)
            nsq.rope_kv_prep(dev(proj, dtype), (pad, pad + nq, pad + nq + nk), H, G, D, V, freqs, rot, True, False, 1e-5, q, kp, vp, b,
                             q_norm_w=dev(wq if whole else wq[:D], dtype), k_norm_w=dev(wk if whole else wk[:D], dtype), norm_whole=whole, impl=impl)
            close(q.view(8, H, D), qw, tol, f"queries, whole {whole}, impl {impl}")
            rows = torch.cat([kp[2, :, :5].transpose(0, 1), kp[0, :, 5000:5003].transpose(0, 1)])
            close(rows, kw, tol, f"key rows, whole {whole}, impl {impl}")
            close(torch.cat([vp[2, :, :5].transpose(0, 1), vp[0, :, 5000:5003].transpose(0, 1)]), v0.view(8, G, V), 1e-7, "value rows")
            assert float(kp[1].min()) == 7.0 and float(kp[2, :, 5:].min()) == 7.0 and float(vp[0, :, :5000].min()) == 7.0
    # values that are the keys as projected, beside normed key rows (no rotation)
    for impl in (0, 1):
        kp, vp = torch.zeros(3, G, cap, D, device=DEV, dtype=dtype), torch.zeros(3, G, cap, D, device=DEV, dtype=dtype)
        q = torch.empty(8, nq, device=DEV, dtype=dtype)
        nsq.rope_kv_prep(dev(proj, dtype), (pad, pad + nq, pad + nq), H, G, D, D, None, 0, True, False, 1e-5, q, kp, vp, b, q_norm_w=dev(wq[:D], dtype),
                         k_norm_w=dev(wk[:D], dtype), impl=impl)
        close(kp[2, :, :5].transpose(0, 1), O.unit_rms(k0.view(8, G, D), 1e-5, wk[:D])[:5], tol, "normed key rows")
        close(vp[2, :, :5].transpose(0, 1), k0.view(8, G, D)[:5], 1e-7, "the values are the keys before their norm")


def test_distance_table_matches_the_buckets():
    from promptcache_b200.model.zovolorn import distance_bias_table
    for n_buckets, far in ((8, 14), (6, 100), (16, 60), (12, 6), (2, 5), (10, 5), (32, 128)):
        rel = torch.arange(n_buckets * 3, dtype=F64).view(n_buckets, 3)
        t = distance_bias_table(rel, far)
        for n in range(3 * far + 40):
            assert t[:, min(n, t.shape[1] - 1)].tolist() == rel[O.distance_bucket(n, n_buckets, far)].tolist(), (n_buckets, far, n)
        assert distance_bias_table(rel, far, 3).shape[1] <= 4


def attention_case(nsq, dtype, H, G, D, V, pos0, lens, chunk=0, table=None, temp=None, sink=None, gate=False, impl=0, scale=0.3, out_scale=1.0, seed=0, special=None):
    """Entries that go on beside entries that start, in shuffled slots; other slots and later rows hold numbers that must not show.  `special` =
    (entry, key position): that key outweighs all others for the entry's last query, and its value stands out."""
    g = torch.Generator().manual_seed(seed + H * 1000 + sum(lens))
    rq = lambda *s: torch.randn(*s, generator=g, dtype=F64).to(dtype).to(F64)
    B, T = len(lens), sum(lens)
    slots = [(2 * i + 1) % (B + 2) if (B + 2) % 2 else i + 1 for i in range(B)]
    ks, vs, q = [rq(p + n, G, D) for p, n in zip(pos0, lens)], [rq(p + n, G, V) for p, n in zip(pos0, lens)], rq(T, H, D)
    if special is not None:
        e, at = special
        last = sum(lens[:e + 1]) - 1
        ks[e] *= 0.1
        q[last] = 0.0
        q[last, :, 1] = 6.0
        ks[e][at, :] = 0.0
        ks[e][at, :, 1] = 24.0
        vs[e][at] = 40.0
        ks, q = [k.to(dtype).to(F64) for k in ks], q.to(dtype).to(F64)
    cap = (max(p + n for p, n in zip(pos0, lens)) + 127) // 128 * 128
    kp, vp = (torch.randn(B + 2, G, cap, D, generator=g) * 3).to(DEV, dtype), (torch.randn(B + 2, G, cap, V, generator=g) * 3).to(DEV, dtype)
    for s, k, v in zip(slots, ks, vs):
        kp[s, :, :k.shape[0]], vp[s, :, :v.shape[0]] = dev(k, dtype).transpose(0, 1), dev(v, dtype).transpose(0, 1)
    gt = rq(T, H + 3)
    wide = torch.full((T, H * V + 6), 9.0, device=DEV, dtype=dtype)     # the result is a column range of a wider matrix
    out = wide[:, 2:2 + H * V]
    ws = nsq.attn_workspace(T, H, V, DEV) if T <= 16 else None
    rel, far = table if table is not None else (None, 0)
    from promptcache_b200.model.zovolorn import distance_bias_table
    nsq.attention(dev(q.reshape(T, H * D), dtype), kp, vp, out, H, scale, None, None, sink is not None, batch_of(nsq, slots, pos0, lens), impl=impl,
                  max_keys=min(cap, chunk) if chunk else cap, workspace=ws, sink_logit=dev(sink) if sink is not None else None,
                  head_scale=dev(temp) if temp is not None else None, bias_table=dev(distance_bias_table(rel, far)) if rel is not None else None, chunk=chunk,
                  head_gate=dev(gt, dtype)[:, 1:1 + H] if gate else None, out_scale=out_scale)
    want, o = [], 0
    for p, n, k, v in zip(pos0, lens, ks, vs):
        want.append(O.softmax_attention(q[o:o + n], k, v, torch.arange(p, p + n), torch.arange(p + n), scale, sink=sink, temp=temp,
                                        rel=rel.to(F32).to(F64) if rel is not None else None, bias_max=far, chunk=chunk))
        o += n
    want = torch.cat(want)
    if gate:
        want = want * torch.sigmoid(gt[:, 1:1 + H])[:, :, None]
    assert float(wide[:, :2].min()) == 9.0 and float(wide[:, 2 + H * V:].min()) == 9.0
    return out.reshape(T, H, V), want * out_scale


@pytest.mark.parametrize("dtype,H,G,D,V", [(F32, 4, 2, 12, 10), (F32, 3, 3, 7, 5), (BF16, 4, 2, 32, 32), (BF16, 2, 1, 72, 40), (BF16, 3, 1, 136, 24)])
@pytest.mark.parametrize("pos0,lens", [([0, 37, 130], [50, 17, 90]), ([200, 3, 71, 0], [1, 1, 1, 1]), ([0], [3]), ([130], [2])])
def test_chunked_attention_with_bias_table_and_head_scales(nsq, dtype, H, G, D, V, pos0, lens):
    g = torch.Generator().manual_seed(H + D)
    temp = (torch.randn(H, generator=g, dtype=F64) * 0.4 + 1.0).to(F32).to(F64)
    rel = torch.randn(10, H, generator=g, dtype=F64).to(F32).to(F64)
    tol = 2e-5 if dtype == F32 else 2e-2
    for chunk in (0, 1, 48, 64, 70):
        for impl in ((0, 1) if chunk in (48, 0) else (0,)):
            got, want = attention_case(nsq, dtype, H, G, D, V, pos0, lens, chunk=chunk, table=(rel, 33), temp=temp, impl=impl, out_scale=0.6)
            close(got, want, tol, f"chunk {chunk}, impl {impl}")


@pytest.mark.parametrize("dtype,H,G,D,V", [(F32, 4, 2, 12, 10), (F32, 1, 1, 6, 9), (BF16, 4, 2, 96, 64), (BF16, 6, 3, 24, 16)])
@pytest.mark.parametrize("pos0,lens", [([0, 37, 130], [50, 17, 90]), ([700, 3, 71, 0], [1, 1, 1, 1]), ([260], [2])])
def test_attention_with_sinks_and_head_gates(nsq, dtype, H, G, D, V, pos0, lens):
    sink = torch.tensor([2.5, -1.0, 4.0, 0.3, 6.0, -3.0][:H], dtype=F64)
    for impl in (0, 1):
        got, want = attention_case(nsq, dtype, H, G, D, V, pos0, lens, sink=sink, gate=True, impl=impl)
        close(got, want, 2e-5 if dtype == F32 else 2e-2, f"sink and gate, impl {impl}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n_new", [1, 2, 40])
def test_chunk_edges_and_far_keys_decide(nsq, dtype, n_new):
    """One key outweighs all others for the last query.  In its chunk (the first position, the last) it answers; one position before the
    chunk's start it must not; without chunks a key hundreds of positions back answers; a strong sink silences it."""
    tol = 2e-5 if dtype == F32 else 2e-2
    H, G, D, V = 2, 1, 16, 8
    for chunk, n, at, seen in ((50, 320, 300, True), (50, 320, 299, False), (50, 320, 319, True), (50, 301, 300, True), (50, 301, 299, False), (64, 320, 256, True),
                               (64, 320, 255, False), (64, 257, 256, True), (64, 257, 255, False), (0, 700, 2, True), (0, 700, 0, True), (0, 700, 513, True)):
        got, want = attention_case(nsq, dtype, H, G, D, V, [n - n_new], [n_new], chunk=chunk, special=(0, at), seed=at)
        close(got, want, tol, f"chunk {chunk}, key {at} of {n}")
        for h in range(H):
            assert (float(got[-1, h].float().mean()) > 30.0) == seen, f"chunk {chunk}: key {at} for the query at {n - 1}, seen {seen}"
    got, want = attention_case(nsq, dtype, H, G, D, V, [700 - n_new], [n_new], special=(0, 2), sink=torch.tensor([100.0, -5.0], dtype=F64))
    close(got, want, tol, "sink against the far key")
    assert abs(float(got[-1, 0].float().mean())) < 1e-3 and float(got[-1, 1].float().mean()) > 30.0     # head 0: the sink has no value


@pytest.mark.parametrize("dtype,G,D,vw,taps", [(F32, 2, 8, 12, 4), (F32, 3, 7, 10, 3), (BF16, 2, 32, 64, 4), (F32, 1, 5, 3, 1), (BF16, 4, 96, 200, 2), (F32, 2, 12, 8, 6),
                                               (BF16, 8, 128, 2048, 4)])
def test_short_convolution_and_unit_vectors(nsq, dtype, G, D, vw, taps):
    g = torch.Generator().manual_seed(G * 10 + taps)
    T, U, R = 26, 2 * G * D, taps - 1
    ch, off = U + vw, 8
    width = (off + ch + 5 + 7) // 8 * 8
    proj = torch.randn(T, width, generator=g, dtype=F64).to(dtype).to(F64)
    cw = (torch.randn(ch, taps, generator=g, dtype=F64) * 0.7).to(dtype).to(F64)
    a = O.silu(O.causal_conv(proj[:, off:off + ch], cw))
    qk = O.unit_vector(a[:, :U].view(T, 2 * G, D))
    qk[:, :G] *= 0.25
    tol = 3e-6 if dtype == F32 else 6e-3
    pd, cd = dev(proj, dtype), dev(cw.T, dtype)
    for impl in (0, 1):
        for cuts in ([26], [1] * 26, [2, 1, 3, 20], [5, 21]):
            tail = torch.full((3, 2, max(R, 1), ch), 5.0, device=DEV)
            q, v, p0 = [], [], 0
            for k, n in enumerate(cuts):
                x, y = nsq.short_conv(pd[p0:p0 + n], off, G, D, vw, cd, tail if R else None, 0.25, O.UNIT_EPS, batch_of(nsq, [1], [p0], [n], [k & 1]), impl=impl)
                q.append(x)
                v.append(y)
                p0 += n
            close(torch.cat(q).view(T, 2 * G, D), qk, 3e-6, f"unit vectors in 32-bit, impl {impl}, portions {cuts[:4]}")
            close(torch.cat(v), a[:, U:], tol, f"values, impl {impl}, portions {cuts[:4]}")
            assert float(tail[0].min()) == 5.0 and float(tail[2].min()) == 5.0
    # a step long enough for tiles of tokens, entries beginning inside a tile
    lens = [3, 1, 650, 2]
    rep = torch.cat([proj] * 26)[:sum(lens)]
    q, v = nsq.short_conv(dev(rep, dtype), off, G, D, vw, cd, torch.full((5, 2, max(R, 1), ch), 5.0, device=DEV) if R else None, 0.25, O.UNIT_EPS,
                          batch_of(nsq, [4, 0, 3, 1], [0] * 4, lens))
    o = 0
    for n in lens:
        a = O.silu(O.causal_conv(rep[o:o + n, off:off + ch], cw))
        w = O.unit_vector(a[:, :U].view(n, 2 * G, D))
        w[:, :G] *= 0.25
        close(q[o:o + n].view(n, 2 * G, D), w, 3e-6, f"entry of {n}")
        close(v[o:o + n], a[:, U:], tol, f"entry of {n}")
        o += n


def delta_inputs(dtype, H, G, D, V, T, seed, decay_scale=1.0):
    g = torch.Generator().manual_seed(seed)
    q = O.unit_vector(torch.randn(T, G, D, generator=g, dtype=F64)) * D ** -0.5
    k = torch.randn(T, G, D, generator=g, dtype=F64)
    k[1:] = 0.7 * k[:-1] + 0.5 * k[1:]                       # neighbouring keys overlap: the corrections matter
    k = O.unit_vector(k)
    qk = torch.cat([q.reshape(T, G * D), k.reshape(T, G * D)], 1).to(F32).to(F64)
    v, b, gate = (torch.randn(T, n, generator=g, dtype=F64).to(dtype).to(F64) for n in (H * V, H + 2, H * V + 1))
    ld = (-torch.rand(T, H * D, generator=g, dtype=F64) ** 3 * decay_scale).to(F32).to(F64)
    nw = (torch.randn(V, generator=g, dtype=F64) * 0.3 + 1.0).to(dtype).to(F64)
    return qk, v, b, gate, ld, nw


def delta_want(qk, v, b, gate, ld, nw, H, G, D, V, eps, state=None):
    T = qk.shape[0]
    q, k = (t.view(T, G, D).repeat_interleave(H // G, 1) for t in (qk[:, :G * D], qk[:, G * D:]))
    o, S = O.delta_recurrence(q, k, v.view(T, H, V), ld.view(T, H, D), torch.sigmoid(b[:, 1:1 + H]), state)
    return O.unit_rms(o, eps, nw).reshape(T, H * V) * torch.sigmoid(gate[:, 1:]), S


@pytest.mark.parametrize("dtype,H,G,D,V,decay", [(F32, 4, 2, 8, 12, 1.0), (F32, 3, 3, 7, 5, 3.0), (BF16, 4, 2, 32, 64, 0.2), (BF16, 2, 1, 64, 24, 30.0), (F32, 2, 2, 128, 40, 0.05),
                                                  (BF16, 2, 1, 96, 16, 1.0), (F32, 1, 1, 256, 20, 0.5), (F32, 2, 1, 180, 8, 6.0), (F32, 1, 1, 300, 9, 1.0)])
def test_gated_delta_rule_in_portions(nsq, dtype, H, G, D, V, decay):
    """The recurrence with its norm and gate against the oracle: a prompt at once, in portions down to one token, two entries in a batch, the
    state carried in the pool, a slot that was used before; token by token (registers, shared memory) and in chunks of 64."""
    T, eps = 200, 1e-5
    qk, v, b, gate, ld, nw = delta_inputs(dtype, H, G, D, V, T, D + V, decay)
    want, S = delta_want(qk, v, b, gate, ld, nw, H, G, D, V, eps)
    tol = 5e-5 if dtype == F32 else 1.2e-2
    qkd, vd, bd, gd, nwd = dev(qk), dev(v, dtype), dev(b, dtype)[:, 1:1 + H], dev(gate, dtype)[:, 1:], dev(nw, dtype)
    dec = {False: dev(torch.exp(ld)), True: dev(ld)}
    impls = (0, 1, 2, 3) if D <= 256 else (0, 1)
    for impl in impls:
        for cuts in ([T], [1] * T, [2] * 100, [17, 2, 1, 180], [64, 64, 72], [63, 65, 72], [33, 167]):
            if impl in (1, 3) and len(cuts) > 10:
                continue
            pool = torch.full((3, H, D, V), 9.0, device=DEV)
            wide = torch.full((T, H * V + 5), 3.0, device=DEV, dtype=dtype)
            out, p0 = wide[:, 2:2 + H * V], 0
            for n in cuts:
                s = slice(p0, p0 + n)
                bt = batch_of(nsq, [1], [p0], [n])
                nsq.delta_scan(qkd[s], vd[s], dec[nsq.delta_takes_chunks(bt, D, impl)][s], bd[s], G, pool, nwd, gd[s], out[s], eps, bt, out_scale=0.8, impl=impl)
                p0 += n
            close(out, want * 0.8, tol, f"impl {impl}, portions {cuts[:4]}")
            close(pool[1], S, 5e-5, f"state, impl {impl}, portions {cuts[:4]}")
            assert float(pool[0].min()) == 9.0 and float(pool[2].min()) == 9.0 and float(wide[:, :2].min()) == 3.0 and float(wide[:, -3:].min()) == 3.0
    # unequal entries in one launch, one of them going on from a state
    for impl in [i for i in (2, 3) if i in impls]:
        pool = torch.zeros(4, H, D, V, device=DEV)
        pick = lambda t: torch.cat([t[:7], t[20:]])
        b1, b2 = batch_of(nsq, [3], [0], [20]), batch_of(nsq, [0, 3], [0, 20], [7, T - 20])
        d = dec[impl == 3]
        o1, o2 = torch.empty(20, H * V, device=DEV, dtype=dtype), torch.empty(7 + T - 20, H * V, device=DEV, dtype=dtype)
        nsq.delta_scan(qkd[:20], vd[:20], d[:20], bd[:20], G, pool, nwd, gd[:20], o1, eps, b1, impl=impl)
        nsq.delta_scan(pick(qkd), pick(vd), pick(d), pick(bd), G, pool, nwd, pick(gd), o2, eps, b2, impl=impl)
        close(torch.cat([o1, o2[7:]]), want, tol, f"the entry that goes on (impl {impl})")
        close(o2[:7], want[:7], tol, f"the entry that starts beside it (impl {impl})")


def test_delta_rule_overwrites_forgets_and_keeps(nsq):
    """A key written twice holds its second value (a plain sum would hold both); a channel with a strong decay forgets, one without keeps over
    hundreds of tokens; a decay of e^-60 per token overflows no factor of the chunked form."""
    H, D, V, T = 1, 4, 8, 300
    e = torch.eye(D, dtype=F64)
    q, k = torch.zeros(T, D, dtype=F64), torch.zeros(T, D, dtype=F64)
    v, ld, b = torch.zeros(T, V, dtype=F64), torch.zeros(T, D, dtype=F64), torch.full((T, 1), -40.0, dtype=F64)
    for t, ch, val in ((0, 0, 1.0), (1, 1, 2.0), (2, 2, 3.0), (70, 1, 5.0)):     # channel 1 is written again, in another chunk
        k[t], v[t], b[t] = e[ch], val, 40.0
    ld[3:, 2] = -60.0
    q[:] = torch.tensor([1.0, 10.0, 100.0, 1000.0], dtype=F64)
    qk = torch.cat([q, k], 1)
    want, _ = O.delta_recurrence(q.view(T, 1, D), k.view(T, 1, D), v.view(T, 1, V), ld.view(T, 1, D), torch.sigmoid(b))
    assert abs(float(want[2, 0, 0]) - 321.0) < 1e-9 and abs(float(want[5, 0, 0]) - 21.0) < 1e-9 and abs(float(want[-1, 0, 0]) - 51.0) < 1e-9
    gate = torch.full((T, V), 40.0, dtype=F64)
    for impl in (1, 2, 3):
        pool, out = torch.zeros(1, H, D, V, device=DEV), torch.empty(T, V, device=DEV)
        nsq.delta_scan(dev(qk), dev(v), dev(ld if impl == 3 else torch.exp(ld)), dev(b), 1, pool, torch.ones(V, device=DEV), dev(gate), out, 1e-12, batch_of(nsq, [0], [0], [T]),
                       impl=impl)
        close(pool[0, 0, :, 0], torch.tensor([1.0, 5.0, 0.0, 0.0], dtype=F64), 1e-6, f"state (impl {impl})")
        close(out, O.unit_rms(want, 1e-12).view(T, V), 1e-5, f"read-out (impl {impl})")


@pytest.mark.parametrize("dtype,T,H,D,r", [(F32, 5, 3, 7, 4), (F32, 90, 2, 8, 5), (BF16, 130, 4, 32, 24), (BF16, 1, 2, 16, 3)])
def test_decays_from_softplus_rates(nsq, dtype, T, H, D, r):
    g = torch.Generator().manual_seed(T)
    a, a2 = (torch.randn(T, r + 3, generator=g, dtype=F64) * 2).to(dtype).to(F64), torch.randn(H * D, r, generator=g, dtype=F64).to(dtype).to(F64)
    bias, a_log = torch.randn(H * D, generator=g, dtype=F64).to(F32).to(F64) * 3, torch.randn(H, generator=g, dtype=F64).to(F32).to(F64)
    want = O.log_decay(a[:, 2:2 + r] @ a2.T + bias, a_log, D).reshape(T, H * D)
    args = (dev(a, dtype)[:, 2:2 + r], dev(a2, dtype), dev(bias), 1.0)
    close(nsq.gla_decay(*args, rate=torch.exp(dev(a_log))), want, 3e-6, "log decays")
    close(nsq.gla_decay(*args, rate=torch.exp(dev(a_log)), expo=True), torch.exp(want), 3e-6, "decays")


@pytest.mark.parametrize("dtype,G,H,D,V,ra,rg,taps", [(F32, 2, 4, 8, 12, 5, 3, 4), (BF16, 2, 2, 32, 48, 24, 16, 4), (BF16, 1, 4, 64, 16, 8, 130, 3), (F32, 3, 3, 12, 4, 64, 40, 2),
                                                         (BF16, 2, 2, 24, 8, 1, 7, 1)])
def test_inputs_of_the_delta_rule_in_one_launch(nsq, dtype, G, H, D, V, ra, rg, taps):
    """A few tokens of several sequences: the convolution, the decays and the gate product from one launch against the oracle, and tails that the
    separate kernels go on from."""
    g = torch.Generator().manual_seed(ra + rg)
    U, vw, R = 2 * G * D, H * V, taps - 1
    ch = U + vw
    offs = (8, 8 + ch, 8 + ch + rg)                       # convolution | gate inputs | decay inputs
    width = (8 + ch + rg + ra + 7) // 8 * 8
    rq = lambda *s, sc=1.0: (torch.randn(*s, generator=g, dtype=F64) * sc).to(dtype).to(F64)
    proj, cw, a2, g2 = rq(14, width), rq(ch, taps, sc=0.6), rq(H * D, ra), rq(H * V, rg)
    dtb, rate = torch.randn(H * D, generator=g, dtype=F64).to(F32).to(F64), torch.rand(H, generator=g, dtype=F64).to(F32).to(F64)
    a = O.silu(O.causal_conv(proj[:, 8:8 + ch], cw))
    qk = O.unit_vector(a[:, :U].view(14, 2 * G, D))
    qk[:, :G] *= 0.5
    decay = torch.exp(O.log_decay(proj[:, offs[2]:offs[2] + ra] @ a2.T + dtb, torch.log(rate), D)).reshape(14, H * D)
    gate = proj[:, offs[1]:offs[1] + rg] @ g2.T
    tol = 3e-6 if dtype == F32 else 6e-3
    pd, tail = dev(proj, dtype), torch.full((2, 2, max(R, 1), ch), 5.0, device=DEV)
    out, p0 = [], 0
    for k, (n, fused) in enumerate([(1, True), (1, True), (2, False), (1, True), (5, True), (4, None)]):
        b = batch_of(nsq, [1], [p0], [n], [k & 1])
        out.append(nsq.delta_inputs(pd[p0:p0 + n], 8, G, H, D, V, dev(cw.T, dtype), tail if R else None, 0.5, O.UNIT_EPS, (offs[2], offs[2] + ra), dev(a2, dtype), dev(dtb), dev(rate),
                                    (offs[1], offs[1] + rg), dev(g2, dtype), b, True, fused=fused))
        p0 += n
    got = [torch.cat(x) for x in zip(*out)]
    close(got[0].view(14, 2 * G, D), qk, 3e-6, "unit vectors")
    close(got[1], a[:, U:], tol, "values")
    close(got[2], decay, 3e-6, "decays")
    close(got[3], gate, 3e-6 if dtype == F32 else 1e-2, "gate inputs")


def test_gelu_with_a_gate_and_soft_cap(nsq):
    g = torch.Generator().manual_seed(1)
    gu, z = torch.randn(9, 34, generator=g, dtype=F64) * 2, torch.randn(5, 77, generator=g, dtype=F64) * 30
    close(nsq.glu_mul(dev(gu), 17, (nsq.GLU_GELU_TANH, 0.0, 0.0)), O.gelu_tanh(gu[:, :17]) * gu[:, 17:], 3e-6, "gelu(g) * u")
    close(nsq.soft_cap(dev(z), 12.0), O.soft_cap(z, 12.0), 3e-6, "capped")
    assert float(nsq.soft_cap(dev(z), 12.0).abs().max()) <= 12.0
    zb = z.to(BF16)
    assert torch.equal(nsq.soft_cap(dev(zb, BF16)[:, 5:], 0.0).cpu(), zb[:, 5:].float())     # no cap: a widened copy


# ---- whole models -------------------------------------------------------------------------------------------------
def layer_sets():
    A, P = O.attention_layer, O.parallel_layer
    return {
        "mixed": dict(layers=[A(), P(), A(heads=2, kv_heads=1, dim=8, vdim=16, rot_dims=8, ff=0), P(heads=2, kv_heads=1, chunk=16, r_heads=2, r_kv_heads=2, r_vdim=8, ff=24)]),
        "parallel_first": dict(layers=[P(ff=0), P(heads=3, kv_heads=3, dim=16, chunk=5, bias_max=40, buckets=6, r_heads=6, r_kv_heads=2, r_dim=16, r_vdim=16, conv=2), A()],
                               taps=4, groups=2, cap=7.0),
        # sizes off the 16-byte pieces, one group, one tap, one head, chunks of one token, more taps than the register kernels take
        "odd": dict(layers=[P(heads=1, kv_heads=1, dim=5, chunk=1, bias_max=3, buckets=4, r_heads=3, r_kv_heads=1, r_dim=7, r_vdim=5, conv=6, rank=1, g_rank=2, ff=11),
                            A(heads=3, kv_heads=3, dim=7, vdim=5, rot_dims=2, ff=7)], groups=1, taps=1),
        "odd_taps": dict(layers=[A(heads=1, kv_heads=1, dim=6, vdim=3, rot_dims=6), P(r_heads=1, r_kv_heads=1, r_dim=3, r_vdim=9, conv=1, chunk=200)], taps=6, groups=3),
        "attention_only": dict(layers=[A(rot_dims=12, base=10000.0), A(heads=8, kv_heads=2, dim=16, vdim=16, rot_dims=4)], taps=2),
        "parallel_only": dict(layers=[P(left_scale=1.0, right_scale=1.0), P(chunk=64, bias_max=30, buckets=12)], cap=50.0),
    }


def model_set(name, width):
    spec = dict(layer_sets()[name])
    return O.make_config(spec.pop("layers"), width=width, **spec)


@pytest.mark.parametrize("name,width", [("mixed", 40), ("mixed", 64), ("parallel_first", 48), ("odd", 30), ("odd", 37), ("odd_taps", 33), ("attention_only", 64), ("parallel_only", 32)])
def test_model_whole_prompt_against_oracle(tmp_path, name, width):
    cfg = model_set(name, width)
    W = O.random_model(cfg, seed=len(name) + width)
    toks = tokens(75, cfg["vocab"], 5)
    lo = []
    want = O.forward(cfg, W, toks, lo)
    m = load(tmp_path, cfg, W, F32)
    for impl in (0, 2, 3):                  # the delta rule by step, token by token, in chunks
        m.scan_impl, m.layer_trace = impl, []
        seq = m.new_sequence()
        got = m.step([(seq, toks)], [list(range(len(toks)))])
        assert len(m.layer_trace) == len(lo)
        for i, (a, b) in enumerate(zip(m.layer_trace, lo)):
            close(a, b, 3e-5, f"{name}: stream after layer {i}, scan {impl}")
        close(got, want, 5e-5, f"{name}: logits, scan {impl}")
        seq.free()
    m.layer_trace, m.scan_impl = None, 0
    seq = m.new_sequence()                  # prompt, then token by token
    got = torch.cat([m.step([(seq, toks[:20])], [list(range(20))])] + [m.step([(seq, [t])]) for t in toks[20:]])
    close(got, want, 5e-5, f"{name}: decoded")
    mb = load(tmp_path, cfg, W, BF16, "b")
    close_rows(mb.step([(mb.new_sequence(), toks)], [list(range(len(toks)))]), want, 6e-2, f"{name}: bfloat16 logits")


@pytest.mark.parametrize("dtype,tol", [(F32, 5e-5), (BF16, 6e-2)])
def test_portions_decoding_batches_and_slot_reuse(tmp_path, dtype, tol):
    """One set of sequences run whole, in portions of several sizes down to two tokens, token by token (through the replayed graph), in unequal
    batches whose shorter members leave early, and through slots that were used before.  Chunks of 9 and 16 positions begin inside portions."""
    cfg = model_set("mixed", 40)
    W = O.random_model(cfg, seed=11)
    V = cfg["vocab"]
    seqs = [tokens(n, V, 20 + n) for n in (61, 9, 30, 1)]
    want = [O.forward(cfg, W, s) for s in seqs]
    m = load(tmp_path, cfg, W, dtype)
    cmp = close if dtype == F32 else close_rows

    def run(toks, cuts):
        seq, out, p = m.new_sequence(), [], 0
        for n in cuts:
            out.append(m.step([(seq, toks[p:p + n])], [list(range(n))]))
            p += n
        seq.free()
        return torch.cat(out)

    for cuts in ([61], [2] * 30 + [1], [1] * 61, [17, 2, 3, 1, 1, 30, 7], [40] + [1] * 21, [20, 25, 16], [1, 60], [9, 7, 2, 43]):
        cmp(run(seqs[0], cuts), want[0], tol, f"portions {cuts[:6]}...")
    from promptcache_b200.batch_engine import BatchEngine
    eng = BatchEngine(m)
    pre = [40, 4, 22, 1]
    got = [[] for _ in seqs]
    lg = eng.step([(f"r{i}", s[:n], list(range(n))) for i, (s, n) in enumerate(zip(seqs, pre))])
    o = 0
    for i, n in enumerate(pre):
        got[i].append(lg[o:o + n])
        o += n
    at = list(pre)
    while any(a < len(s) for a, s in zip(at, seqs)):
        live = [i for i, s in enumerate(seqs) if at[i] < len(s)]
        done = [f"r{i}" for i in live if at[i] + 1 == len(seqs[i])]
        lg = eng.step([(f"r{i}", [seqs[i][at[i]]], [0]) for i in live], done)
        for k_, i in enumerate(live):
            got[i].append(lg[k_:k_ + 1])
            at[i] += 1
    eng.end("r3")
    for i in range(len(seqs)):
        cmp(torch.cat(got[i]), want[i], tol, f"request {i} in a batch")
    # the freed slots are handed out again, to other sequences and in another order: nothing of the old states shows
    lg = eng.step([("x", seqs[2], None), ("y", seqs[0], None), ("z", seqs[1], None)], ["x", "y", "z"])
    cmp(lg, torch.stack([want[2][-1], want[0][-1], want[1][-1]]), tol, "reused slots")
    # requests that join a running batch, and a portion beside decoded tokens
    a, b = m.new_sequence(), m.new_sequence()
    m.step([(a, seqs[0][:30])])
    lg = m.step([(a, [seqs[0][30]]), (b, seqs[2][:25])], [[0], [24]])
    cmp(lg, torch.stack([want[0][30], want[2][24]]), tol, "a prompt beside a decoded token")
    lg = m.step([(b, seqs[2][25:]), (a, seqs[0][31:33])], [[4], [1]])
    cmp(lg, torch.stack([want[2][29], want[0][32]]), tol, "two portions")


@pytest.mark.parametrize("dtype,tol", [(F32, 5e-5), (BF16, 6e-2)])
def test_tensor_core_sizes_in_portions_and_batches(tmp_path, dtype, tol):
    """Head sizes the tensor-core kernel serves, prompts in portions of 16 tokens and more, chunks of 24 and 128 positions, an unequal batch."""
    A, P = O.attention_layer, O.parallel_layer
    cfg = O.make_config([P(heads=4, kv_heads=2, dim=32, chunk=24, bias_max=20, r_heads=4, r_kv_heads=2, r_dim=32, r_vdim=32, rank=8, g_rank=8),
                         A(heads=4, kv_heads=2, dim=64, vdim=32, rot_dims=32), P(heads=2, kv_heads=2, dim=64, chunk=128, bias_max=90, buckets=14, r_heads=2, r_kv_heads=1, r_dim=64, r_vdim=48)],
                        width=96, groups=3)
    W = O.random_model(cfg, seed=17)
    seqs = [tokens(n, cfg["vocab"], 70 + n) for n in (150, 33, 80)]
    want = [O.forward(cfg, W, s) for s in seqs]
    m = load(tmp_path, cfg, W, dtype)
    cmp = close if dtype == F32 else close_rows
    for cuts in ([150], [40, 17, 64, 29], [16, 16, 100, 2, 16], [149, 1], [128, 22]):
        seq, out, p_ = m.new_sequence(), [], 0
        for n in cuts:
            out.append(m.step([(seq, seqs[0][p_:p_ + n])], [list(range(n))]))
            p_ += n
        seq.free()
        cmp(torch.cat(out), want[0], tol, f"portions {cuts}")
    ss = [m.new_sequence() for _ in seqs]
    first = [70, 17, 40]
    a = m.step([(q_, s_[:n]) for q_, s_, n in zip(ss, seqs, first)], [list(range(n)) for n in first])
    b = m.step([(q_, s_[n:]) for q_, s_, n in zip(ss, seqs, first)], [list(range(len(s_) - n)) for s_, n in zip(seqs, first)])
    oa = ob = 0
    for i, (s_, n) in enumerate(zip(seqs, first)):
        cmp(torch.cat([a[oa:oa + n], b[ob:ob + len(s_) - n]]), want[i], tol, f"request {i} of the batch")
        oa += n
        ob += len(s_) - n
    for q_ in ss:
        q_.free()


def test_long_decoding_chunks_pass_and_the_pool_grows(tmp_path):
    """300 tokens decoded one by one after a short prompt: chunks of 44 and 100 positions begin and end in decoded tokens, the pool grows while the
    sequence lives (captured graphs are rebuilt, the full attention splits its keys), a second sequence joins and leaves."""
    A, P = O.attention_layer, O.parallel_layer
    cfg = O.make_config([P(chunk=44, bias_max=30), A(heads=2, kv_heads=1, dim=16, vdim=8, rot_dims=8), P(heads=2, kv_heads=2, chunk=100, bias_max=60, buckets=10, ff=0)])
    W = O.random_model(cfg, seed=3)
    toks = tokens(330, cfg["vocab"], 8)
    want = O.forward(cfg, W, toks)
    m = load(tmp_path, cfg, W, F32)
    seq = m.new_sequence()
    out = [m.step([(seq, toks[:30])], [list(range(30))])]
    other = None
    for p in range(30, 330):
        if p == 100:
            other = m.new_sequence()
            m.step([(other, toks[:50])])
        if other is not None and 100 <= p < 140:
            lg = m.step([(seq, [toks[p]]), (other, [toks[p - 50]])])
            close(lg[1], want[p - 50], 5e-5, f"second sequence at {p - 50}")
            out.append(lg[:1])
        else:
            if other is not None and p == 140:
                other.free()
            out.append(m.step([(seq, [toks[p]])]))
    close(torch.cat(out), want, 5e-5, "long decoding")


def test_medium_model_long_prompt(tmp_path):
    """Sizes at which the other code paths run: full attention over many key tiles on the tensor cores, twenty chunks of the delta rule with 128 key
    channels, rows for the tiled boundary kernel, decoding that splits the keys."""
    A, P = O.attention_layer, O.parallel_layer
    cfg = O.make_config([P(heads=8, kv_heads=2, dim=64, chunk=200, bias_max=150, buckets=24, scale=0.2, r_heads=4, r_kv_heads=2, r_dim=128, r_vdim=64, rank=16, g_rank=16, ff=256),
                         A(heads=8, kv_heads=2, dim=48, vdim=64, rot_dims=48, base=10000.0, scale=0.2, ff=256),
                         P(heads=2, kv_heads=1, dim=128, chunk=512, bias_max=300, buckets=32, r_heads=8, r_kv_heads=4, r_dim=32, r_vdim=32, ff=0)], width=192, vocab=300, groups=6,
                        embed_scale=4.0)
    W = O.random_model(cfg, seed=21)
    toks = tokens(1320, 300, 4)
    rows = sorted(list(range(0, 1300, 97)) + [399, 400, 511, 512, 1023, 1024, 1297, 1298, 1299])
    want = O.forward(cfg, W, toks)
    for dtype in (F32, BF16):
        m = load(tmp_path, cfg, W, dtype, str(dtype)[-4:])
        for cuts in ([1300], [700, 600]):
            seq, p, got = m.new_sequence(), 0, []
            for n in cuts:
                got.append(m.step([(seq, toks[p:p + n])], [[r - p for r in rows if p <= r < p + n]]))
                p += n
            for t in toks[1300:]:
                got.append(m.step([(seq, [t])]))
            got = torch.cat(got)
            ref = want[rows + list(range(1300, 1320))]
            if dtype == F32:
                close(got, ref, 1e-4, f"medium model, float32, {cuts}")
            else:
                close_rows(got, ref, 5e-2, f"medium model, bfloat16, {cuts}")
            seq.free()


def test_greedy_generation_through_the_engines(tmp_path):
    from promptcache_b200.batch_engine import BatchEngine
    from promptcache_b200.generation_engine import GenerationEngine, GenerationParameters
    from promptcache_b200.model import Zovolorn
    cfg = model_set("mixed", 48)
    W = O.random_model(cfg, seed=5)
    prompts = [tokens(n, cfg["vocab"], 40 + n) for n in (12, 3, 25)]
    n_new = 10
    want = [O.greedy(cfg, W, p, n_new) for p in prompts]
    folder = str(tmp_path / "g")
    write_checkpoint(folder, cfg, W)
    lm = Zovolorn(folder, device=DEV, dtype=F32)
    params = GenerationParameters(temperature=0.0, max_new_tokens=n_new, stop_token_ids=[], stop_str=[])
    assert BatchEngine(lm.hf_model, max_tokens=4096).generate(prompts, params) == want
    for p, w in zip(prompts, want):
        outs = list(GenerationEngine(lm).generate(p, list(range(len(p))), params, None, stream_interval=2))
        assert outs[-1].new_text == lm.decode(w)
    assert not lm.hf_model.pool.rows                         # the engines gave their slots back
    stop = want[2][3]
    stopped = BatchEngine(lm.hf_model, max_tokens=64).generate(prompts, GenerationParameters(temperature=0.0, max_new_tokens=n_new, stop_token_ids=[stop]))
    assert stopped[2] == want[2][:want[2].index(stop) + 1]


def test_trace_replay_end_to_end(tmp_path):
    import numpy as np
    cfg = model_set("parallel_first", 48)
    W = O.random_model(cfg, seed=9)
    folder = str(tmp_path / "t")
    write_checkpoint(folder, cfg, W)
    a, b = tokens(20, cfg["vocab"], 1), tokens(7, cfg["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:15], "want": [0, 14]}, {"id": "b", "tokens": b[:6], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[15:16], "want": [0]}, {"id": "b", "tokens": b[6:], "want": [0]}], "end": ["b"]}] + \
            [{"step": 2 + i, "entries": [{"id": "a", "tokens": [a[16 + i]], "want": [0]}], "end": ["a"] if i == 3 else []} for i in range(4)]
    out = str(tmp_path / "out")
    wa, wb = O.forward(cfg, W, a), O.forward(cfg, W, b)
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 0.1)):
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out, "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(6)]
        rd = lambda i: torch.from_numpy(np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]).copy())
        cmp = close if dtype == "float32" else (lambda g_, w_, t_, s_: close_rows(g_, w_, t_, s_, share=1.0))
        cmp(rd(0), wa[[0, 14]], tol, "step 0")
        cmp(rd(1), torch.stack([wa[15], wb[6]]), tol, "step 1")
        for i in range(4):
            cmp(rd(2 + i), wa[16 + i:17 + i], tol, f"step {2 + i}")
