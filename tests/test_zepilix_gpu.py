"""The Zepilix design on the GPU against the float64 oracle (tests/zepilix_oracle.py): each mechanism alone through the kernels'
bindings, then whole models through the step function, the batch engine, the generation engine and bin/trace_run."""
import json
import os
import subprocess

import pytest
import torch

from tests import zepilix_oracle as O

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
        json.dump(cfg, fh)
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
@pytest.mark.parametrize("width", [40, 37, 64, 1000, 2304, 4096, 4600])
def test_sums_and_rms_norms_of_the_stream(nsq, width):
    """Two results, or one result through its own norm with the embedding output and a pass's vector, then two norms stored around zero; a copy in
    the compute type; the last norm at some rows."""
    g = torch.Generator().manual_seed(width)
    T, eps = 5, 1e-4
    for dtype, tol in ((F32, 3e-6), (BF16, 6e-3)):
        rq = lambda *s: torch.randn(*s, generator=g, dtype=F64).to(dtype).to(F64)
        x, x0 = (torch.randn(T, width, generator=g, dtype=F64).to(F32).to(F64) for _ in range(2))
        y, f, w1, w2, yn, step = rq(T, width), rq(T, width), rq(width) * 0.5, rq(width) * 0.5, rq(width), rq(width)
        h1, h2, cp = (torch.empty(T, width, device=DEV, dtype=dtype) for _ in range(3))
        xd = dev(x)
        nsq.add_rms_norm(xd, [(dev(y, dtype), 1.0), (dev(f, dtype), 1.0)], eps, copy=cp)
        s = x + y + f
        close(xd, s, 3e-6, "sum")
        close(cp, s, tol, "copy")
        for with_x0 in (False, True):
            xd = dev(s)
            sv = dev(step, dtype).expand(T, width)
            adds = [(dev(y, dtype), 1.0)] + ([(dev(x0), 1.0)] if with_x0 else []) + [(sv, 1.0)]
            nsq.add_rms_norm(xd, adds, eps, dev(w1, dtype), h1, dev(w2, dtype), h2, w_offset=1.0, y_norm_w=dev(yn, dtype))
            want = s + O.unit_rms(y, eps, yn) + (x0 if with_x0 else 0) + step
            close(xd, want, 3e-6, "normed result, embedding output, pass vector")
            close(h1, O.stream_norm(want, w1, eps), tol, "first norm")
            close(h2, O.stream_norm(want, w2, eps), tol, "second norm")
        rows = torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
        hr = torch.empty(3, width, device=DEV, dtype=dtype)
        nsq.add_rms_norm(dev(x), [], eps, dev(w1, dtype), hr, rows=rows, w_offset=1.0)
        close(hr, O.stream_norm(x, w1, eps)[[4, 0, 4]], tol, "some rows")


@pytest.mark.parametrize("width,dim", [(40, 6), (64, 16), (37, 5), (256, 24), (1000, 40), (2048, 128), (2048, 256), (4608, 64), (8, 8), (136, 200)])
def test_token_side_input(nsq, width, dim):
    """Both forms of a layer's end: products around the gate kernel, and everything in one launch; the layer's part of the table's row."""
    g = torch.Generator().manual_seed(width + dim)
    T, eps, vocab, layers, li = 6, 1e-4, 11, 3, 1
    ids = [3, 10, 0, 3, 7, 1]
    for dtype, tol in ((F32, 5e-6), (BF16, 2e-2)):
        rq = lambda *s, sc=1.0: (torch.randn(*s, generator=g, dtype=F64) * sc).to(dtype).to(F64)
        x, x0 = (torch.randn(T, width, generator=g, dtype=F64).to(F32).to(F64) for _ in range(2))
        y, f, table = rq(T, width), rq(T, width), rq(vocab, layers * dim)
        gate, proj, wn, step, w1, w2 = rq(dim, width, sc=width ** -0.5), rq(width, dim, sc=dim ** -0.5), rq(width), rq(width), rq(width), rq(width)
        idd, e = torch.tensor(ids, device=DEV), table[ids, li * dim:(li + 1) * dim]
        for n_res, entering, norms in ((2, 2, 2), (1, 1, 1), (2, 0, 0), (0, 1, 2)):
            s = x + (y if n_res else 0) + (f if n_res > 1 else 0)
            want = s + O.side_input(s, e, gate, proj, wn, eps) + (x0 if entering > 1 else 0) + (step if entering else 0)
            xd, h1, h2 = dev(x), torch.empty(T, width, device=DEV, dtype=dtype), torch.empty(T, width, device=DEV, dtype=dtype)
            nsq.side_boundary(xd, [dev(y, dtype), dev(f, dtype)][:n_res], idd, dev(table, dtype), li * dim, dev(gate, dtype), dev(proj, dtype), dev(wn, dtype), eps,
                              x0=dev(x0) if entering > 1 else None, step=dev(step, dtype) if entering else None, w1=dev(w1, dtype) if norms else None, h1=h1,
                              w2=dev(w2, dtype) if norms > 1 else None, h2=h2, w_offset=1.0)
            close(xd, want, 5e-6, f"one launch: stream, {n_res} results, {entering} entering")
            if norms:
                close(h1, O.stream_norm(want, w1, eps), tol, "one launch: first norm")
            if norms > 1:
                close(h2, O.stream_norm(want, w2, eps), tol, "one launch: second norm")
        u = rq(T, dim + 3)
        close(nsq.side_gate(dev(u, dtype)[:, 2:2 + dim], dev(table, dtype), li * dim, idd), O.gelu_tanh(u[:, 2:2 + dim]) * e, 3e-6 if dtype == F32 else 6e-3, "gate kernel")


@pytest.mark.parametrize("dtype,H,G,D,rot", [(F32, 4, 2, 12, 8), (F32, 3, 1, 7, 6), (BF16, 6, 2, 32, 32), (BF16, 4, 4, 24, 10), (F32, 2, 1, 8, 2)])
def test_rotated_unit_heads_and_values_that_are_the_keys(nsq, dtype, H, G, D, rot):
    g = torch.Generator().manual_seed(H * 100 + D)
    lens, pos0, slots, cap = [5, 3], [0, 5000], [2, 0], 5120
    b, pos = batch_of(nsq, slots, pos0, lens), torch.tensor(list(range(5)) + list(range(5000, 5003)))
    nq, nk = H * D, G * D
    proj = torch.randn(8, (nq + nk + 7) // 8 * 8, generator=g, dtype=F64).to(dtype).to(F64) * 2
    proj[:, :D] *= 8.0
    q0, k0 = proj[:, :nq].view(8, H, D), proj[:, nq:nq + nk].view(8, G, D)
    qw, kw = (O.unit_rms(O.rotate_pairs(t, pos, rot, 700.0), 1e-5) for t in (q0, k0))
    freqs = torch.tensor([700.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F64, device=DEV)
    one, tol = torch.ones(D, device=DEV, dtype=dtype), 3e-6 if dtype == F32 else 6e-3
    for impl in (0, 1):
        kp, vp = torch.full((3, G, cap, D), 7.0, device=DEV, dtype=dtype), torch.full((3, G, cap, D), 7.0, device=DEV, dtype=dtype)
        q = torch.empty(8, nq, device=DEV, dtype=dtype)
        nsq.rope_kv_prep(dev(proj, dtype), (0, nq, nq), H, G, D, D, freqs, rot, True, False, 1e-5, q, kp, vp, b, q_norm_w=one, k_norm_w=one, impl=impl)
        close(q.view(8, H, D), qw, tol, f"queries, impl {impl}")
        rows = lambda p: torch.cat([p[2, :, :5].transpose(0, 1), p[0, :, 5000:5003].transpose(0, 1)])
        close(rows(kp), kw, tol, f"key rows, impl {impl}")
        close(rows(vp), k0, 1e-7, "values: the keys as projected")
        assert float(kp[1].min()) == 7.0 and float(vp[2, :, 5:].min()) == 7.0


def latent_case(dtype, H, D, R, V, C, Q, width, window, T, seed, special=None):
    """A random latent mixer and inputs, the oracle's result per head; `special` = (query, key): the key outweighs all others for that query, its
    value stands out (the plain parts of the scores are silenced for it)."""
    g = torch.Generator().manual_seed(seed)
    rq = lambda *s, sc=1.0: (torch.randn(*s, generator=g, dtype=F64) * sc).to(dtype).to(F64)
    W = {"m.dq": rq(Q, width, sc=width ** -0.5), "m.dq.norm": rq(Q), "m.uq": rq(H * (D + R), Q, sc=Q ** -0.5), "m.dkv": rq(C + R, width, sc=width ** -0.5),
         "m.dkv.norm": rq(C) + 1.0, "m.uk": rq(H * D, C, sc=C ** -0.5), "m.uv": rq(H * V, C, sc=C ** -0.5), "m.o": torch.eye(H * V, dtype=F64)}
    h = rq(T, width)
    if special is not None:                     # inputs channel 0 drives one latent channel, which one key and value part read
        qi, kj = special
        h[:, 0] = 0.0
        h[kj] = 0.0
        h[kj, 0] = 4.0
        W["m.dkv"][:, 0] = 0.0
        W["m.dkv"][0, 0] = 64.0
        W["m.dkv"][0, 1:] = 0.0
        W["m.dkv.norm"][0] = 1.0
        W["m.uk"][:, 0] = 0.0
        W["m.uv"][:, 0] = 0.0
        h[qi] = 0.0
        h[qi, 1] = 4.0
        W["m.dq"][:, 1] = 0.0
        W["m.dq"][0, 1] = 64.0
        W["m.dq"][0, 2:] = 0.0
        W["m.dq.norm"][0] = 1.0
        W["m.uq"][:, 0] = 0.0
        for hd in range(H):
            W["m.uk"][hd * D, 0] = 4.0
            W["m.uv"][hd * V:(hd + 1) * V, 0] = 32.0
            W["m.uq"][hd * (D + R), 0] = 4.0
    cfg = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": C, "q_rank": Q, "rot": {"base": 90.0, "dims": R}, "scale": 0.5, "mask": {"size": window}}
    want = O.latent_attention_mixer(W, "m.", h, cfg, 1e-5, torch.arange(T))
    return W, cfg, h, want


def run_latent(nsq, dtype, W, cfg, h, cuts, form, window, slot=1, pool=None):
    from promptcache_b200.model._latent import latent_attention, load_latent
    R = cfg["rot_dim"]
    freqs = [90.0 ** (-2.0 * i / R) for i in range(R // 2)]
    blk = load_latent(lambda n: dev(W[n], dtype), "m.", "layer", cfg, freqs, interleaved=True, window=window, device=DEV)
    T = h.shape[0]
    cap = (T + 127) // 128 * 128
    ckv = pool if pool is not None else torch.full((3, 1, cap, cfg["kv_rank"] + R), 50.0, device=DEV, dtype=dtype)
    out, p0 = [], 0
    for n in cuts:
        b = batch_of(nsq, [slot], [p0], [n])
        out.append(latent_attention(dev(h[p0:p0 + n], dtype), blk, ckv, b, {}, 1e-5, cap, form=form))
        p0 += n
    return torch.cat(out)


@pytest.mark.parametrize("dtype,H,D,R,V,C,Q", [(F32, 3, 7, 4, 5, 9, 6), (F32, 2, 8, 6, 12, 16, 10), (BF16, 4, 32, 16, 48, 64, 40), (BF16, 20, 16, 8, 24, 128, 24), (BF16, 2, 64, 32, 64, 560, 32)])
def test_latent_attention_under_a_window(nsq, dtype, H, D, R, V, C, Q):
    """Both forms, whole and in portions down to one token, windows of one token to more than the prompt."""
    width, T = 32, 150
    tol = 2e-5 if dtype == F32 else 3e-2
    for window in (1, 5, 64, 96, 400):
        W, cfg, h, want = latent_case(dtype, H, D, R, V, C, Q, width, window, T, H + window)
        for form in (None, "expanded", "latent"):
            for cuts in ([T], [70, 80], [64, 1, 2, 83], [130, 20], [17] * 8 + [14]) + (([100] + [1] * 50,) if form is None else ()):
                close(run_latent(nsq, dtype, W, cfg, h, cuts, form, window), want, tol, f"window {window}, {form}, portions {cuts[:4]}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n_new", [1, 2, 40])
def test_window_edges_decide(nsq, dtype, n_new):
    """One key outweighs all others for the last query: window - 1 tokens back it answers, window tokens back it must not."""
    H, D, R, V, C, Q = 2, 16, 8, 8, 32, 16
    for window, T, back, seen in ((64, 300, 63, True), (64, 300, 64, False), (50, 300, 49, True), (50, 300, 50, False), (50, 300, 0 + 1, True), (128, 321, 127, True), (128, 321, 128, False),
                                  (1000, 321, 320, True), (1000, 321, 200, True)):
        W, cfg, h, want = latent_case(dtype, H, D, R, V, C, Q, 24, window, T, window + back, special=(T - 1, T - 1 - back))
        assert (float(want[-1].mean()) > 20.0) == seen, (window, back, float(want[-1].mean()))
        for form in ("expanded", "latent"):
            got = run_latent(nsq, dtype, W, cfg, h, [T - n_new, n_new], form, window)
            close(got[-1:], want[-1:], 2e-5 if dtype == F32 else 3e-2, f"window {window}, {back} back, {form}, {n_new} new")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n_new", [1, 2, 40])
def test_far_keys_answer_in_full_attention(nsq, dtype, n_new):
    H, G, D, T = 4, 2, 32, 700
    g = torch.Generator().manual_seed(n_new)
    for at in (0, 2, 63, 64, 127, 128, 511, 512, T - 1):
        rq = lambda *s: torch.randn(*s, generator=g, dtype=F64).to(dtype).to(F64)
        k, v, q = rq(T, G, D) * 0.125, rq(T, G, D), rq(n_new, H, D)
        q[-1], k[at] = 0.0, 0.0
        q[-1, :, 1], k[at, :, 1], v[at] = 6.0, 24.0, 40.0
        k = k.to(dtype).to(F64)
        kp, vp = torch.randn(2, G, 768, D, device=DEV).to(dtype) * 30, torch.randn(2, G, 768, D, device=DEV).to(dtype) * 30
        kp[1, :, :T], vp[1, :, :T] = dev(k, dtype).transpose(0, 1), dev(v, dtype).transpose(0, 1)
        out = torch.empty(n_new, H * D, device=DEV, dtype=dtype)
        nsq.attention(dev(q.reshape(n_new, H * D), dtype), kp, vp, out, H, 0.3, None, None, False, batch_of(nsq, [1], [T - n_new], [n_new]), max_keys=768,
                      workspace=nsq.attn_workspace(n_new, H, D, DEV) if n_new <= 16 else None)
        want = O.softmax_attention(q, k, v, torch.arange(T - n_new, T), torch.arange(T), 0.3)
        close(out.view(n_new, H, D), want, 2e-5 if dtype == F32 else 2e-2, f"key {at}")
        assert float(out[-1].float().min()) > 30.0


def delta_case(dtype, H, G, D, V, T, seed, strong=0.0):
    g = torch.Generator().manual_seed(seed)
    q = O.unit_vector(torch.randn(T, G, D, generator=g, dtype=F64)) * D ** -0.5
    k = torch.randn(T, G, D, generator=g, dtype=F64)
    k[1:] = 0.7 * k[:-1] + 0.5 * k[1:]                       # neighbouring keys overlap: the corrections matter
    qk = torch.cat([q.reshape(T, G * D), O.unit_vector(k).reshape(T, G * D)], 1).to(F32).to(F64)
    v, b, a, gate = (torch.randn(T, n, generator=g, dtype=F64).to(dtype).to(F64) for n in (H * V, H + 2, H + 1, H * V + 1))
    a_log, dtb = (torch.randn(H, generator=g, dtype=F64) * 0.5 - 2.0 + strong).to(F32).to(F64), torch.randn(H, generator=g, dtype=F64).to(F32).to(F64)
    nw = (torch.randn(V, generator=g, dtype=F64) * 0.3 + 1.0).to(dtype).to(F64)
    q, k = (t.view(T, G, D).repeat_interleave(H // G, 1) for t in (qk[:, :G * D], qk[:, G * D:]))
    o, S = O.delta_recurrence(q, k, v.view(T, H, V), O.log_decay(a[:, 1:], a_log, dtb), torch.sigmoid(b[:, 1:1 + H]))
    return qk, v, b, a, a_log, dtb, gate, nw, O.unit_rms(o, 1e-5, nw).reshape(T, H * V) * O.silu(gate[:, 1:]), S


@pytest.mark.parametrize("dtype,H,G,D,V,strong", [(F32, 4, 2, 8, 12, 0.0), (F32, 3, 3, 7, 5, 1.0), (BF16, 4, 2, 32, 64, 0.0), (BF16, 2, 1, 64, 24, 4.0), (F32, 2, 2, 128, 40, -3.0),
                                                   (BF16, 2, 1, 96, 16, 0.0), (F32, 1, 1, 256, 20, 2.0), (F32, 2, 1, 180, 8, 5.0), (F32, 1, 1, 300, 9, 1.0), (BF16, 6, 3, 20, 9, 1.0),
                                                   (BF16, 2, 2, 136, 32, 0.0)])
def test_delta_rule_with_a_decay_per_head_in_portions(nsq, dtype, H, G, D, V, strong):
    T = 200
    qk, v, b, a, a_log, dtb, gate, nw, want, S = delta_case(dtype, H, G, D, V, T, D + V, strong)
    tol = 5e-5 if dtype == F32 else 1.2e-2
    qkd, vd, bd, ad, gd, nwd = dev(qk), dev(v, dtype), dev(b, dtype)[:, 1:1 + H], dev(a, dtype)[:, 1:], dev(gate, dtype)[:, 1:], dev(nw, dtype)
    rate, dtd = torch.exp(dev(a_log)), dev(dtb)
    run = lambda s, pool, out, bt, impl: nsq.delta_scan(qkd[s], vd[s], None, bd[s], G, pool, nwd, gd[s], out, 1e-5, bt, impl=impl, head_decay=(ad[s], dtd, rate), gate_silu=True)
    impls = (0, 1, 2, 3) if D <= 256 else (0, 1)
    for impl in impls:
        for cuts in ([T], [1] * T, [2] * 100, [17, 2, 1, 180], [64, 64, 72], [63, 65, 72], [33, 167]):
            if impl in (1, 3) and len(cuts) > 10:
                continue
            pool, out, p0 = torch.full((3, H, D, V), 9.0, device=DEV), torch.empty(T, H * V, device=DEV, dtype=dtype), 0
            for n in cuts:
                s = slice(p0, p0 + n)
                run(s, pool, out[s], batch_of(nsq, [1], [p0], [n]), impl)
                p0 += n
            close(out, want, tol, f"impl {impl}, portions {cuts[:4]}")
            close(pool[1], S, 5e-5, f"state, impl {impl}, portions {cuts[:4]}")
            assert float(pool[0].min()) == 9.0 and float(pool[2].min()) == 9.0
    # unequal entries in one launch, one of them going on from a state
    for impl in [i for i in (2, 3) if i in impls]:
        pool = torch.zeros(4, H, D, V, device=DEV)
        o1, o2 = torch.empty(20, H * V, device=DEV, dtype=dtype), torch.empty(7 + T - 20, H * V, device=DEV, dtype=dtype)
        run(slice(0, 20), pool, o1, batch_of(nsq, [3], [0], [20]), impl)
        pick = lambda t: torch.cat([t[:7], t[20:]])
        nsq.delta_scan(pick(qkd), pick(vd), None, pick(bd), G, pool, nwd, pick(gd), o2, 1e-5, batch_of(nsq, [0, 3], [0, 20], [7, T - 20]), impl=impl,
                       head_decay=(pick(ad), dtd, rate), gate_silu=True)
        close(torch.cat([o1, o2[7:]]), want, tol, f"the entry that goes on (impl {impl})")
        close(o2[:7], want[:7], tol, f"the entry that starts beside it (impl {impl})")


def test_delta_rule_overwrites_forgets_and_keeps_per_head(nsq):
    """Two heads on the same keys: one keeps for hundreds of tokens (a key written twice holds its second value), the other forgets with e^-60 per
    token, which overflows no factor of the chunked form."""
    H, D, V, T = 2, 4, 8, 300
    e = torch.eye(D, dtype=F64)
    q, k, v = torch.zeros(T, 1, D, dtype=F64), torch.zeros(T, 1, D, dtype=F64), torch.zeros(T, H * V, dtype=F64)
    a, b = torch.full((T, H), -200.0, dtype=F64), torch.full((T, H), -40.0, dtype=F64)
    for t, ch, val in ((0, 0, 1.0), (1, 1, 2.0), (2, 2, 3.0), (70, 1, 5.0)):
        k[t, 0], v[t], b[t] = e[ch], val, 40.0
    a[3:70, 1], a[71:, 1] = 60.0, 60.0          # head 1 forgets between the writes and after the last one
    q[:] = torch.tensor([1.0, 10.0, 100.0, 1000.0], dtype=F64)
    ld = O.log_decay(a, torch.zeros(H, dtype=F64), torch.zeros(H, dtype=F64))
    want, S = O.delta_recurrence(q.expand(T, H, D), k.expand(T, H, D), v.view(T, H, V), ld, torch.sigmoid(b))
    assert abs(float(want[-1, 0, 0]) - 351.0) < 1e-9 and float(want[-1, 1].abs().max()) < 1e-9 and abs(float(want[70, 1, 0]) - 50.0) < 1e-9
    one, gate = torch.ones(H, device=DEV), torch.full((T, H * V), 40.0, device=DEV)
    for impl in (1, 2, 3):
        pool, out = torch.zeros(1, H, D, V, device=DEV), torch.empty(T, H * V, device=DEV)
        nsq.delta_scan(dev(torch.cat([q, k], 1).reshape(T, 2 * D)), dev(v), None, dev(b), 1, pool, torch.ones(V, device=DEV), gate, out, 1e-12, batch_of(nsq, [0], [0], [T]), impl=impl,
                       head_decay=(dev(a), torch.zeros(H, device=DEV), one), gate_silu=True)
        close(pool[0], S, 1e-6, f"state (impl {impl})")
        got, w = out.view(T, H, V)[:, :, 0].cpu().to(F64) / 40.0, O.unit_rms(want, 1e-12)[:, :, 0]
        close(got[:, 0], w[:, 0], 1e-5, f"the head that keeps (impl {impl})")
        close(got[:3, 1], w[:3, 1], 1e-5, f"the head that forgets, before (impl {impl})")


# ---- whole models -------------------------------------------------------------------------------------------------
def layer_sets():
    A, D, L = O.attention_layer, O.delta_layer, O.latent_layer
    return {
        "mixed": dict(layers=[D(), L(), A(), D(heads=2, kv_heads=1, dim=16, vdim=8, conv=3, ff=24), L(heads=2, window=20, ff=0)], loop=(1, 4, 2)),
        "loop_first": dict(layers=[A(rot_dims=12, base=10000.0), D(heads=6, kv_heads=2, dim=8, vdim=16, conv=2, ff=0), L(window=30), A(heads=8, kv_heads=4, dim=16, rot_dims=4)],
                           loop=(0, 2, 3), side=8),
        # sizes off the 16-byte pieces, one head, a window of one token, more taps than the register kernels take, one pass
        "odd": dict(layers=[D(heads=3, kv_heads=1, dim=7, vdim=5, conv=6, ff=11), L(heads=1, dim=3, rot_dim=2, vdim=5, kv_rank=7, q_rank=3, window=1, ff=7),
                            A(heads=3, kv_heads=1, dim=7, rot_dims=2, ff=5)], side=5, loop=(1, 3, 1)),
        "no_side": dict(layers=[D(conv=1), L(window=200), A()], side=0, loop=(0, 3, 2)),
        "no_loop": dict(layers=[L(heads=4, dim=16, rot_dim=8, vdim=24, kv_rank=32, q_rank=16, window=16), A(heads=1, kv_heads=1, dim=6, rot_dims=6), D()], side=16),
        "delta_only": dict(layers=[D(heads=4, kv_heads=4), D(heads=8, kv_heads=2, dim=16, vdim=24)], loop=(1, 2, 4)),
    }


def model_set(name, width):
    spec = dict(layer_sets()[name])
    return O.make_config(spec.pop("layers"), width=width, **spec)


@pytest.mark.parametrize("name,width", [("mixed", 40), ("mixed", 64), ("loop_first", 48), ("odd", 30), ("odd", 37), ("no_side", 33), ("no_loop", 64), ("delta_only", 32)])
def test_model_whole_prompt_against_oracle(tmp_path, name, width):
    cfg = model_set(name, width)
    W = O.random_model(cfg, seed=len(name) + width)
    toks = tokens(75, cfg["vocab"], 5)
    lo = []
    want = O.forward(cfg, W, toks, lo)
    m = load(tmp_path, cfg, W, F32)
    for impl in (0, 2, 3):                  # the delta rule by step, token by token, in chunks
        for fused in ((None, True) if impl == 0 else (None,)):
            m.scan_impl, m.fused_side, m.layer_trace = impl, fused, None if fused else []
            seq = m.new_sequence()
            got = m.step([(seq, toks)], [list(range(len(toks)))])
            if not fused:
                assert len(m.layer_trace) == len(lo)
                for i, (a, b) in enumerate(zip(m.layer_trace, lo)):
                    close(a, b, 3e-5, f"{name}: stream after run {i}, scan {impl}")
            close(got, want, 5e-5, f"{name}: logits, scan {impl}, one launch per layer end {fused}")
            seq.free()
    m.layer_trace, m.scan_impl, m.fused_side = None, 0, None
    seq = m.new_sequence()                  # prompt, then token by token
    got = torch.cat([m.step([(seq, toks[:20])], [list(range(20))])] + [m.step([(seq, [t])]) for t in toks[20:]])
    close(got, want, 5e-5, f"{name}: decoded")
    mb = load(tmp_path, cfg, W, BF16, "b")
    close_rows(mb.step([(mb.new_sequence(), toks)], [list(range(len(toks)))]), want, 6e-2, f"{name}: bfloat16 logits")


@pytest.mark.parametrize("dtype,tol", [(F32, 5e-5), (BF16, 6e-2)])
def test_portions_decoding_batches_and_slot_reuse(tmp_path, dtype, tol):
    """One set of sequences run whole, in portions of several sizes down to two tokens, token by token (through the replayed graph), in unequal
    batches whose shorter members leave early, and through slots that were used before.  Windows of 11 and 20 tokens end inside portions, the looped layers keep a state per pass."""
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
    """Head sizes the tensor-core kernels serve, prompts in portions of 16 tokens and more, windows of 24 and 70 tokens, an unequal batch."""
    A, D, L = O.attention_layer, O.delta_layer, O.latent_layer
    cfg = O.make_config([D(heads=4, kv_heads=2, dim=32, vdim=32), L(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=32, window=24), A(heads=4, kv_heads=2, dim=64, rot_dims=32),
                         L(heads=2, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=48, window=70, ff=0)], width=96, side=16, loop=(0, 3, 2))
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


def test_long_decoding_windows_pass_and_the_pool_grows(tmp_path):
    """300 tokens decoded one by one after a short prompt: windows of 44 and 100 tokens pass over decoded tokens, the pool grows while the sequence
    lives (captured graphs are rebuilt, the full attention splits its keys), a second sequence joins and leaves."""
    A, D, L = O.attention_layer, O.delta_layer, O.latent_layer
    cfg = O.make_config([L(window=44), A(heads=2, kv_heads=1, dim=16, rot_dims=8), D(), L(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=16, q_rank=8, window=100, ff=0)], loop=(1, 3, 2))
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
    channels, a window far shorter than the prompt, whose context is expanded from inside the prompt, decoding that splits the keys."""
    A, D, L = O.attention_layer, O.delta_layer, O.latent_layer
    cfg = O.make_config([D(heads=4, kv_heads=2, dim=128, vdim=64, ff=256), L(heads=6, dim=32, rot_dim=32, vdim=64, kv_rank=96, q_rank=64, window=200, base=10000.0, scale=0.2, ff=256),
                         A(heads=8, kv_heads=2, dim=64, rot_dims=64, base=10000.0, scale=0.2, ff=256), L(heads=2, dim=64, rot_dim=16, vdim=32, kv_rank=64, q_rank=40, window=520, ff=0)],
                        width=192, vocab=300, side=32, loop=(1, 3, 2))
    W = O.random_model(cfg, seed=21)
    toks = tokens(1320, 300, 4)
    rows = sorted(list(range(0, 1300, 97)) + [399, 400, 511, 512, 1023, 1024, 1297, 1298, 1299])
    want = O.forward(cfg, W, toks)
    for dtype in (F32, BF16):
        m = load(tmp_path, cfg, W, dtype, str(dtype)[-4:])
        for cuts in ([1300], [700, 600], [3, 1200, 97]):
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
    from promptcache_b200.model import Zepilix
    cfg = model_set("mixed", 48)
    W = O.random_model(cfg, seed=5)
    prompts = [tokens(n, cfg["vocab"], 40 + n) for n in (12, 3, 25)]
    n_new = 10
    want = [O.greedy(cfg, W, p, n_new) for p in prompts]
    folder = str(tmp_path / "g")
    write_checkpoint(folder, cfg, W)
    lm = Zepilix(folder, device=DEV, dtype=F32)
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
    cfg = model_set("loop_first", 48)
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
