"""Host-side parts of the Zepilix design that need no GPU: the configuration reader, the registry, the order of layer runs, the pool's layout with a
state per run, and the oracle's own consistency (causality, windows, loops, the delta rule in chunks)."""
import pytest
import torch

from tests import zepilix_oracle as O

F64 = torch.float64


def test_config_reader_and_registry():
    from promptcache_b200.model import MODEL_REGISTRY, Zepilix  # noqa: F401
    from promptcache_b200.model.zepilix import ZepilixConfig
    assert "Zepilix" in MODEL_REGISTRY
    cfg = ZepilixConfig(O.make_config([O.delta_layer(), O.latent_layer(ff=0), O.attention_layer()], width=48, side=10, loop=(1, 3, 3), eps=1e-4))
    assert (cfg.width, cfg.num_hidden_layers, cfg.eps, cfg.side_dim) == (48, 3, 1e-4, 10)
    assert cfg.runs == [0, 1, 2, 1, 2, 1, 2] and cfg.passes == {1: 0, 3: 1, 5: 2}
    assert cfg.layers[1]["mlp"] is None and cfg.layers[0]["mlp"]["kind"] == "dense"
    plain = ZepilixConfig(O.make_config([O.attention_layer()], side=0))
    assert plain.runs == [0] and plain.passes == {} and plain.side_dim == 0
    for key, value in (("type", "conv"), ("mlp", {"kind": "moe"})):
        bad = O.make_config([O.attention_layer()])
        bad["layers"][0][key] = value
        with pytest.raises(ValueError):
            ZepilixConfig(bad)
    with pytest.raises(ValueError):
        ZepilixConfig(O.make_config([O.attention_layer()], loop=(0, 2, 2)))


def test_runs_match_the_oracle():
    from promptcache_b200.model.zepilix import ZepilixConfig
    for n, loop in ((4, None), (4, (0, 4, 1)), (4, (0, 2, 3)), (5, (2, 5, 2)), (5, (1, 2, 4)), (3, (2, 3, 2))):
        cfg = O.make_config([O.delta_layer() for _ in range(n)], loop=loop)
        got, want = ZepilixConfig(cfg), O.run_order(cfg)
        assert got.runs == [i for i, _ in want]
        assert got.passes == {r: t for r, (_, t) in enumerate(want) if t is not None}


def test_pool_layout_with_a_state_per_run():
    from promptcache_b200.model._state import ConvTailSpec, DecayStateSpec, KVSpec, LatentKVSpec, SeqState, SlotPool
    delta, full, latent = (DecayStateSpec(4, 6, 5), ConvTailSpec(3, 44, "conv_tail")), KVSpec(2, 6, 6), LatentKVSpec(12, 4)
    pool = SlotPool([delta, latent, delta, latent, full], torch.bfloat16, "cpu", n_slots=1, cap=128)
    assert [set(x) for x in pool.layers] == [{"s", "conv_tail"}, {"ckv"}, {"s", "conv_tail"}, {"ckv"}, {"k", "v"}]
    assert tuple(pool.layers[2]["s"].shape) == (1, 4, 6, 5) and tuple(pool.layers[3]["ckv"].shape) == (1, 1, 128, 16) and pool.layers[0]["s"].dtype == torch.float32
    a = SeqState(pool)
    pool.layers[0]["s"][a.slot], pool.layers[2]["s"][a.slot], pool.layers[3]["ckv"][a.slot] = 1.0, 2.0, 3.0
    b = SeqState(pool)                       # the pool doubles, then its rows grow: what live slots hold is carried over, run by run
    pool.reserve(b.slot, 300)
    assert pool.n_slots == 2 and pool.cap >= 300
    assert float(pool.layers[0]["s"][a.slot].min()) == 1.0 and float(pool.layers[2]["s"][a.slot].min()) == 2.0 and float(pool.layers[3]["ckv"][a.slot, :, :128].float().min()) == 3.0


def test_oracle_is_causal_and_loops_matter():
    cfg = O.make_config([O.delta_layer(conv=3), O.latent_layer(window=3), O.attention_layer(), O.delta_layer(ff=0)], width=24, loop=(1, 3, 2))
    W = O.random_model(cfg, seed=1)
    toks = [3, 9, 27, 20, 1, 2, 3, 4, 5, 6, 7, 8]
    full = O.forward(cfg, W, toks)
    assert torch.allclose(O.forward(cfg, W, toks[:7]), full[:7], atol=1e-12)
    # one pass more, another vector of a pass, another part of the side table: all of them show
    assert not torch.allclose(O.forward(dict(cfg, loop=dict(cfg["loop"], times=1)), W, toks), full, atol=1e-3)
    for name, where in (("loop.step", (1, slice(None))), ("side.embed", (slice(None), slice(6, 12)))):
        W2 = {k: v.clone() for k, v in W.items()}
        W2[name][where] += 0.5
        assert not torch.allclose(O.forward(cfg, W2, toks), full, atol=1e-3), name


def test_oracle_window_edges():
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(1, 2, 4, generator=g, dtype=F64), torch.randn(8, 1, 4, generator=g, dtype=F64), torch.randn(8, 1, 3, generator=g, dtype=F64)
    pq, pk = torch.tensor([6]), torch.arange(8)
    o = O.softmax_attention(q, k, v, pq, pk, 0.5, window=3)
    for at, seen in ((3, False), (4, True), (6, True), (7, False), (0, False)):
        v2 = v.clone()
        v2[at] += 100.0
        assert torch.equal(O.softmax_attention(q, k, v2, pq, pk, 0.5, window=3), o) != seen


def test_unit_heads_do_not_feel_the_order_of_norm_and_turn():
    """A turn keeps a head's root mean square, so the product takes the norm first."""
    g = torch.Generator().manual_seed(4)
    t, pos = torch.randn(5, 3, 10, generator=g, dtype=F64), torch.tensor([0, 1, 7, 500, 90000])
    a, b = O.unit_rms(O.rotate_pairs(t, pos, 6, 100.0), 1e-5), O.rotate_pairs(O.unit_rms(t, 1e-5), pos, 6, 100.0)
    assert torch.allclose(a, b, atol=1e-12)


def test_delta_rule_in_chunks_is_the_recurrence():
    """What the chunked kernels compute with one decay per head, in float64: plain products scaled pair by pair, corrections from a triangular
    system, states from chunk to chunk."""
    g = torch.Generator().manual_seed(2)
    T, D, V, C = 22, 5, 4, 8
    q, k, v = torch.randn(T, 1, D, generator=g, dtype=F64), O.unit_vector(torch.randn(T, 1, D, generator=g, dtype=F64)), torch.randn(T, 1, V, generator=g, dtype=F64)
    ld, beta = -torch.rand(T, 1, generator=g, dtype=F64), torch.rand(T, 1, generator=g, dtype=F64)
    want, S_want = O.delta_recurrence(q, k, v, ld, beta)
    S, out = torch.zeros(D, V, dtype=F64), []
    for c in range(0, T, C):
        qc, kc, vc, bc = q[c:c + C, 0], k[c:c + C, 0], v[c:c + C, 0], beta[c:c + C]
        B = torch.cumsum(ld[c:c + C], 0)
        E = torch.exp(B - B.T)
        M = torch.eye(len(qc), dtype=F64) + bc * (kc @ kc.T * E).tril(-1)
        u = torch.linalg.solve(M, bc * vc) - torch.linalg.solve(M, bc * kc * torch.exp(B)) @ S
        out.append((qc * torch.exp(B)) @ S + (qc @ kc.T * E).tril() @ u)
        S = torch.exp(B[-1]) * S + (kc * torch.exp(B[-1] - B)).T @ u
    assert torch.allclose(torch.cat(out), want[:, 0], atol=1e-12) and torch.allclose(S, S_want[0], atol=1e-12)


def test_oracle_pieces_by_hand():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    assert torch.allclose(O.stream_norm(x, torch.tensor([0.0, 1.0], dtype=F64), 0.0), torch.tensor([[3.0, 8.0]], dtype=F64) / (12.5 ** 0.5))
    c = O.causal_conv(torch.tensor([[1.0], [10.0], [100.0]], dtype=F64), torch.tensor([[0.5, 2.0]], dtype=F64))
    assert c[:, 0].tolist() == [2.0, 20.5, 205.0]
    one = torch.ones(1, 1, dtype=F64)
    assert float(O.side_input(one, one * -2.0, one, one * 3.0, one * 0.5, 0.0)) == -0.5      # a norm over one number keeps its sign
