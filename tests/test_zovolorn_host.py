"""Host-side parts of the Zovolorn design that need no GPU: the configuration reader, the registry, the distance buckets, the pool's layout for
layers with several convolutions, and the oracle's own consistency (causality, chunks, the delta rule in chunks)."""
import math

import pytest
import torch

from tests import zovolorn_oracle as O

F64 = torch.float64


def test_config_reader_and_registry():
    from promptcache_b200.model import MODEL_REGISTRY, Zovolorn  # noqa: F401
    from promptcache_b200.model.zovolorn import ZovolornConfig
    assert "Zovolorn" in MODEL_REGISTRY
    cfg = ZovolornConfig(O.make_config([O.attention_layer(), O.parallel_layer(ff=0)], width=48, embed_scale=2.25, groups=6, taps=4, cap=9.0))
    assert (cfg.width, cfg.num_hidden_layers, cfg.embedding_scale, cfg.eps, cfg.groups, cfg.taps, cfg.softcap) == (48, 2, 2.25, 1e-5, 6, 4, 9.0)
    assert cfg.layers[1]["mlp"] is None and cfg.layers[0]["mlp"]["kind"] == "dense" and cfg.bigram["buckets"] == 37
    bad = O.make_config([O.attention_layer()])
    bad["layers"][0]["type"] = "conv"
    with pytest.raises(ValueError):
        ZovolornConfig(bad)
    bad = O.make_config([O.attention_layer()])
    bad["layers"][0]["mlp"]["kind"] = "moe"
    with pytest.raises(ValueError):
        ZovolornConfig(bad)
    with pytest.raises(ValueError):
        ZovolornConfig(O.make_config([O.attention_layer()], width=30, groups=4))


def test_distance_buckets():
    """The product's buckets (logarithms) against whole-number arithmetic, also where a distance sits exactly on a border."""
    from promptcache_b200.model.zovolorn import distance_bucket
    for n_buckets in (2, 6, 8, 12, 16, 32, 64):
        for far in (1, 5, 14, 48, 64, 96, 100, 128, 250, 256, 512, 1000):
            got = [distance_bucket(n, n_buckets, far) for n in range(far + 50)]
            assert got == [O.distance_bucket(n, n_buckets, far) for n in range(far + 50)], (n_buckets, far)
            assert got == sorted(got) and got[-1] == n_buckets - 1 and got[:n_buckets // 2] == list(range(n_buckets // 2))
    assert [distance_bucket(n, 8, 64) for n in (3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 900)] == [3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]   # powers of two are the borders


def test_pool_layout_with_several_convolutions():
    from promptcache_b200.model._state import ConvTailSpec, DecayStateSpec, KVSpec, SeqState, SlotPool
    specs = [(KVSpec(2, 6, 6), DecayStateSpec(3, 4, 5), ConvTailSpec(4, 21, "conv_tail"), ConvTailSpec(3, 16, "tail1"), ConvTailSpec(3, 16, "tail2")), (KVSpec(1, 8, 4), ConvTailSpec(3, 16))]
    pool = SlotPool(specs, torch.bfloat16, "cpu", n_slots=1, cap=128)
    assert set(pool.layers[0]) == {"k", "v", "s", "conv_tail", "tail1", "tail2"} and set(pool.layers[1]) == {"k", "v", "tail"}
    assert tuple(pool.layers[0]["conv_tail"].shape) == (1, 2, 3, 21) and tuple(pool.layers[0]["tail2"].shape) == (1, 2, 2, 16)
    a = SeqState(pool)
    for n in ("conv_tail", "tail1", "tail2", "s"):
        pool.layers[0][n][a.slot] = 3.0
    b = SeqState(pool)                       # the pool doubles, then its rows grow: what live slots hold is carried over
    pool.reserve(b.slot, 300)
    assert pool.n_slots == 2 and pool.cap >= 300
    for n in ("conv_tail", "tail1", "tail2", "s"):
        assert float(pool.layers[0][n][a.slot].min()) == 3.0


def test_oracle_is_causal_and_chunks_forget():
    cfg = O.make_config([O.parallel_layer(chunk=4), O.attention_layer(), O.parallel_layer(chunk=3, ff=0)], width=24, groups=3)
    W = O.random_model(cfg, seed=1)
    toks = [3, 9, 27, 20, 1, 2, 3, 4, 5, 6, 7, 8]
    full = O.forward(cfg, W, toks)
    assert torch.allclose(O.forward(cfg, W, toks[:7]), full[:7], atol=1e-12)
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(1, 2, 4, generator=g, dtype=F64), torch.randn(8, 2, 4, generator=g, dtype=F64), torch.randn(8, 2, 3, generator=g, dtype=F64)
    pq, pk = torch.tensor([7]), torch.arange(8)
    o = O.softmax_attention(q, k, v, pq, pk, 0.5, chunk=3)
    for at, seen in ((5, False), (6, True), (7, True), (0, False)):      # 7 // 3 = 2: positions 6 and 7
        v2 = v.clone()
        v2[at] += 100.0
        assert torch.equal(O.softmax_attention(q, k, v2, pq, pk, 0.5, chunk=3), o) != seen
    # a sink takes weight and gives nothing
    s = torch.tensor([50.0, -50.0], dtype=F64)
    os_ = O.softmax_attention(q, k, v, pq, pk, 0.5, sink=s)
    assert float(os_[0, 0].abs().max()) < 1e-15 and torch.allclose(os_[0, 1], O.softmax_attention(q, k, v, pq, pk, 0.5)[0, 1])


def test_delta_rule_in_chunks_is_the_recurrence():
    """What the chunked kernels compute, in float64: corrections from a triangular system, states from chunk to chunk."""
    g = torch.Generator().manual_seed(2)
    T, D, V, C = 22, 5, 4, 8
    q, k, v = torch.randn(T, 1, D, generator=g, dtype=F64), O.unit_vector(torch.randn(T, 1, D, generator=g, dtype=F64)), torch.randn(T, 1, V, generator=g, dtype=F64)
    ld, beta = -torch.rand(T, 1, D, generator=g, dtype=F64), torch.rand(T, 1, generator=g, dtype=F64)
    want, S_want = O.delta_recurrence(q, k, v, ld, beta)
    S, out = torch.zeros(D, V, dtype=F64), []
    for c in range(0, T, C):
        qc, kc, vc, bc = q[c:c + C, 0], k[c:c + C, 0], v[c:c + C, 0], beta[c:c + C]
        B = torch.cumsum(ld[c:c + C, 0], 0)
        E = torch.exp(B[:, None] - B[None])                                   # [i, s, channel]
        A = torch.einsum("id,sd,isd->is", kc, kc, E).tril(-1)
        Q = torch.einsum("id,sd,isd->is", qc, kc, E).tril()
        M = torch.eye(len(qc), dtype=F64) + bc * A
        u = torch.linalg.solve(M, bc * vc) - torch.linalg.solve(M, bc * kc * torch.exp(B)) @ S
        out.append((qc * torch.exp(B)) @ S + Q @ u)
        S = torch.exp(B[-1])[:, None] * S + (kc * torch.exp(B[-1] - B)).T @ u
    assert torch.allclose(torch.cat(out), want[:, 0], atol=1e-12) and torch.allclose(S, S_want[0], atol=1e-12)


def test_oracle_pieces_by_hand():
    assert O.pair_rows([4, 9], 10, 3, 2) == [10, (4 * 3 + 9 * 2) % 10]
    x = torch.tensor([[3.0, 4.0, 0.0, 2.0]], dtype=F64)
    n = O.grouped_norm(x, torch.tensor([1.0, 1.0, 1.0, 10.0], dtype=F64), 2, 0.0)
    assert torch.allclose(n, torch.tensor([[3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 0.0, 10 * 2 / math.sqrt(2.0)]], dtype=F64))
    c = O.causal_conv(torch.tensor([[1.0], [10.0], [100.0]], dtype=F64), torch.tensor([[0.5, 2.0]], dtype=F64))
    assert c[:, 0].tolist() == [2.0, 20.5, 205.0]
