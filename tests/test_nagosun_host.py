"""CPU tests of the Nagosun family's host side: config parser and registry, cache storage, the pages a windowed prompt portion lays out, and
the float64 restatement on cases worked out by hand."""
import math

import pytest
import torch

from tests import nagosun_oracle as O
from tests.nagosun_util import attention_layer, dense, latent_layer, make_config, make_weights


def test_parser_and_registry():
    from qserve_b200.modelcfg import ARCHITECTURES, AttentionMixerConfig, LatentAttentionMixerConfig, MlpConfig

    cfg = make_config([attention_layer(heads=6, kv_heads=3, dim=8, vdim=10, size=9, softcap=7.5, mlp=None), latent_layer(heads=1, dim=4, rot_dim=2, vdim=6, kv_rank=5, size=11, mlp=dense(9)),
                       attention_layer(size=0, softcap=0)], groups=4, mult=0.25, logit_scale=3.5)
    c = ARCHITECTURES["Nagosun"](cfg)
    assert c.architecture == "Nagosun" and c.block == "sandwich" and c.norm_kind == "rms" and c.norm_offset == 0.0 and c.norm_groups == 4
    assert c.residual_mult == 0.25 and c.residual_gate and c.embed_norm and c.logit_scale == 3.5 and c.logit_softcap == 0.0
    assert c.embed_scale == 1.0 and c.schedule() == [0, 1, 2] and c.pair_buckets == 0 and not c.layer_scale
    a = c.layers[0].mixer
    assert isinstance(a, AttentionMixerConfig) and (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.softcap) == (6, 3, 8, 10, 9, 7.5)
    assert a.rot is None and a.bias and a.out_bias and a.value_norm and a.gate_wide and a.sink_score == 0.0 and a.maps == 1 and a.keep_first == 0
    assert not (a.qk_norm or a.qk_gain or a.head_temp or a.sink or a.tied_values or a.head_gate or a.head_norm) and c.layers[0].mlp is None
    assert a.slopes() == pytest.approx([2.0 ** (-8.0 * (h + 1) / 6) for h in range(6)])
    m = c.layers[1].mixer
    assert isinstance(m, LatentAttentionMixerConfig) and (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank, m.window) == (1, 4, 2, 6, 5, 0, 11)
    assert m.rot.layout == "interleaved" and m.rot.factor is None and m.rot.dims == 2 and not (m.sink or m.gate or m.gate_wide)
    f = c.layers[1].mlp
    assert isinstance(f, MlpConfig) and f.gated and not f.bias and f.act == "silu" and f.ff == 9
    assert c.layers[2].mixer.window == 0 and c.layers[2].mixer.softcap == 0.0


def test_parser_rejects_what_it_does_not_know():
    from qserve_b200.modelcfg import ARCHITECTURES

    parse = ARCHITECTURES["Nagosun"]
    for bad in ([{"type": "gla", "mixer": {}, "mlp": None}], [attention_layer(mlp={"kind": "moe", "ff": 8})], [attention_layer(heads=4, kv_heads=3)]):
        with pytest.raises(ValueError):
            parse(make_config(bad))
    with pytest.raises(ValueError):
        parse(make_config([attention_layer()], width=44, groups=3))
    odd = latent_layer(rot_dim=4)
    odd["mixer"]["rot"]["dims"] = 6
    with pytest.raises(ValueError):
        parse(make_config([odd]))


def test_other_families_keep_their_defaults():
    from qserve_b200.modelcfg import ARCHITECTURES
    from tests.zuzezen_util import attention_layer as zuzezen_attention, make_config as zuzezen_config

    c = ARCHITECTURES["Zuzezen"](zuzezen_config([zuzezen_attention()]))
    a = c.layers[0].mixer
    assert c.block == "post" and not (c.residual_gate or c.embed_norm) and c.residual_mult == c.logit_scale == 1.0
    assert not (a.gate_wide or a.value_norm or a.out_bias) and a.softcap == 0.0 and a.sink_score is None


def test_cache_storage_and_release():
    from qserve_b200.cache import HybridCache
    from qserve_b200.modelcfg import ARCHITECTURES

    c = ARCHITECTURES["Nagosun"](make_config([latent_layer(kv_rank=10, rot_dim=2), attention_layer(heads=4, kv_heads=2, dim=8, vdim=6)]))
    cache = HybridCache(c, torch.float32, torch.device("cpu"), max_tokens=200, max_seqs=3, page_size=16)
    assert tuple(cache.runs[0]["c"].shape) == (13, 16, 12)
    assert tuple(cache.runs[1]["k"].shape) == (13, 16, 2, 8) and tuple(cache.runs[1]["v"].shape) == (13, 16, 2, 6)
    cache.admit("a")
    cache.reserve("a", 40)
    assert cache.free_pages() == 10
    cache.release("a")
    assert cache.free_pages() == 13 and cache.can_admit()


@pytest.mark.parametrize("page", [16, 64, 128])
def test_windowed_context_holds_the_visible_pages(page):
    """The run of pages a prompt portion lays out per step covers every position a window shows its tokens (to the key tile), not those
    before; entries of fewer tokens than a tile needs are not part of it."""
    from qserve_b200.hybrid import StepBatch

    n_blocks = 2048 // page
    table = (torch.randperm(3 * n_blocks, generator=torch.Generator().manual_seed(page)).to(torch.int32)).reshape(3, n_blocks)
    b = StepBatch.build([(2, 700, 1, [1] * 130), (0, 5, 1, [1]), (1, 0, -1, [1] * 40)], table, torch.device("cpu"), page)
    for window, first in ((0, 0), (1, 700), (100, 601), (701, 0), (5000, 0)):
        src, ctx = b.context(0, window)
        lo = first // 64 * 64 // page
        pages = list(range(lo, -(-830 // page)))
        assert src.tolist() == [int(table[2, i]) for i in pages] + [int(table[1, i]) for i in range(-(-40 // page))]
        for k, i in enumerate(pages):
            assert int(ctx[2, i]) == k
        assert int(ctx[1, 0]) == len(pages)
        assert b.context(0, window)[1] is ctx   # laid out once per mask
    src, _ = b.context(256, 0)   # chunks of 256: position 700 is in the chunk that starts at 512
    assert src.numel() == -(-830 // page) - 512 // page + -(-40 // page)
    assert StepBatch.build([(0, 5, 1, [1, 2])], table, torch.device("cpu"), page).context() is None


# ------------------------------------------------------------------------------------------------------------------------
# the restatement by hand
# ------------------------------------------------------------------------------------------------------------------------
def test_oracle_grouped_norm_by_hand():
    x = torch.tensor([[3.0, 4.0, 0.0, 2.0]], dtype=torch.float64)
    g = torch.tensor([1.0, 2.0, 5.0, 1.0], dtype=torch.float64)
    r = math.sqrt(12.5)
    assert torch.allclose(O.grouped_norm(x, g, 2, 0.0), torch.tensor([[3 / r, 8 / r, 0.0, math.sqrt(2.0)]], dtype=torch.float64))
    assert torch.allclose(O.grouped_norm(x, g, 1, 0.0), x / math.sqrt(29 / 4) * g)
    assert torch.allclose(O.grouped_norm(x, g, 4, 7.0), x / torch.sqrt(x * x + 7.0) * g)   # eps is inside the root


def test_oracle_turn_by_hand():
    x = torch.arange(18, dtype=torch.float64).reshape(3, 6)
    y = O.turn_neighbours(x, 10.0, 4)
    assert torch.equal(y[0], x[0]) and torch.equal(y[:, 4:], x[:, 4:])
    for i, a in ((0, 2.0), (1, 2.0 * 10.0 ** -0.5)):
        u, v = x[2, 2 * i], x[2, 2 * i + 1]
        assert float(y[2, 2 * i]) == pytest.approx(float(u) * math.cos(a) - float(v) * math.sin(a))
        assert float(y[2, 2 * i + 1]) == pytest.approx(float(v) * math.cos(a) + float(u) * math.sin(a))


def test_oracle_softmax_with_a_spare_term():
    s = torch.tensor([[0.0, 0.0, 900.0], [-800.0, -900.0, -1000.0], [1.0, 2.0, 3.0]], dtype=torch.float64)
    seen = torch.tensor([[True, True, False], [True, True, True], [True, False, True]])
    p = O.softmax_plus_one(s, seen)
    assert p[0].tolist() == pytest.approx([1 / 3, 1 / 3, 0.0])
    assert float(p[1].sum()) < 1e-300   # scores far below the spare term's 0: nothing is left for the keys
    e = [math.exp(1.0), math.exp(3.0)]
    assert p[2].tolist() == pytest.approx([e[0] / (1 + sum(e)), 0.0, e[1] / (1 + sum(e))])


def test_oracle_attention_by_hand():
    """One head, window of 2: at position 3 only positions 2 and 3 count; the cap comes ahead of the distance penalty; the value has unit RMS."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.5, "softcap": 2.0, "mask": {"size": 2}}
    eye, zero = torch.eye(2, dtype=torch.float64), torch.zeros(2, dtype=torch.float64)
    w = {"q": eye, "q.b": zero, "k": eye, "k.b": zero, "v": eye, "v.b": zero, "g": 0 * eye, "o": eye, "o.b": torch.tensor([10.0, 20.0], dtype=torch.float64)}
    h = torch.tensor([[5.0, 5.0], [9.0, 9.0], [1.0, 3.0], [2.0, 6.0]], dtype=torch.float64)
    s2, s3 = 2.0 * math.tanh(20 * 0.5 / 2.0) - 2.0 ** -8, 2.0 * math.tanh(40 * 0.5 / 2.0)
    v = torch.tensor([1.0, 3.0], dtype=torch.float64) / math.sqrt(5.0)   # positions 2 and 3 have the same direction
    share = (math.exp(s2) + math.exp(s3)) / (1.0 + math.exp(s2) + math.exp(s3))
    want = 0.5 * share * v + w["o.b"]
    assert torch.allclose(O.attention(h, m, w, 0.0)[3], want, atol=1e-12)


def test_oracle_window_and_causality():
    cfg = make_config([attention_layer(size=3), latent_layer(size=5), attention_layer(size=0, softcap=0)])
    w = make_weights(cfg, 5, sharp=2.0)
    toks = [3, 9, 1, 44, 7, 7, 20]
    full = O.forward(cfg, w, toks)
    assert torch.allclose(O.forward(cfg, w, toks[:4]), full[:4], atol=1e-12)
    for layer, reach in ((attention_layer(size=3, mlp=None), 3), (latent_layer(size=5, mlp=None), 5)):
        c1 = make_config([layer])
        w1 = make_weights(c1, 6, sharp=2.0)
        base = O.forward(c1, w1, toks)[6]
        for j in range(6):
            other = list(toks)
            other[j] += 1
            assert torch.equal(O.forward(c1, w1, other)[6], base) == (6 - j >= reach), j
