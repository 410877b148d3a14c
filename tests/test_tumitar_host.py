"""CPU tests of the Tumitar family's host side: config parser and registry, cache storage, and the float64 restatement on cases worked out by
hand."""
import math

import pytest
import torch

from tests import tumitar_oracle as O
from tests.tumitar_util import dense, make_config, make_weights, moe, side_layer, unit_layer

F64 = torch.float64


def test_parser_and_registry():
    from qserve_b200.modelcfg import ARCHITECTURES, AttentionMixerConfig, GatedUnitMixerConfig, MlpConfig, MoeConfig, ParallelMixerConfig, StateSpaceMixerConfig

    cfg = make_config([side_layer(heads=6, kv_heads=3, dim=8, vdim=10, coef=0.2, every=7, scale=0.4, left_scale=0.9, right_scale=0.1, sheads=10, state=9, svdim=6,
                                  groups=5, conv=3, norm_groups=4, mlp=moe(5, 3, 11, 0.25)), unit_layer(30, 5, 2, dense(9)), unit_layer(mlp=None)],
                      loop=(0, 2, 3), scale=7.5)
    c = ARCHITECTURES["Tumitar"](cfg)
    assert c.architecture == "Tumitar" and c.block == "sequential" and c.streams == 0 and c.norm_kind == "rms" and c.norm_offset == 0.0 and c.norm_groups == 1
    assert c.tied_head and c.loop_add and not c.loop_in and c.embed_scale == 7.5 and c.logit_scale == 1.0 and c.logit_softcap == 0.0 and c.pair_buckets == 0
    assert c.schedule() == [0, 1, 0, 1, 0, 1, 2] and c.pass_starts() == [0, 2, 4]
    m = c.layers[0].mixer
    assert isinstance(m, ParallelMixerConfig) and not m.branch_norm and (m.left_scale, m.right_scale) == (0.9, 0.1)
    a, s = m.left, m.right
    assert isinstance(a, AttentionMixerConfig) and (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.temp_coef, a.temp_every) == (6, 3, 8, 10, 0.4, 0.2, 7.0)
    assert a.rot is None and a.bias and a.row_norm and a.sink_score == 0.0 and a.maps == 1 and a.window == a.chunk == 0
    assert not (a.qk_norm or a.qk_gain or a.head_temp or a.sink or a.out_bias or a.head_gate or a.gate_wide or a.value_norm or a.tied_values)
    assert isinstance(s, StateSpaceMixerConfig) and (s.heads, s.state, s.vdim, s.groups, s.conv, s.norm_groups) == (10, 9, 6, 5, 3, 4)
    f = c.layers[0].mlp
    assert isinstance(f, MoeConfig) and (f.experts, f.top, f.ff, f.weight_scale) == (5, 3, 11, 0.25) and f.limit == math.inf and f.alpha == 1.0 and f.up_shift == 0.0
    assert f.router == "sigmoid" and not (f.renormalize or f.correction or f.shared_ff) and f.groups == f.keep == 1
    u = c.layers[1].mixer
    assert isinstance(u, GatedUnitMixerConfig) and (u.width, u.blocks, u.conv, u.decay_rate) == (30, 5, 2, 8.0)
    d = c.layers[1].mlp
    assert isinstance(d, MlpConfig) and d.ff == 9 and not d.gated and not d.bias and d.act == "relu2" and c.layers[2].mlp is None
    assert ARCHITECTURES["Tumitar"](make_config([unit_layer()])).pass_starts() == []


def test_parser_rejects_what_it_does_not_know():
    from qserve_b200.modelcfg import ARCHITECTURES

    parse = ARCHITECTURES["Tumitar"]
    for bad in (dict(unit_layer(), type="gla"), unit_layer(mlp={"kind": "other"}), unit_layer(width=36, blocks=5), side_layer(heads=4, kv_heads=3),
                side_layer(sheads=4, groups=3), side_layer(norm_groups=5), unit_layer(mlp=moe(4, 5))):
        with pytest.raises(ValueError):
            parse(make_config([bad]))


def test_other_families_keep_their_defaults():
    from qserve_b200.modelcfg import ARCHITECTURES
    from tests.nagosun_util import attention_layer, make_config as nagosun_config
    from tests.nusuvik_util import make_config as nusuvik_config

    c = ARCHITECTURES["Nagosun"](nagosun_config([attention_layer()]))
    assert not (c.tied_head or c.loop_add or c.layers[0].mixer.row_norm) and c.layers[0].mixer.temp_coef == 0.0
    assert ARCHITECTURES["Nusuvik"](nusuvik_config([])).loop_add is False


def test_cache_storage_and_release():
    from qserve_b200.cache import HybridCache
    from qserve_b200.modelcfg import ARCHITECTURES

    c = ARCHITECTURES["Tumitar"](make_config([side_layer(heads=4, kv_heads=2, dim=8, vdim=6, sheads=3, state=5, svdim=7, groups=1, conv=4, norm_groups=1),
                                              unit_layer(20, 2, 1)], loop=(0, 1, 2)))
    cache = HybridCache(c, torch.float32, torch.device("cpu"), max_tokens=200, max_seqs=3, page_size=16)
    assert len(cache.runs) == 3   # a looped layer has storage per pass
    for run in cache.runs[:2]:
        assert tuple(run["left"]["k"].shape) == (13, 16, 2, 8) and tuple(run["left"]["v"].shape) == (13, 16, 2, 6)
        assert tuple(run["right"]["state"].shape) == (3, 3, 5, 7) and tuple(run["right"]["conv"].shape) == (3, 3, 3 * 7 + 2 * 5)
    assert tuple(cache.runs[2]["state"].shape) == (3, 20) and cache.runs[2]["state"].dtype == torch.float32
    assert cache.runs[0]["right"]["state"].data_ptr() != cache.runs[1]["right"]["state"].data_ptr()
    cache.admit("a")
    cache.reserve("a", 40)
    assert cache.free_pages() == 10
    cache.release("a")
    assert cache.free_pages() == 13 and cache.can_admit()


# ------------------------------------------------------------------------------------------------------------------------
# the restatement by hand
# ------------------------------------------------------------------------------------------------------------------------
def test_oracle_convolution_by_hand():
    x = torch.tensor([[1.0, 10.0], [2.0, 20.0], [4.0, 40.0]], dtype=F64)
    taps = torch.tensor([[100.0, 10.0, 1.0], [0.0, 0.0, 2.0]], dtype=F64)   # the last column weighs the current token
    y = O.short_conv(x, taps, torch.tensor([0.5, 0.0], dtype=F64))
    assert y.tolist() == [[1.5, 20.0], [12.5, 40.0], [124.5, 80.0]]


def test_oracle_query_temperature_by_hand():
    t = O.query_temperature(9, 0.5, 4)
    assert t[:3].tolist() == [1.0] * 3   # positions 0 .. 2: floor((p + 1) / 4) is 0
    assert t[3:7].tolist() == pytest.approx([1 + 0.5 * math.log(2.0)] * 4) and t[7:].tolist() == pytest.approx([1 + 0.5 * math.log(3.0)] * 2)


def test_oracle_spare_term_by_hand():
    p = O.softmax_plus_one(torch.tensor([[0.0, 9.0], [-800.0, 700.0]], dtype=F64))
    assert p[0].tolist() == pytest.approx([0.5, 0.0]) and p[1].tolist() == pytest.approx([0.0, 1.0])
    low = O.softmax_plus_one(torch.tensor([[-700.0]], dtype=F64))
    assert 0.0 < float(low[0, 0]) < 1e-300


def test_oracle_attention_norms_rows_not_heads():
    """Two heads whose parts of the q row differ in size keep that difference: the row has one root mean square."""
    m = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0, "q_temp": {"coef": 0.0, "every": 1}}
    one, zero = torch.ones(1, dtype=F64), torch.zeros(1, dtype=F64)
    w = {"q": torch.tensor([[1.0], [7.0]], dtype=F64), "q.b": torch.zeros(2, dtype=F64), "q.norm": torch.tensor([1.0, 2.0], dtype=F64), "k": one[None], "k.b": zero,
         "k.norm": 3 * one, "v": one[None], "v.b": 4 * one, "o": torch.eye(2, dtype=F64)}
    got = O.attention(torch.tensor([[1.0]], dtype=F64), m, w, 0.0)[0]   # q = (1, 7) / 5, k = 1
    for g, s in zip(got.tolist(), (3 * 1 / 5, 3 * 2 * 7 / 5)):
        assert g == pytest.approx(5.0 * math.exp(s) / (1 + math.exp(s)))


def test_oracle_state_space_by_hand():
    """One head, one state row, no convolution memory: the second output holds the first input, decayed once."""
    m = {"heads": 1, "state": 1, "vdim": 1, "groups": 1, "norm_groups": 1}
    w = {"in": torch.tensor([[1.0], [1.0], [1.0], [1.0], [0.0]], dtype=F64), "conv": torch.ones(3, 1, dtype=F64), "conv.b": torch.zeros(3, dtype=F64),
         "dt_bias": torch.tensor([0.3], dtype=F64), "A_log": torch.tensor([-0.4], dtype=F64), "D": torch.tensor([2.0], dtype=F64), "norm": torch.ones(1, dtype=F64),
         "o": torch.ones(1, 1, dtype=F64)}
    h = torch.tensor([[0.5], [-1.5]], dtype=F64)
    s = [float(v) / (1 + math.exp(-float(v))) for v in h]
    dt = math.log1p(math.exp(0.3))
    S0 = dt * s[0] * s[0]
    S1 = math.exp(-math.exp(-0.4) * dt) * S0 + dt * s[1] * s[1]
    eps = 0.7   # large, so that the norm of a single number keeps its size
    for got, S, c in zip(O.state_space(h, m, w, eps)[:, 0].tolist(), (S0, S1), s):
        y = (S * c + 2.0 * c) * c
        assert got == pytest.approx(y / math.sqrt(y * y + eps))


def test_oracle_gated_unit_by_hand():
    m = {"blocks": 1}
    one, zero = torch.ones(1, dtype=F64), torch.zeros(1, dtype=F64)
    w = {"y": one[None], "y.b": zero, "x": one[None], "x.b": one, "conv": one[None], "conv.b": zero, "ra": one[None, None], "ra.b": zero[None], "ri": -one[None, None],
         "ri.b": zero[None], "lam": -2.0 * one, "o": one[None]}
    h, S = [0.5, 2.0], 0.0
    got = O.gated_linear_unit(torch.tensor(h, dtype=F64)[:, None], m, w, 0.0)[:, 0].tolist()
    for x, y in zip(h, got):
        u, sig = x + 1.0, lambda z: 1 / (1 + math.exp(-z))
        a = math.exp(-8.0 * sig(u) * math.log1p(math.exp(-2.0)))
        S = a * S + math.sqrt(1 - a * a) * sig(-u) * u   # the first token has no special case
        assert y == pytest.approx(S * 0.5 * x * (1 + math.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3))))


def test_oracle_experts_by_hand():
    w = {"router": torch.tensor([[0.0], [2.0], [1.0]], dtype=F64)}
    for e in range(3):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = torch.ones(1, 1, dtype=F64), torch.full((1, 1), 10.0 ** e, dtype=F64), torch.ones(1, 1, dtype=F64)
    sig = lambda z: 1 / (1 + math.exp(-z))
    got = float(O.experts_ff(torch.ones(1, 1, dtype=F64), moe(3, 2, 1, 1.5), w))
    assert got == pytest.approx(1.5 * sig(1.0) * (sig(2.0) * 10 + sig(1.0) * 100))   # scores as they are: not divided by their sum


def test_oracle_loop_and_causality():
    assert O.layer_runs(make_config([unit_layer()] * 4, loop=(1, 3, 3))) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    cfg = make_config([side_layer(), unit_layer(mlp=moe())], loop=(0, 1, 2))
    w = make_weights(cfg, 5, sharp=2.0)
    toks = [3, 9, 1, 44, 7, 7, 20]
    full = O.forward(cfg, w, toks)
    assert torch.allclose(O.forward(cfg, w, toks[:4]), full[:4], atol=1e-12)
    assert float((O.forward(cfg, w, [4] + toks[1:])[6] - full[6]).norm()) > 1e-6   # the first token is not forgotten
