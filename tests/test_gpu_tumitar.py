"""GPU tests of the Tumitar family: the engine (model, page pool, slots, scheduler, kernels) against the plain float64 restatement in
tests/tumitar_oracle.py, on small random models of several shapes."""
import json
import math

import pytest
import torch

from tests import tumitar_oracle as O
from tests.hybrid_util import bf16_close, random_tokens, row_err
from tests.tumitar_util import dense, make_config, make_weights, moe, side_layer, unit_layer

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4   # float32 engine vs float64 oracle
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def _engine(cfg, w, dtype=torch.float32, max_tokens=1024, **kw):
    from qserve_b200.engine import Engine
    from qserve_b200.hybrid import HybridDecoder
    from qserve_b200.modelcfg import ARCHITECTURES

    model = HybridDecoder(ARCHITECTURES[cfg["architecture"]](cfg), w, dtype, torch.device("cuda:0"))
    return Engine(model, max_tokens=max_tokens, **kw)


def _whole(eng, sid, toks):
    out = eng.step([(sid, toks, list(range(len(toks))))])
    eng.release(sid)
    return out


def _portions(eng, sid, toks, sizes):
    """Feed toks in portions of the given sizes (cycled), wanting every position."""
    outs, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - at)
        outs.append(eng.step([(sid, toks[at:at + n], list(range(n)))]))
        at, i = at + n, i + 1
    return torch.cat(outs)


def _raw():
    return torch.cuda.current_stream().cuda_stream


def _bf(t):
    return t.to(torch.bfloat16).to(torch.float32)


def _close(got, want, dtype, routed=False):
    """routed: tokens choose experts, and bfloat16's rounding may turn a close choice -- of few tokens, whose rows then differ."""
    if dtype == torch.float32:
        return row_err(got, want) < F32_TOL
    if not routed:
        return bf16_close(got, want)
    got, want = got.double().cpu(), want.double().cpu()
    e = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    return float(e.median()) < 0.03 and float((e > 0.15).double().mean()) < 0.15


class _impl:
    """Keep the attention kernels on one implementation for a while (None: the engine's own choice)."""

    def __init__(self, attention=None):
        self.want = attention

    def __enter__(self):
        import qserve_b200.hybrid as hyb

        hyb.ATTENTION_IMPL = self.want

    def __exit__(self, *exc):
        import qserve_b200.hybrid as hyb

        hyb.ATTENTION_IMPL = None


STACK = [side_layer(), unit_layer(), side_layer(heads=6, kv_heads=3, dim=8, vdim=20, coef=0.2, every=17, sheads=3, state=9, svdim=7, groups=1, conv=3, norm_groups=1, mlp=moe()),
         unit_layer(width=20, blocks=1, conv=2, mlp=None), side_layer(heads=2, kv_heads=1, dim=24, vdim=8, sheads=2, state=33, svdim=16, conv=1, norm_groups=2, mlp=dense(24))]
LOOP = (1, 4, 2)


def _stack(dtype):
    """In bfloat16 the tokens use every expert: no close choice that rounding may turn."""
    return STACK if dtype == torch.float32 else [dict(l, mlp=moe(4, 4, 24, 0.4)) if l["mlp"] and l["mlp"]["kind"] == "moe" else l for l in STACK]


# ------------------------------------------------------------------------------------------------------------------------
# kernels alone
# ------------------------------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("H,G,D,Dv,coef,every,bias", [(4, 2, 16, 24, 0.5, 8.0, True), (3, 1, 5, 7, 0.0, 1.0, True), (1, 1, 1, 1, 0.3, 1.0, True), (32, 8, 128, 128, 0.1, 1000.0, True),
                                                      (6, 6, 10, 2, -0.2, 3.0, False), (2, 1, 64, 3, 0.7, 2.5, True)])
def test_row_norm_append_kernel(dev, dtype, H, G, D, Dv, coef, every, bias):
    """q in place, k and v in shuffled pages; positions on both sides of every step of the temperature."""
    from qserve_b200._lib import check, lib

    g = torch.Generator().manual_seed(H * D + G)
    NQ, NK, NV, page, T, eps = H * D, G * D, G * Dv, 16, 41, 1e-3
    stride = (NQ + NK + NV + 7) // 8 * 8
    rows = _bf(torch.randn(T, stride, generator=g) * 2.0)
    b, qg, kg = (torch.randn(n, generator=g) for n in (NQ + NK + NV, NQ, NK))
    pos = torch.arange(T) + 7
    table = torch.randperm(8, generator=g).to(torch.int32).reshape(2, 4)
    z = rows[:, :NQ + NK + NV].double() + (b.double() if bias else 0.0)
    temp = torch.tensor([1.0 + coef * math.log(math.floor((int(p) + 1) / every) + 1) for p in pos], dtype=torch.float64)
    want_q = O.rms_norm(z[:, :NQ], qg.double(), eps) * temp[:, None]
    want_k = O.rms_norm(z[:, NQ:NQ + NK], kg.double(), eps)
    proj = rows.to(dev).to(dtype)
    kp, vp = torch.zeros(8, page, NK, dtype=dtype, device=dev), torch.zeros(8, page, NV, dtype=dtype, device=dev)
    slot, posd, td = torch.ones(T, dtype=torch.int32, device=dev), pos.to(torch.int32).to(dev), table.to(dev)
    bd, qd, kd = b.to(dev), qg.to(dev), kg.to(dev)
    check(lib.qs_hyb_qk_row_norm_append(proj.data_ptr(), stride, bd.data_ptr() if bias else None, qd.data_ptr(), kd.data_ptr(), coef, every, slot.data_ptr(),
                                        posd.data_ptr(), td.data_ptr(), 4, kp.data_ptr(), vp.data_ptr(), eps, T, NQ, NK, NV, page,
                                        0 if dtype == torch.bfloat16 else 1, _raw()))
    tol = 2e-5 if dtype == torch.float32 else 2.0 ** -8
    near = lambda got, want: float(((got.double().cpu() - want).abs() / (want.abs() + 1.0)).max()) < tol
    cell = [(int(table[1, int(p) // page]), int(p) % page) for p in pos]
    assert near(proj[:, :NQ], want_q)
    assert near(torch.stack([kp[i, j] for i, j in cell]), want_k) and near(torch.stack([vp[i, j] for i, j in cell]), z[:, NQ + NK:])
    assert torch.equal(proj[:, NQ:].float().cpu(), rows[:, NQ:])   # the row's other parts stay as they were


@BOTH
@pytest.mark.parametrize("ff,pad,bias", [(40, 0, False), (33, 3, True), (1, 0, False), (4096, 8, True)])
def test_relu_squared_kernel(dev, dtype, ff, pad, bias):
    from qserve_b200._lib import check, lib

    g = torch.Generator().manual_seed(ff)
    x, b = _bf(torch.randn(5, ff + pad, generator=g) * 2.0), torch.randn(ff, generator=g)
    want = (x[:, :ff].double() + (b.double() if bias else 0.0)).clamp_min(0.0) ** 2
    xd, bd, out = x.to(dev).to(dtype), b.to(dev), torch.full((5, ff), 9.0, dtype=dtype, device=dev)
    check(lib.qs_hyb_bias_relu_squared(out.data_ptr(), ff, xd.data_ptr(), ff + pad, bd.data_ptr() if bias else None, 5, ff, 0 if dtype == torch.bfloat16 else 1, _raw()))
    assert float(((out.double().cpu() - want).abs() / (want + 1e-3)).max()) < (1e-5 if dtype == torch.float32 else 2.0 ** -8)


@pytest.mark.parametrize("T", [3, 600])
@pytest.mark.parametrize("experts,top,scale", [(6, 2, 1.5), (5, 5, 0.3), (1, 1, 2.0), (70, 33, 1.0)])
def test_router_weights_as_they_are(dev, T, experts, top, scale):
    from qserve_b200._lib import check, lib

    g = torch.Generator().manual_seed(experts)
    h, wr = torch.randn(T, 24, generator=g), torch.randn(experts, 24, generator=g)
    route, idx, wt = torch.empty(T, experts, device=dev), torch.empty(T, top, dtype=torch.int32, device=dev), torch.empty(T, top, device=dev)
    hd, wd = h.to(dev), wr.to(dev)
    check(lib.qs_hyb_moe_router(route.data_ptr(), idx.data_ptr(), wt.data_ptr(), hd.data_ptr(), wd.data_ptr(), T, 24, experts, top, 1, None, 1, 1, 0, scale, 1, _raw()))
    s = O.logistic(h.double() @ wr.double().T)
    val, order = torch.sort(s, descending=True)
    clear = torch.ones(T, dtype=torch.bool) if top == experts else (val[:, top - 1] - val[:, top] > 1e-5)   # tokens whose choice rounding cannot turn
    assert clear.sum() >= T * 9 // 10
    assert float((torch.sort(wt.double().cpu(), descending=True).values - scale * val[:, :top]).abs().max()) < 1e-5 * scale
    want = torch.zeros(T, experts, dtype=torch.float64).scatter(1, order[:, :top], scale * val[:, :top])
    assert float((route.double().cpu() - want)[clear].abs().max()) < 1e-5 * scale


# ------------------------------------------------------------------------------------------------------------------------
# every mechanism alone, through the engine
# ------------------------------------------------------------------------------------------------------------------------
LAYERS = [
    side_layer(mlp=None), side_layer(heads=1, kv_heads=1, dim=4, vdim=1, sheads=1, state=1, svdim=1, groups=1, conv=1, norm_groups=1, mlp=None),
    side_layer(heads=6, kv_heads=2, dim=10, vdim=33, every=1, sheads=6, state=48, svdim=9, groups=3, conv=5, norm_groups=6, mlp=None),
    side_layer(heads=3, kv_heads=3, dim=32, vdim=32, coef=0.0, left_scale=1.0, right_scale=1.0, sheads=8, state=64, svdim=40, groups=1, norm_groups=1, mlp=None),
    side_layer(heads=8, kv_heads=1, dim=16, vdim=16, left_scale=-0.5, sheads=2, state=100, svdim=72, groups=2, conv=2, norm_groups=1, mlp=None),
    side_layer(heads=2, kv_heads=2, dim=64, vdim=64, scale=0.2, sheads=5, state=128, svdim=130, groups=1, conv=4, norm_groups=5, mlp=None),
    side_layer(heads=4, kv_heads=4, dim=16, vdim=16, sheads=4, state=16, svdim=16, groups=4, conv=4, norm_groups=4, mlp=None),   # equal sizes everywhere
    side_layer(right_scale=0.0, mlp=None), side_layer(left_scale=0.0, sheads=3, state=300, svdim=5, groups=3, conv=17, norm_groups=1, mlp=None),
    unit_layer(mlp=None), unit_layer(width=1, blocks=1, conv=1, mlp=None), unit_layer(width=130, blocks=1, conv=3, mlp=None), unit_layer(width=44, blocks=44, conv=4, mlp=None),
    unit_layer(width=21, blocks=7, conv=17, mlp=None), unit_layer(width=512, blocks=4, conv=2, mlp=None),
]


def _layer_id(l):
    m = l["mixer"]
    parts = (m["left"], m["right"]) if l["type"] == "parallel" else (m,)
    return l["type"][:3] + "".join("-" + "x".join(str(v) for v in p.values() if isinstance(v, int)) for p in parts)


@pytest.mark.parametrize("layer", LAYERS, ids=_layer_id)
def test_single_layer(dev, layer):
    cfg = make_config([layer])
    w = make_weights(cfg, 2, sharp=2.0)
    toks = random_tokens(150, cfg["vocab"], 2)
    taps, layers = [], []
    eng = _engine(cfg, w)
    got = eng.step([("a", toks, list(range(len(toks))))], tap=lambda r, x: taps.append(x.clone()))
    want = O.forward(cfg, w, toks, layers)
    assert row_err(taps[0], layers[0]) < F32_TOL
    assert row_err(got, want) < F32_TOL
    eng.release("a")
    assert row_err(_portions(eng, "b", toks, [40, 1, 1, 2, 19]), want) < F32_TOL


@pytest.mark.parametrize("layer", [l for l in LAYERS if l["mixer"].get("width", 9) > 1 and l["mixer"].get("left", {}).get("vdim", 9) > 1], ids=_layer_id)
def test_single_layer_bf16(dev, layer):
    """(Without sizes whose norms see one number only: they keep a sign, which rounding may flip.)"""
    cfg = make_config([layer])
    w = make_weights(cfg, 2)
    toks = random_tokens(150, cfg["vocab"], 2)
    assert bf16_close(_portions(_engine(cfg, w, torch.bfloat16), "b", toks, [40, 1, 1, 2, 19, 80]), O.forward(cfg, w, toks))


@BOTH
@pytest.mark.parametrize("mlp", [dense(56), dense(1), dense(301), moe(), moe(1, 1, 8, 1.0), moe(5, 5, 7, 0.5), moe(4, 4, 8, 0.5), moe(40, 3, 16, 3.0)], ids=lambda m: json.dumps(m).replace(" ", ""))
def test_feed_forward_after_mixer(dev, mlp, dtype):
    cfg = make_config([unit_layer(mlp=mlp), side_layer(mlp=mlp)], width=48)
    w = make_weights(cfg, 3)
    toks = random_tokens(70, cfg["vocab"], 3)
    routed = mlp["kind"] == "moe" and mlp["router"]["top"] < mlp["router"]["experts"]
    assert _close(_whole(_engine(cfg, w, dtype), "a", toks), O.forward(cfg, w, toks), dtype, routed)


@BOTH
@pytest.mark.parametrize("kw", [dict(loop=LOOP), dict(loop=(0, 5, 2)), dict(loop=(2, 3, 4)), dict(loop=(4, 5, 1)), dict(loop=(1, 1, 3)), dict(scale=1.0), dict(scale=20.0), dict(eps=0.3),
                                dict(width=7, vocab=5), dict(width=128, vocab=131)], ids=str)
def test_constants_of_the_stack(dev, kw, dtype):
    cfg = make_config(_stack(dtype), **kw)
    w = make_weights(cfg, 4)
    toks = random_tokens(50, cfg["vocab"], 5)
    if dtype == torch.bfloat16 and (kw.get("width") == 7 or kw.get("loop", (0, 0, 1))[2] > 2):
        pytest.skip("few channels or many layer runs: rounding noise grows past a fixed bound")
    assert _close(_portions(_engine(cfg, w, dtype), "a", toks, [30, 1]), O.forward(cfg, w, toks), dtype)


def test_stack_and_taps(dev):
    cfg = make_config(STACK, width=52, vocab=131, loop=LOOP)
    w = make_weights(cfg, 4, sharp=2.0)
    toks = random_tokens(120, cfg["vocab"], 4)
    taps, layers = [], []
    got = _engine(cfg, w).step([("a", toks, list(range(len(toks))))], tap=lambda r, x: taps.append(x.clone()))
    want = O.forward(cfg, w, toks, layers)
    assert len(taps) == len(layers) == len(STACK) + 3
    for t, l in zip(taps, layers):
        assert row_err(t, l) < F32_TOL
    assert row_err(got, want) < F32_TOL


# ------------------------------------------------------------------------------------------------------------------------
# cuts, batches, reuse
# ------------------------------------------------------------------------------------------------------------------------
@BOTH
def test_prefill_against_token_by_token(dev, dtype):
    cfg = make_config(_stack(dtype), loop=LOOP)
    w = make_weights(cfg, 6, sharp=2.0 if dtype == torch.float32 else 1.0)   # peaked maps multiply bfloat16's rounding noise layer by layer
    toks = random_tokens(140, cfg["vocab"], 6)
    want = O.forward(cfg, w, toks)
    eng = _engine(cfg, w, dtype)
    whole = _whole(eng, "a", toks)
    single = _portions(eng, "b", toks, [1])   # from the first token on: graph replay from the second
    eng.release("b")
    assert _close(whole, want, dtype) and _close(single, want, dtype) and _close(single, whole, dtype)


@BOTH
@pytest.mark.parametrize("sizes", [[2], [3, 2, 7], [64], [63, 1, 65], [17, 100, 5, 2], [130, 2], [15, 16, 17]])
def test_portions(dev, sizes, dtype):
    """Portions shorter than the convolutions' memory, around the length from which rows run as tiles (16), around tiles (64), in the middle of
    pages (16)."""
    cfg = make_config(_stack(dtype), loop=LOOP)
    w = make_weights(cfg, 7, sharp=2.0 if dtype == torch.float32 else 1.0)
    toks = random_tokens(210, cfg["vocab"], 7)
    assert _close(_portions(_engine(cfg, w, dtype, page_size=16), "a", toks, sizes), O.forward(cfg, w, toks), dtype)


@BOTH
def test_mixed_batches_with_reuse(dev, dtype):
    """Unequal requests in one batch (portions beside single tokens) against each alone; four slots and a page pool that is far smaller than
    the sum of all requests, so that pages and slots are handed out again."""
    cfg = make_config(_stack(dtype), loop=LOOP)
    w = make_weights(cfg, 8, sharp=2.0 if dtype == torch.float32 else 1.0, slow=1.5)
    lens = [70, 33, 120, 5, 64, 97, 18, 2, 1, 50]
    reqs = {f"r{i}": random_tokens(n, cfg["vocab"], 20 + i) for i, n in enumerate(lens)}
    eng = _engine(cfg, w, dtype, max_tokens=4 * 128, page_size=16)
    alone = {k: O.forward(cfg, w, v) for k, v in reqs.items()}
    fed = {k: 0 for k in reqs}
    got = {k: [] for k in reqs}
    waiting, live, step = list(reqs), [], 0
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        entries = []
        for j, k in enumerate(live):
            left = len(reqs[k]) - fed[k]
            n = min(left, 1 if (step + j) % 3 == 0 and fed[k] > 0 else [29, 2, 64, 7][(step + j) % 4])
            if (step + j) % 5 == 4 and len(live) > 1:
                continue   # a live request may sit out a step
            entries.append((k, reqs[k][fed[k]:fed[k] + n], list(range(n))))
        out = eng.step(entries)
        r = 0
        for k, toks, want in entries:
            got[k].append(out[r:r + len(toks)])
            r += len(toks)
            fed[k] += len(toks)
        for k in [k for k in live if fed[k] == len(reqs[k])]:
            live.remove(k)
            eng.release(k)
        step += 1
    assert eng.cache.free_pages() == eng.cache.num_pages and len(eng.cache.seqs) == 0
    for k in reqs:
        assert _close(torch.cat(got[k]), alone[k], dtype), k


def test_used_slots_start_clean(dev):
    """A request's slots and pages are filled with large numbers before it starts: nothing of them shows, whether its first step is one token,
    shorter than the convolutions' memory, or a prompt."""
    cfg = make_config(STACK, loop=LOOP)
    w = make_weights(cfg, 18, slow=3.0)
    toks = random_tokens(40, cfg["vocab"], 18)
    want = O.forward(cfg, w, toks)
    eng = _engine(cfg, w, page_size=16)

    def spoil(t):
        for v in t.values():
            spoil(v) if isinstance(v, dict) else v.fill_(1e4)

    for sizes in ([1], [2, 1], [3, 20], [16], [40]):
        for run in eng.cache.runs:
            spoil(run)
        assert row_err(_portions(eng, "a", toks, sizes), want) < F32_TOL, sizes
        eng.release("a")


def test_long_decoding_and_graph_replay(dev):
    """Hundreds of single tokens through captured graphs against eager launches and the oracle; two sequences side by side."""
    cfg = make_config(STACK, loop=(0, 2, 2))
    w = make_weights(cfg, 9, sharp=2.0, slow=2.0)
    a, b = random_tokens(330, cfg["vocab"], 9), random_tokens(300, cfg["vocab"], 10)
    outs = {}
    for graphs in (True, False):
        eng = _engine(cfg, w, use_graphs=graphs, page_size=16)
        eng.step([("a", a[:30], []), ("b", b[:1], [])])
        rows = []
        for i in range(299):
            rows.append(eng.step([("a", a[30 + i:31 + i], [0]), ("b", b[1 + i:2 + i], [0])]))
        outs[graphs] = torch.stack(rows)
        assert eng.use_graphs == graphs   # no capture failed
    assert torch.equal(outs[True], outs[False])
    wa, wb = O.forward(cfg, w, a[:329]), O.forward(cfg, w, b)
    assert row_err(outs[True][:, 0], wa[30:]) < F32_TOL and row_err(outs[True][:, 1], wb[1:]) < F32_TOL


# ------------------------------------------------------------------------------------------------------------------------
# far tokens, the first tokens, needles
# ------------------------------------------------------------------------------------------------------------------------
FAR_LAYERS = {"attention": side_layer(heads=8, kv_heads=2, dim=16, vdim=16, right_scale=0.0, mlp=None), "state space": side_layer(left_scale=0.0, mlp=None),
              "gated unit": unit_layer(mlp=None)}


@pytest.mark.parametrize("far", [0, 1, 3, 15, 16, 17, 63, 64, 300])
@pytest.mark.parametrize("kind", list(FAR_LAYERS))
def test_far_token_is_seen(dev, far, kind):
    """A long prompt whose token at `far` (first positions, page, tile and portion borders) is changed: the oracle's answer at the last positions
    moves by a small but definite amount, and the engine's distance to the right answer is a small fraction of that move -- in a prompt
    portion and for decoded tokens.  The recurrent layers' states barely forget."""
    cfg = make_config([FAR_LAYERS[kind]])
    w = make_weights(cfg, 11, slow=6.0)
    toks = random_tokens(420, cfg["vocab"], 11)
    other = list(toks)
    other[far] = (toks[far] + 1) % cfg["vocab"]
    want, moved = O.forward(cfg, w, toks), O.forward(cfg, w, other)
    assert row_err(moved[-40:], want[-40:]) > 5e-5
    eng = _engine(cfg, w, page_size=16)
    eng.step([("a", toks[:301], [])])
    part = eng.step([("a", toks[301:400], list(range(99)))])
    tail = torch.cat([eng.step([("a", [t], [0])]) for t in toks[400:]])
    assert row_err(part[-20:], want[380:400]) < 0.1 * row_err(moved[380:400], want[380:400])
    assert row_err(tail, want[400:]) < 0.1 * row_err(moved[400:], want[400:])


@BOTH
@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 6, 7])
def test_first_tokens(dev, n, dtype):
    """Sequences shorter than the convolutions' memory and just past it, whole and one by one."""
    cfg = make_config(_stack(dtype), loop=LOOP)
    w = make_weights(cfg, 13)
    toks = random_tokens(n, cfg["vocab"], 13 + n)
    want = O.forward(cfg, w, toks)
    eng = _engine(cfg, w, dtype, page_size=16)
    assert _close(_whole(eng, "a", toks), want, dtype) and _close(_portions(eng, "b", toks, [1]), want, dtype)


@pytest.mark.parametrize("kind", ["state space", "gated unit"])
@pytest.mark.parametrize("cut", [1, 2, 3, 4, 15, 16, 63, 64, 65])
def test_convolution_reaches_back_over_a_cut(dev, kind, cut):
    """One token ahead of a portion's border is changed: the next tokens' convolutions read it from the slot."""
    cfg = make_config([side_layer(left_scale=0.0, conv=4, mlp=None) if kind == "state space" else unit_layer(conv=4, mlp=None)])
    w = make_weights(cfg, 19)
    toks = random_tokens(cut + 6, cfg["vocab"], 19)
    for back in range(1, min(cut, 3) + 1):
        seq = list(toks)
        seq[cut - back] = (seq[cut - back] + 1) % cfg["vocab"]
        want, eng = O.forward(cfg, w, seq), _engine(cfg, w)
        eng.step([("a", seq[:cut], [])])
        assert row_err(eng.step([("a", seq[cut:], list(range(6)))]), want[cut:]) < F32_TOL
        eng.release("a")
        eng.step([("a", seq[:cut], [])])
        assert row_err(torch.cat([eng.step([("a", [t], [0])]) for t in seq[cut:]]), want[cut:]) < F32_TOL


ATT_PATHS = [(torch.float32, None), (torch.bfloat16, None), (torch.bfloat16, "plain")]
ATT_IDS = ["f32", "bf16-tensor-core", "bf16-plain"]


def _run_rows(eng, rows, cuts, dtype, dev, slot_id="a"):
    """The first layer's left mixer on hand-made projection rows of one sequence, fed in portions that end at `cuts`; the head outputs."""
    from qserve_b200.hybrid import StepBatch, _stream

    mixer, cache = eng.model.layers[0].mixer.left, eng.cache
    st = cache.admit(slot_id)
    cache.reserve(slot_id, cuts[-1])
    table = cache.sync_block_table()
    scratch = torch.empty(max(1, eng.model.scratch_floats(cuts[-1])), dtype=torch.float32, device=dev)
    outs, lo = [], 0
    for hi in cuts:
        b = StepBatch.build([(st.slot, lo, -1, list(range(hi - lo)))], table, dev, cache.page_size)
        proj = rows[lo:hi].to(dev).to(dtype).contiguous()
        out = torch.zeros(hi - lo, mixer.out_features, dtype=dtype, device=dev)
        mixer.run(proj, out, b, cache.runs[0]["left"], cache.page_size, scratch, eng.model.dt, _stream(dev))
        outs.append(out.double().cpu())
        lo = hi
    cache.release(slot_id)
    return torch.cat(outs)


@pytest.mark.parametrize("dtype,impl", ATT_PATHS, ids=ATT_IDS)
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("scale,coef,every", [(0.05, 0.0, 1), (-2.0, 0.0, 1), (0.02, 3.0, 32), (-0.1, 0.6, 1), (0.3, 0.5, 50)])
def test_spare_term_and_temperature_by_hand(dev, dtype, impl, decoded, scale, coef, every):
    """Rows whose every query-key product is the same number s: a head's output at position i is the shared value times E / (1 + E),
    E = (i + 1) exp(s f(i)) with the temperature f, times the left factor.  Negative scores leave most of the softmax to the spare term."""
    H, G, D, Dv, n = 4, 2, 32, 64, 90
    cfg = make_config([side_layer(heads=H, kv_heads=G, dim=D, vdim=Dv, coef=coef, every=every, scale=scale, mlp=None)], width=16)
    eng = _engine(cfg, make_weights(cfg, 3), dtype, page_size=16)
    mixer = eng.model.layers[0].mixer.left
    mixer.bias.zero_()
    mixer.q_gain.fill_(1.0)
    mixer.k_gain.fill_(1.0)
    assert dtype == torch.float32 or _fast_ok(mixer)
    g = torch.Generator().manual_seed(7)
    rows = torch.ones(n, mixer.in_features)   # q and k rows of ones have unit RMS: every product is D
    v = _bf(torch.randn(G * Dv, generator=g))
    rows[:, (H + G) * D:(H + G) * D + G * Dv] = v
    with _impl(attention=impl):
        got = _run_rows(eng, rows, [n - 30] + list(range(n - 29, n + 1)) if decoded else [n - 30, n], dtype, dev)
    for h in range(H):
        value = v.double()[(h // 2) * Dv:(h // 2 + 1) * Dv]
        for i in (n - 1, n - 28, n - 17, n - 30, 63, 62):
            f = 1.0 + coef * math.log(math.floor((i + 1) / every) + 1)
            unit = 1.0 / (1.0 + cfg["norm"]["eps"])   # the product of the two unit rows
            if dtype == torch.bfloat16:   # the query and the key as they are stored
                f, unit = float(torch.tensor(f).to(torch.bfloat16).double()), 1.0
            e = (i + 1) * math.exp(D * scale * f * unit)
            want = 0.7 * value * e / (1.0 + e)
            err = float((got[i, h * Dv:(h + 1) * Dv] - want).norm() / want.norm())
            assert err < (2e-4 if dtype == torch.float32 else 8e-3), (h, i, err)


def _fast_ok(mixer) -> bool:
    from qserve_b200._lib import lib

    m = mixer.m
    return lib.qs_hyb_attention_fast_supported(0, m.heads, m.kv_heads, 1, m.dim, m.vdim, mixer.in_features) == 1


@pytest.mark.parametrize("dtype,impl", ATT_PATHS, ids=ATT_IDS)
@pytest.mark.parametrize("decoded", [False, True])
def test_attention_needles(dev, dtype, impl, decoded):
    """The probe token's query is ONE key's direction with a large scale, so that key owns the softmax and the head's output is its value.
    Needles at the first positions, at page and tile borders, far away, and the probe's own position; the probe as the last row of a prompt
    portion (tiles on the tensor cores in bfloat16) and as a token of its own (the head-group kernel)."""
    H, G, D, Dv, probe = 8, 2, 64, 96, 191
    cfg = make_config([side_layer(heads=H, kv_heads=G, dim=D, vdim=Dv, scale=1.0, coef=0.2, every=64, left_scale=1.0, mlp=None)], width=16)
    eng = _engine(cfg, make_weights(cfg, 21), dtype, page_size=16)
    mixer = eng.model.layers[0].mixer.left
    mixer.bias.zero_()
    mixer.q_gain.fill_(1.0)
    mixer.k_gain.fill_(1.0)
    assert dtype != torch.bfloat16 or _fast_ok(mixer)
    g = torch.Generator().manual_seed(5)
    rows = _bf(torch.randn(probe + 1, mixer.in_features, generator=g))
    k0, v0 = (H + G - 1) * D, (H + G) * D + (G - 1) * Dv   # the last key / value head, which the last query head reads
    with _impl(attention=impl):
        for j in (0, 1, 15, 16, 63, 64, 127, 128, probe - 16, probe - 1, probe):
            r = rows.clone()
            r[probe, (H - 1) * D:H * D] = _bf(2.0 * rows[j, k0:k0 + D])
            got = _run_rows(eng, r, [100, probe, probe + 1] if decoded else [100, probe + 1], dtype, dev)
            value = rows[j, v0:v0 + Dv].double()
            err = float((got[probe, (H - 1) * Dv:] - value).norm() / value.norm())
            assert err < (1e-4 if dtype == torch.float32 else 6e-3), (j, err)


# ------------------------------------------------------------------------------------------------------------------------
# sizes that take the tensor-core and vector paths
# ------------------------------------------------------------------------------------------------------------------------
TC_LAYERS = [side_layer(heads=8, kv_heads=2, dim=32, vdim=64, sheads=8, state=64, svdim=32, groups=2, norm_groups=2, mlp=moe(4, 4, 32, 0.4)),
             unit_layer(width=192, blocks=3, mlp=dense(128)),
             side_layer(heads=4, kv_heads=1, dim=64, vdim=96, sheads=4, state=128, svdim=64, groups=1, norm_groups=1, mlp=dense(96))]


def _engine_runs(cfg, w, a, b):
    """a whole, a in portions with b beside it, a's prefix then single tokens, b alone (bfloat16)."""
    eng = _engine(cfg, w, torch.bfloat16, page_size=16)
    whole = _whole(eng, "a", a)
    rows = {"a": [], "b": []}
    for lo, hi, bl, bh in ((0, 50, 0, 3), (50, 114, 3, 40), (114, 116, 40, 41), (116, len(a), 41, len(b))):
        out = eng.step([("a", a[lo:hi], list(range(hi - lo))), ("b", b[bl:bh], list(range(bh - bl)))])
        rows["a"].append(out[:hi - lo])
        rows["b"].append(out[hi - lo:])
    eng.release("a")
    eng.release("b")
    n = 150
    single = torch.cat([eng.step([("a", a[:n], list(range(n)))])] + [eng.step([("a", [t], [0])]) for t in a[n:190]])
    return whole, torch.cat(rows["a"]), single, torch.cat(rows["b"])


@pytest.mark.parametrize("layers", [[0], [1], [2], [0, 1, 2]], ids=str)
def test_tensor_core_paths(dev, layers):
    cfg = make_config([TC_LAYERS[i] for i in layers], width=128, vocab=160, loop=(0, len(layers), 2) if len(layers) == 1 else (1, 2, 2))
    w = make_weights(cfg, 14)
    a, b = random_tokens(200, cfg["vocab"], 14), random_tokens(90, cfg["vocab"], 15)
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    for got, want in zip(_engine_runs(cfg, w, a, b), (wa, wa, wa[:190], wb)):
        assert bf16_close(got, want)


def test_long_prompt(dev):
    """A prompt of many tiles and blocks of several tokens per convolution block, in two portions, then single tokens: 32-bit engine."""
    cfg = make_config([side_layer(mlp=None), unit_layer(mlp=None)])
    w = make_weights(cfg, 22, slow=5.0)
    toks = random_tokens(2300, cfg["vocab"], 22)
    want = O.forward(cfg, w, toks)
    eng = _engine(cfg, w, max_tokens=4096)
    first = eng.step([("a", toks[:2201], list(range(2201)))])
    rest = torch.cat([eng.step([("a", toks[2201:2290], list(range(89)))])] + [eng.step([("a", [t], [0])]) for t in toks[2290:]])
    assert row_err(first, want[:2201]) < F32_TOL and row_err(rest, want[2201:]) < F32_TOL


# ------------------------------------------------------------------------------------------------------------------------
# the framework's own entry points
# ------------------------------------------------------------------------------------------------------------------------
def test_generate_through_scheduler(dev):
    """Greedy generation through Engine.generate: admission, prompt chunks, decoding, retirement; against the oracle's argmax."""
    from qserve_b200.engine import SamplingParams

    cfg = make_config(STACK, loop=LOOP)
    w = make_weights(cfg, 16)
    prompts = [random_tokens(n, cfg["vocab"], 40 + n) for n in (5, 37, 1, 70, 12, 20)]
    eng = _engine(cfg, w, max_tokens=4 * 96, page_size=16, chunk=24, max_batch_tokens=48)
    outs = eng.generate(prompts, [SamplingParams(max_new_tokens=6)] * len(prompts))
    for p, o in zip(prompts, outs):
        assert o == O.greedy(cfg, w, p, 6)
    assert eng.cache.free_pages() == eng.cache.num_pages


def _write_model(path, cfg, w):
    import struct

    path.mkdir()
    (path / "config.json").write_text(json.dumps(cfg))
    header, blobs, at = {}, [], 0
    for k, v in w.items():
        raw = v.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        header[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))


def test_model_folder_trace_replay_and_command_line(dev, tmp_path, capsys):
    """config.json + model.safetensors on disk -> Engine.from_dir -> a replayed trace with portions, a request that sits out, and reuse; then
    greedy generation from the same folder through the command line."""
    import io

    import numpy as np

    from qserve_b200.cli import main
    from qserve_b200.engine import Engine, replay_trace

    cfg = make_config(STACK[:3], loop=(0, 2, 2))
    w = make_weights(cfg, 17)
    _write_model(tmp_path / "m", cfg, w)
    (tmp_path / "out").mkdir()
    a, b = random_tokens(50, cfg["vocab"], 17), random_tokens(9, cfg["vocab"], 18)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[30:], "want": [0, 19]}, {"id": "b", "tokens": b[2:], "want": [6]}], "end": ["a", "b"]}]
    eng = Engine.from_dir(str(tmp_path / "m"), torch.float32, max_tokens=128, max_seqs=2, page_size=64)
    log = io.StringIO()
    assert replay_trace(eng, [json.dumps(s) for s in steps], str(tmp_path / "out"), log) == 3
    assert log.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    got0 = torch.from_numpy(np.fromfile(tmp_path / "out" / "0.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
    got2 = torch.from_numpy(np.fromfile(tmp_path / "out" / "2.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
    assert not (tmp_path / "out" / "1.f32").exists()
    assert row_err(got0, wa[29:30]) < F32_TOL and row_err(got2, torch.stack([wa[30], wa[49], wb[8]])) < F32_TOL
    assert eng.cache.free_pages() == eng.cache.num_pages
    capsys.readouterr()
    assert main(["generate", "--model", str(tmp_path / "m"), "--dtype", "float32", "--prompt", ",".join(map(str, b)), "--max-new-tokens", "4"]) == 0
    assert [int(t) for t in capsys.readouterr().out.strip().splitlines()[-1].split(",")] == O.greedy(cfg, w, b, 4)
