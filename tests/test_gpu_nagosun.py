"""GPU tests of the Nagosun family: the engine (model, page pool, slots, scheduler, kernels) against the plain float64 restatement in
tests/nagosun_oracle.py, on small random models of several shapes."""
import json
import math

import pytest
import torch

from tests import nagosun_oracle as O
from tests.hybrid_util import bf16_close, random_tokens, row_err
from tests.nagosun_util import attention_layer, dense, latent_layer, make_config, make_weights

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4   # float32 engine vs float64 oracle


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


class _impl:
    """Keep the attention kernels on one implementation for a while (None: the engine's own choice)."""

    def __init__(self, latent=None, attention=None):
        self.want = (latent, attention)

    def __enter__(self):
        import qserve_b200.hybrid as hyb

        hyb.LATENT_IMPL, hyb.ATTENTION_IMPL = self.want

    def __exit__(self, *exc):
        import qserve_b200.hybrid as hyb

        hyb.LATENT_IMPL = hyb.ATTENTION_IMPL = None


STACK = [latent_layer(), attention_layer(), attention_layer(heads=6, kv_heads=3, dim=8, vdim=20, size=17, softcap=2.0, mlp=None),
         latent_layer(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=16, size=40, mlp=None), attention_layer(heads=2, kv_heads=1, size=0, softcap=0, mlp=dense(24))]


# ------------------------------------------------------------------------------------------------------------------------
# kernels alone
# ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,groups,add_f32,bias,gate,fresh", [
    (40, 1, True, True, True, False), (48, 4, False, True, True, False), (33, 3, True, False, True, True), (2048, 4, True, True, True, False),
    (2048, 1, True, False, False, True), (1030, 2, False, False, True, False), (44, 44, True, True, True, False), (64, 32, True, False, True, False),
    (1536, 3, True, True, True, False), (8192, 16, True, True, True, False), (16384, 2, True, False, True, False), (20000, 5, False, True, True, False),
    (16384, 16, True, True, False, True), (640, 8, True, True, True, False)])
def test_gated_norm_update_kernel(dev, dtype, width, groups, add_f32, bias, gate, fresh):
    from qserve_b200._lib import check, lib

    g = torch.Generator().manual_seed(width + groups)
    T, dt, mult, eps, off = 7, 0 if dtype == torch.bfloat16 else 1, 0.6, 1e-3, 0.25
    x, y, z = torch.randn(T, width, generator=g), _bf(torch.randn(T, width, generator=g) * 3.0), _bf(torch.randn(T, width + 8, generator=g) * 2.0)
    z[0, 8], z[0, 9] = -200.0, 200.0   # gates shut and wide open
    w, wn, b, gb = (torch.randn(width, generator=g) for _ in range(4))
    want = y.double() + (b.double() if bias else 0.0)
    if gate:
        want = want * torch.sigmoid(z[:, 8:].double() + gb.double())
    want = O.grouped_norm(want, off + w.double(), groups, eps) * mult + (0.0 if fresh else x.double())
    want_h = O.grouped_norm(want, off + wn.double(), groups, eps)
    xd, wd, wnd, bd, gbd = x.to(dev), w.to(dev), wn.to(dev), b.to(dev), gb.to(dev)
    yd = y.to(dev) if add_f32 else y.to(dev).to(dtype)
    zd = z.to(dev).to(dtype)
    h = torch.zeros(T, width, dtype=dtype, device=dev)

    def run(out, xx):
        check(lib.qs_hyb_gated_norm_update(out.data_ptr() if out is not None else None, xx.data_ptr(), 1 if fresh else 0, yd.data_ptr(), 1 if add_f32 else 0,
                                           bd.data_ptr() if bias else None, zd[:, 8:].data_ptr() if gate else None, width + 8, gbd.data_ptr(), wd.data_ptr(),
                                           mult, wnd.data_ptr(), groups, off, eps, T, width, dt, _raw()))

    run(h, xd)
    assert float((xd.double().cpu() - want).abs().max()) < 5e-5
    tol = 1e-4 if dtype == torch.float32 else 2.0 ** -8
    assert float(((h.double().cpu() - want_h).abs() / (want_h.abs() + 0.05)).max()) < tol
    x2 = x.to(dev)
    run(None, x2)   # without the next norm the stream is the same, bit for bit
    assert torch.equal(x2, xd)


def test_gated_norm_update_refuses_uneven_groups(dev):
    from qserve_b200._lib import lib

    t = torch.zeros(2, 10, device=dev)
    assert lib.qs_hyb_gated_norm_update(None, t.data_ptr(), 0, t.data_ptr(), 1, None, None, 0, None, t.data_ptr(), 1.0, None, 3, 0.0, 1e-5, 2, 10, 1, _raw()) != 0


def _run_rows(eng, rows, cuts, dtype, dev, slot_id="a"):
    """The first layer's mixer on hand-made projection rows of one sequence, fed in portions that end at `cuts`; the head outputs."""
    from qserve_b200.hybrid import StepBatch, _stream

    mixer, cache = eng.model.layers[0].mixer, eng.cache
    st = cache.admit(slot_id)
    cache.reserve(slot_id, cuts[-1])
    table = cache.sync_block_table()
    scratch = torch.empty(max(1, eng.model.scratch_floats(cuts[-1])), dtype=torch.float32, device=dev)
    outs, lo = [], 0
    for hi in cuts:
        b = StepBatch.build([(st.slot, lo, -1, list(range(hi - lo)))], table, dev, cache.page_size)
        proj = rows[lo:hi].to(dev).to(dtype).contiguous()
        out = torch.zeros(hi - lo, mixer.out_features, dtype=dtype, device=dev)
        mixer.run(proj, out, b, cache.runs[0], cache.page_size, scratch, eng.model.dt, _stream(dev))
        outs.append(out.double().cpu())
        lo = hi
    cache.release(slot_id)
    return torch.cat(outs)


ATT_PATHS = [(torch.float32, None), (torch.bfloat16, None), (torch.bfloat16, "plain")]
ATT_IDS = ["f32", "bf16-tensor-core", "bf16-plain"]


@pytest.mark.parametrize("dtype,impl", ATT_PATHS, ids=ATT_IDS)
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("cap,raw,window", [(3.0, 0.4, 1), (3.0, 90.0, 1), (1.5, -40.0, 1), (50.0, 5.0, 2), (0.0, 2.0, 1), (2.0, 1.0, 30)])
def test_cap_and_spare_term_by_hand(dev, dtype, impl, decoded, cap, raw, window):
    """Rows whose every query-key product is the same number: a head's output is known in closed form -- the shared value at unit RMS, times
    the gate, times the keys' share E / (1 + E), E = sum over the window of exp(cap tanh(raw / cap) - slope distance).  A sink left out, a cap
    missed, applied behind the distance penalty, or a window one position off each show in that share."""
    H, G, D, Dv, n = 4, 2, 32, 64, 90
    cfg = make_config([attention_layer(heads=H, kv_heads=G, dim=D, vdim=Dv, size=window, softcap=cap, scale=0.25, mlp=None)], width=16)
    eng = _engine(cfg, make_weights(cfg, 3), dtype, page_size=16)
    mixer = eng.model.layers[0].mixer
    mixer.bias.zero_()
    assert impl == "plain" or dtype == torch.float32 or _fast_ok(mixer)
    g = torch.Generator().manual_seed(7)
    rows = torch.zeros(n, mixer.in_features)
    rows[:, :H * D:D] = raw          # first entry of every query head; scale 0.25 x key entry 4
    rows[:, H * D:(H + G) * D:D] = 4.0
    v, z = _bf(torch.randn(G * Dv, generator=g) * 0.01), _bf(torch.randn(n, H * Dv, generator=g))   # small values: eps counts in their norm
    rows[:, (H + G) * D:mixer.col_g] = v
    rows[:, mixer.col_g:mixer.col_g + H * Dv] = z
    with _impl(attention=impl):
        got = _run_rows(eng, rows, [n - 30] + list(range(n - 29, n + 1)) if decoded else [n - 30, n], dtype, dev)
    raw_b = float(torch.tensor(raw).to(dtype).double()) if dtype == torch.bfloat16 else raw
    for h in range(H):
        value = O.unit_rms(v.double()[(h // 2) * Dv:(h // 2 + 1) * Dv], 1e-5)
        for i in (n - 1, n - 30, n - 17):
            d = torch.arange(min(window, i + 1), dtype=torch.float64)
            s = (cap * math.tanh(raw_b / cap) if cap else raw_b) - O.slope(h, H) * d
            e = float(torch.exp(s).sum())
            want = value * e / (1.0 + e) * torch.sigmoid(z[i, h * Dv:(h + 1) * Dv].double())
            err = float((got[i, h * Dv:(h + 1) * Dv] - want).norm() / want.norm())
            assert err < (1e-4 if dtype == torch.float32 else 6e-3), (h, i, err)


def _fast_ok(mixer) -> bool:
    from qserve_b200._lib import lib

    m = mixer.m
    return lib.qs_hyb_attention_fast_supported(0, m.heads, m.kv_heads, 1, m.dim, m.vdim, mixer.in_features) == 1


# ------------------------------------------------------------------------------------------------------------------------
# every mechanism alone, through the engine
# ------------------------------------------------------------------------------------------------------------------------
LAYERS = [
    latent_layer(mlp=None), latent_layer(heads=1, dim=4, rot_dim=2, vdim=6, kv_rank=5, size=1, mlp=None), latent_layer(heads=8, dim=16, rot_dim=8, vdim=16, kv_rank=32, size=64, mlp=None),
    latent_layer(heads=5, dim=20, rot_dim=12, vdim=4, kv_rank=9, base=1e6, size=33, mlp=None), latent_layer(heads=2, dim=2, rot_dim=30, vdim=40, kv_rank=64, size=100, mlp=None),
    latent_layer(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=16, scale=0.5, size=16, mlp=None),   # equal sizes everywhere
    latent_layer(heads=7, dim=3, rot_dim=2, vdim=1, kv_rank=48, size=0, mlp=None),                  # no window at all
    attention_layer(mlp=None), attention_layer(heads=1, kv_heads=1, dim=4, vdim=1, size=1, mlp=None), attention_layer(heads=6, kv_heads=2, dim=10, vdim=33, size=40, softcap=1.0, mlp=None),
    attention_layer(heads=3, kv_heads=3, dim=32, vdim=32, size=7, softcap=80.0, mlp=None), attention_layer(heads=8, kv_heads=1, dim=16, vdim=16, size=0, mlp=None),
    attention_layer(heads=2, kv_heads=2, dim=64, vdim=64, size=64, softcap=0, scale=0.2, mlp=None), attention_layer(heads=5, kv_heads=5, dim=1, vdim=130, size=100, softcap=4.0, mlp=None),
]


def _layer_id(l):
    m = l["mixer"]
    return l["type"][:3] + "-" + "x".join(str(v) for v in m.values() if isinstance(v, int)) + "-w" + str((m.get("mask") or {}).get("size", 0))


@pytest.mark.parametrize("layer", LAYERS, ids=_layer_id)
def test_single_layer(dev, layer):
    cfg = make_config([layer])
    w = make_weights(cfg, 2, sharp=3.0)
    toks = random_tokens(150, cfg["vocab"], 2)
    taps, layers = [], []
    eng = _engine(cfg, w)
    got = eng.step([("a", toks, list(range(len(toks))))], tap=lambda r, x: taps.append(x.clone()))
    want = O.forward(cfg, w, toks, layers)
    assert row_err(taps[0], layers[0]) < F32_TOL
    assert row_err(got, want) < F32_TOL
    eng.release("a")
    assert row_err(_portions(eng, "b", toks, [40, 1, 1, 2, 19]), want) < F32_TOL


# (in bfloat16 without sizes whose norms see one number only, a feed-forward of one column or groups of one channel: they keep a sign, which
# rounding may flip)
@pytest.mark.parametrize("ff,dtype", [(56, torch.float32), (1, torch.float32), (300, torch.float32), (56, torch.bfloat16), (300, torch.bfloat16)])
def test_feed_forward_after_mixer(dev, ff, dtype):
    cfg = make_config([latent_layer(mlp=dense(ff)), attention_layer(mlp=dense(ff))])
    w = make_weights(cfg, 3)
    toks = random_tokens(70, cfg["vocab"], 3)
    got = _whole(_engine(cfg, w, dtype), "a", toks)
    want = O.forward(cfg, w, toks)
    assert row_err(got, want) < F32_TOL if dtype == torch.float32 else bf16_close(got, want)


@pytest.mark.parametrize("kw", [dict(groups=1), dict(groups=4), dict(groups=44), dict(groups=11, width=33), dict(mult=1.0), dict(mult=0.05), dict(logit_scale=1.0),
                                dict(logit_scale=0.03), dict(eps=0.5), dict(width=7, groups=7, vocab=5), dict(width=128, groups=8, vocab=131)], ids=str)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_constants_of_the_stack(dev, kw, dtype):
    cfg = make_config(STACK[:3], **kw)
    if dtype == torch.bfloat16 and cfg["width"] == cfg["norm"]["groups"]:
        pytest.skip("groups of one channel keep only the sign, which rounding may flip")
    w = make_weights(cfg, 5)
    toks = random_tokens(50, cfg["vocab"], 5)
    eng = _engine(cfg, w, dtype)
    want = O.forward(cfg, w, toks)
    got = _portions(eng, "a", toks, [30, 1])
    assert row_err(got, want) < F32_TOL if dtype == torch.float32 else bf16_close(got, want)


def test_stack_and_taps(dev):
    cfg = make_config(STACK, width=52, vocab=131, groups=4)
    w = make_weights(cfg, 4, sharp=2.0)
    toks = random_tokens(120, cfg["vocab"], 4)
    taps, layers = [], []
    got = _engine(cfg, w).step([("a", toks, list(range(len(toks))))], tap=lambda r, x: taps.append(x.clone()))
    want = O.forward(cfg, w, toks, layers)
    assert len(taps) == len(layers) == len(STACK)
    for t, l in zip(taps, layers):
        assert row_err(t, l) < F32_TOL
    assert row_err(got, want) < F32_TOL


# ------------------------------------------------------------------------------------------------------------------------
# cuts, batches, reuse
# ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_prefill_against_token_by_token(dev, dtype):
    cfg = make_config(STACK)
    w = make_weights(cfg, 6, sharp=2.0 if dtype == torch.float32 else 1.0)   # peaked maps multiply bfloat16's rounding noise layer by layer
    toks = random_tokens(140, cfg["vocab"], 6)
    want = O.forward(cfg, w, toks)
    eng = _engine(cfg, w, dtype)
    whole = _whole(eng, "a", toks)
    single = _portions(eng, "b", toks, [1])   # from the first token on: graph replay from the second
    eng.release("b")
    if dtype == torch.float32:
        assert row_err(whole, want) < F32_TOL and row_err(single, want) < F32_TOL
    else:
        assert bf16_close(whole, want) and bf16_close(single, want) and bf16_close(single, whole)


@pytest.mark.parametrize("sizes", [[2], [3, 2, 7], [64], [63, 1, 65], [17, 100, 5, 2], [130, 2], [23, 24, 25]])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_portions(dev, sizes, dtype):
    """Portions cut in the middle of pages (16) and of the windows (17, 24, 40)."""
    cfg = make_config(STACK)
    w = make_weights(cfg, 7, sharp=2.0 if dtype == torch.float32 else 1.0)
    toks = random_tokens(210, cfg["vocab"], 7)
    got, want = _portions(_engine(cfg, w, dtype, page_size=16), "a", toks, sizes), O.forward(cfg, w, toks)
    assert row_err(got, want) < F32_TOL if dtype == torch.float32 else bf16_close(got, want)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mixed_batches_with_reuse(dev, dtype):
    """Unequal requests in one batch (portions beside single tokens) against each alone; four slots and a page pool that is far smaller than
    the sum of all requests, so that pages and slots are handed out again."""
    cfg = make_config(STACK)
    w = make_weights(cfg, 8, sharp=2.0 if dtype == torch.float32 else 1.0)
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
        g = torch.cat(got[k])
        assert row_err(g, alone[k]) < F32_TOL if dtype == torch.float32 else bf16_close(g, alone[k]), k


def test_long_decoding_and_graph_replay(dev):
    """Hundreds of single tokens through captured graphs against eager launches and the oracle; two sequences side by side.  The windows pass
    over decoded tokens many times."""
    cfg = make_config(STACK[:4])
    w = make_weights(cfg, 9, sharp=2.0)
    a, b = random_tokens(330, cfg["vocab"], 9), random_tokens(300, cfg["vocab"], 10)
    outs = {}
    for graphs in (True, False):
        eng = _engine(cfg, w, use_graphs=graphs, page_size=16)
        eng.step([("a", a[:30], []), ("b", b[:1], [])])
        rows = []
        for i in range(299):
            rows.append(eng.step([("a", a[30 + i:31 + i], [0]), ("b", b[1 + i:2 + i], [0])]))
        outs[graphs] = torch.stack(rows)
    assert torch.equal(outs[True], outs[False])
    wa, wb = O.forward(cfg, w, a[:329]), O.forward(cfg, w, b)
    assert row_err(outs[True][:, 0], wa[30:]) < F32_TOL and row_err(outs[True][:, 1], wb[1:]) < F32_TOL


# ------------------------------------------------------------------------------------------------------------------------
# keys far away, at page borders, at the window's edges
# ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("far", [0, 1, 15, 16, 17, 63, 64, 300])
@pytest.mark.parametrize("kind", ["latent", "attention"])
def test_far_token_is_seen(dev, far, kind):
    """A long prompt under a window wider than it, whose token at `far` (first positions, page borders, an earlier portion) is changed: the
    oracle's answer at the last positions moves by a small but definite amount, and the engine's distance to the right answer is a small
    fraction of that move -- in a prompt portion and for decoded tokens."""
    layer = latent_layer(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=24, size=4000, mlp=None) if kind == "latent" else \
        attention_layer(heads=16, kv_heads=2, dim=16, vdim=16, size=4000, softcap=30.0, mlp=None)
    cfg = make_config([layer])
    w = make_weights(cfg, 11)
    toks = random_tokens(420, cfg["vocab"], 11)
    other = list(toks)
    other[far] = (toks[far] + 1) % cfg["vocab"]
    want, moved = O.forward(cfg, w, toks), O.forward(cfg, w, other)
    assert row_err(moved[-40:], want[-40:]) > 2e-5
    eng = _engine(cfg, w, page_size=16)
    eng.step([("a", toks[:301], [])])
    part = eng.step([("a", toks[301:400], list(range(99)))])
    tail = torch.cat([eng.step([("a", [t], [0])]) for t in toks[400:]])
    assert row_err(part[-20:], want[380:400]) < 0.05 * row_err(moved[380:400], want[380:400])
    assert row_err(tail, want[400:]) < 0.05 * row_err(moved[400:], want[400:])


WINDOW = 40
EDGE_LAYERS = {"attention": attention_layer(heads=4, kv_heads=2, dim=16, vdim=32, size=WINDOW, mlp=None),
               "latent": latent_layer(heads=4, dim=16, rot_dim=16, vdim=32, kv_rank=32, size=WINDOW, mlp=None)}


@pytest.mark.parametrize("kind,dtype,impl", [("attention", torch.float32, None), ("attention", torch.bfloat16, None), ("attention", torch.bfloat16, "plain"),
                                             ("latent", torch.float32, None), ("latent", torch.bfloat16, None), ("latent", torch.bfloat16, "latent"),
                                             ("latent", torch.bfloat16, "plain")])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("query", [130, 144, 191])   # in the middle of a page, at a page's first cell, at the last cell of a 64-key tile
def test_window_edges(dev, kind, dtype, impl, decoded, query):
    """One layer: the logits at `query` depend on the token at position j exactly when j is inside the window.  Changing a visible token moves
    the oracle's answer and the float32 engine follows it; changing a hidden one (just outside, or farther back) leaves the engine's answer bit
    for bit as it was, in either storage type.  In a prompt portion that starts inside an earlier window and for a token decoded alone."""
    cfg = make_config([EDGE_LAYERS[kind]], width=48)
    w = make_weights(cfg, 12, sharp=2.0)
    toks = random_tokens(query + 1, cfg["vocab"], 12)

    def at_query(seq):
        with _impl(impl, impl if impl == "plain" else None):
            eng = _engine(cfg, w, dtype, page_size=16)
            if decoded:
                eng.step([("a", seq[:query], [])])
                return eng.step([("a", seq[query:], [0])])[0]
            eng.step([("a", seq[:100], [])])
            return eng.step([("a", seq[100:], [query - 100])])[0]

    base, want = at_query(toks), O.forward(cfg, w, toks)[query]
    assert float((base.double().cpu() - want).norm()) < (1e-4 if dtype == torch.float32 else 0.05) * float(want.norm())
    for j, seen in ((query - WINDOW + 1, True), (query - WINDOW, False), (query - 1, True), (query - WINDOW - 1, False), (0, False), (query - WINDOW - 17, False)):
        other = list(toks)
        other[j] = (toks[j] + 7) % cfg["vocab"]
        moved, got = O.forward(cfg, w, other)[query], at_query(other)
        effect = float((moved - want).norm())
        if seen:
            assert effect > 1e-5 * float(want.norm()), j
            if dtype == torch.float32 or effect > 1e-2 * float(want.norm()):   # bfloat16 rounds smaller moves away
                assert not torch.equal(got, base), j
            if dtype == torch.float32:
                assert float((got.double().cpu() - moved).norm()) < 0.2 * effect, j   # a missed key would leave the whole effect
        else:
            assert effect < 1e-12 and torch.equal(got, base), j


@pytest.mark.parametrize("dtype,impl", ATT_PATHS, ids=ATT_IDS)
@pytest.mark.parametrize("decoded", [False, True])
def test_attention_needles(dev, dtype, impl, decoded):
    """The attention mixer on hand-made projection rows: the probe token's query in the flattest head is a large multiple of ONE key's
    direction, so that key owns the softmax whenever it is visible and the head's output is that key's unit-RMS value.  Needles at the window's
    edges, at page and tile borders, far away, and the probe's own position; the probe as the last row of a prompt portion (tiles on the
    tensor cores in bfloat16) and as a token of its own (the head-group kernel)."""
    H, G, D, Dv, probe = 8, 2, 64, 96, 191
    cfg = make_config([attention_layer(heads=H, kv_heads=G, dim=D, vdim=Dv, size=WINDOW, softcap=40.0, scale=0.2, mlp=None)], width=16)
    eng = _engine(cfg, make_weights(cfg, 21), dtype, page_size=16)
    mixer = eng.model.layers[0].mixer
    mixer.bias.zero_()
    assert dtype != torch.bfloat16 or _fast_ok(mixer)
    g = torch.Generator().manual_seed(5)
    rows = _bf(torch.randn(probe + 1, mixer.in_features, generator=g))
    rows[:, mixer.col_g:] = 20.0   # gates wide open
    keys = rows[:, H * D + (G - 1) * D: H * D + G * D]   # the last key / value head, which the last (flattest) query head reads
    values = O.unit_rms(rows[:, mixer.col_g - Dv:mixer.col_g].double(), 1e-5)
    with _impl(attention=impl):
        for j, seen in ((probe - WINDOW + 1, True), (probe - WINDOW, False), (0, False), (15, False), (64, False), (127, False), (128, False),
                        (probe - WINDOW + 9, True), (160, True), (176, True), (probe - 1, True), (probe, True)):
            r = rows.clone()
            r[probe, (H - 1) * D: H * D] = _bf(3.0 * keys[j])
            out = _run_rows(eng, r, [probe, probe + 1] if decoded else [probe - 29, probe + 1], dtype, dev)
            hit = float((out[-1, (H - 1) * Dv:] - values[j]).abs().max()) < 0.05 * float(values[j].abs().max())
            assert hit == seen, (j, seen)


@pytest.mark.parametrize("dtype,impl", [(torch.float32, None), (torch.bfloat16, None), (torch.bfloat16, "latent"), (torch.bfloat16, "plain")],
                         ids=["f32", "bf16", "bf16-latent-tiles", "bf16-plain"])
@pytest.mark.parametrize("decoded", [False, True])
def test_latent_needles(dev, dtype, impl, decoded):
    """Latent attention whose up-projections are the identity: a key is the normed latent itself and so is the value.  The probe's query is a
    large multiple of one position's latent (no rotated part), which then owns the softmax whenever it is visible."""
    H, K, R, probe = 4, 32, 16, 150
    cfg = make_config([latent_layer(heads=H, dim=K, rot_dim=R, vdim=K, kv_rank=K, size=WINDOW, scale=1.0, mlp=None)], width=16)
    w = make_weights(cfg, 22)
    w["l0.mix.uk"] = w["l0.mix.uv"] = torch.eye(K).repeat(H, 1)
    w["l0.mix.dkv.norm"] = torch.ones(K)
    eng = _engine(cfg, w, dtype, page_size=16)
    mixer = eng.model.layers[0].mixer
    rows = torch.zeros(probe + 1, mixer.in_features)
    latents = torch.randn(probe + 1, K, generator=torch.Generator().manual_seed(6))
    rows[:, mixer.col_kv:mixer.col_kv + K] = _bf(latents)
    normed = O.unit_rms(_bf(latents).double(), 1e-5)
    with _impl(latent=impl):
        for j, seen in ((probe - WINDOW + 1, True), (probe - WINDOW, False), (0, False), (63, False), (64, False), (probe - WINDOW + 2, True), (127, True),
                        (128, True), (probe - 1, True), (probe, True)):
            r = rows.clone()
            for h in range(H):
                r[probe, h * (K + R):h * (K + R) + K] = _bf(2.0 * normed[j].float())
            out = _run_rows(eng, r, [probe, probe + 1] if decoded else [probe - 29, probe + 1], dtype, dev)
            for h in (0, H - 1):
                hit = float((out[-1, h * K:(h + 1) * K] - normed[j]).abs().max()) < 0.05 * float(normed[j].abs().max())
                assert hit == seen, (j, seen)


@pytest.mark.parametrize("n", [1, 2, 3, 6, 7])
def test_first_tokens(dev, n):
    """Sequences around the length of their windows, whole and token by token."""
    cfg = make_config([attention_layer(size=3), latent_layer(size=6), attention_layer(size=2, mlp=None)])
    w = make_weights(cfg, 13, sharp=2.0)
    toks = random_tokens(n, cfg["vocab"], 13)
    eng = _engine(cfg, w)
    want = O.forward(cfg, w, toks)
    assert row_err(_whole(eng, "a", toks), want) < F32_TOL
    assert row_err(_portions(eng, "b", toks, [1]), want) < F32_TOL


# ------------------------------------------------------------------------------------------------------------------------
# bfloat16 on the tensor-core kernels
# ------------------------------------------------------------------------------------------------------------------------
TC_LAYERS = [latent_layer(heads=4, dim=16, rot_dim=16, vdim=32, kv_rank=32, size=50),                # prompt portions on per-head keys and values
             attention_layer(heads=8, kv_heads=2, dim=32, vdim=64, size=70, softcap=3.0),
             latent_layer(heads=20, dim=8, rot_dim=16, vdim=8, kv_rank=64, size=90, mlp=None),       # sizes only the latent-space tiles take
             latent_layer(heads=3, dim=40, rot_dim=8, vdim=64, kv_rank=40, size=33, mlp=None),       # per-head portions, single tokens on the plain kernel
             attention_layer(heads=8, kv_heads=8, dim=64, vdim=32, size=33, softcap=30.0, mlp=None),
             attention_layer(heads=6, kv_heads=1, dim=16, vdim=128, size=0, softcap=1.0, mlp=None)]


def _engine_runs(cfg, w, a, b):
    """Whole prompt, portions, and a mixed schedule (a portion of b beside single tokens of a, then both decode) in bfloat16."""
    eng = _engine(cfg, w, torch.bfloat16, page_size=16)
    whole = _whole(eng, "w", a)
    parts = _portions(eng, "p", a, [70, 2, 33, 1, 1, 64])
    eng.release("p")
    ga, gb = [eng.step([("a", a[:100], list(range(100)))])], []
    for i in range(90):
        e = [("a", a[100 + i:101 + i], [0])] + ([("b", b[:40], list(range(40)))] if i == 0 else [("b", b[39 + i:40 + i], [0])] if i <= 50 else [])
        out = eng.step(e)
        ga.append(out[:1])
        if i <= 50:
            gb.append(out[1:])
    return whole, parts, torch.cat(ga), torch.cat(gb)


@pytest.mark.parametrize("layer", range(len(TC_LAYERS)))
def test_tensor_core_paths_layer_by_layer(dev, layer):
    """bfloat16 layers whose sizes the tensor-core kernels take, one at a time (so that rounding noise is not multiplied by later layers):
    whole prompts, portions, single tokens (graph replay) and a mixed batch through the engine, against the oracle and against the same engine
    kept on the plain kernels.  Latent attention: prompt portions on the per-head keys and values of the window's pages where the head sizes
    allow, else (and when told so) on tiles in the latent space, single tokens always there; attention: tiles for portions, head groups for
    single tokens, with the score cap, the distance bias, the spare term of the softmax and the gate per output number."""
    cfg = make_config([TC_LAYERS[layer]], width=64)
    w = make_weights(cfg, 14 + layer, sharp=2.0)
    a, b = random_tokens(200, cfg["vocab"], 14), random_tokens(90, cfg["vocab"], 15)
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    runs = {}
    for impl in (None, "latent", "plain"):
        with _impl(impl, "plain" if impl == "plain" else None):
            runs[impl] = _engine_runs(cfg, w, a, b)
    for impl in (None, "latent", "plain"):
        for got, want in zip(runs[impl], (wa, wa, wa[:190], wb)):
            assert row_err(got, want) < 0.06, impl
    for impl in (None, "latent"):
        for f, p in zip(runs[impl], runs["plain"]):
            assert row_err(f, p) < 0.03, impl


def test_tensor_core_paths_stack(dev):
    cfg = make_config(TC_LAYERS, width=64, groups=4)
    w = make_weights(cfg, 14)
    a, b = random_tokens(200, cfg["vocab"], 14), random_tokens(90, cfg["vocab"], 15)
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    for got, want in zip(_engine_runs(cfg, w, a, b), (wa, wa, wa[:190], wb)):
        assert bf16_close(got, want)


@pytest.mark.parametrize("sharp", [0.3, 3.0, 30.0])
def test_capped_scores_small_and_large(dev, sharp):
    """Scores far below, around and far above the cap on every attention path: the series branch, the exponential branch and saturation."""
    cfg = make_config([attention_layer(heads=8, kv_heads=2, dim=32, vdim=64, size=70, softcap=4.0, mlp=None)], width=64)
    w = make_weights(cfg, 15, sharp=sharp)
    toks = random_tokens(150, cfg["vocab"], 15)
    want = O.forward(cfg, w, toks)
    assert row_err(_portions(_engine(cfg, w, page_size=16), "a", toks, [100, 1]), want) < F32_TOL
    for impl in (None, "plain"):
        with _impl(attention=impl):
            got = _portions(_engine(cfg, w, torch.bfloat16, page_size=16), "a", toks, [100, 1])
        assert row_err(got, want) < 0.06, impl


# ------------------------------------------------------------------------------------------------------------------------
# the framework's own entry points
# ------------------------------------------------------------------------------------------------------------------------
def test_generate_through_scheduler(dev):
    """Greedy generation through Engine.generate: admission, prompt chunks, decoding, retirement; against the oracle's argmax."""
    from qserve_b200.engine import SamplingParams

    cfg = make_config(STACK)
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

    cfg = make_config(STACK[:3])
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
