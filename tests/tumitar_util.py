"""Helpers of the Tumitar tests: small random models (config dict + weights under the design's tensor names)."""
import math

import torch


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, scale=1.5):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def side_layer(heads=4, kv_heads=2, dim=16, vdim=12, coef=0.4, every=24, scale=None, left_scale=0.7, right_scale=0.8, sheads=4, state=20, svdim=12, groups=2,
               conv=4, norm_groups=3, mlp="default"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.3 / math.sqrt(dim),
            "q_temp": {"coef": coef, "every": every}}
    right = {"heads": sheads, "state": state, "vdim": svdim, "groups": groups, "conv": conv, "norm_groups": norm_groups}
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": dense() if mlp == "default" else mlp}


def unit_layer(width=36, blocks=3, conv=4, mlp="default"):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": dense() if mlp == "default" else mlp}


def make_config(layers, vocab=83, width=44, eps=1e-5, loop=None, scale=3.0):
    cfg = {"architecture": "Tumitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def make_weights(cfg, seed=0, sharp=1.0, slow=0.0):
    """Random weights, rounded to bfloat16 values (held as float32) so that every dtype sees the same numbers.  `sharp` scales the query gains:
    large values make the softmax peaked.  `slow` makes the recurrent states forget slower (0: within some tens of tokens)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    bf = lambda t: t.to(torch.bfloat16).to(torch.float32)
    r = lambda *shape, s=1.0: bf(torch.randn(*shape, generator=g) * s)
    gain = lambda n, s=1.0: bf(s * (1.0 + 0.3 * torch.randn(n, generator=g)))
    w = {"embed": r(cfg["vocab"], W, s=0.3), "final.norm": gain(W)}
    for i, ly in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", ly["mixer"]
        w[p + "norm1"] = gain(W)
        if ly["type"] == "parallel":
            a, s = m["left"], m["right"]
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                w[q + "left." + n], w[q + f"left.{n}.b"] = r(rows, W, s=W ** -0.5), r(rows, s=0.3)
            w[q + "left.q.norm"], w[q + "left.k.norm"] = gain(H * D, sharp), gain(G * D)
            w[q + "left.o"] = r(W, H * Dv, s=(H * Dv) ** -0.5)
            q += "right."
            H, inner, gn = s["heads"], s["heads"] * s["vdim"], s["groups"] * s["state"]
            w[q + "in"] = r(2 * inner + 2 * gn + H, W, s=W ** -0.5)
            w[q + "conv"], w[q + "conv.b"] = r(inner + 2 * gn, s["conv"], s=0.6), r(inner + 2 * gn, s=0.3)
            w[q + "dt_bias"], w[q + "A_log"], w[q + "D"] = bf(r(H) - 1.0), bf(r(H, s=0.7) - 0.5 - slow), gain(H)
            w[q + "norm"], w[q + "o"] = gain(inner), r(W, inner, s=inner ** -0.5)
        else:
            R, nb = m["width"], m["blocks"]
            wb = R // nb
            for n in ("y", "x"):
                w[q + n], w[q + n + ".b"] = r(R, W, s=1.5 * W ** -0.5), r(R, s=0.3)
            w[q + "conv"], w[q + "conv.b"] = r(R, m["conv"], s=0.6), r(R, s=0.3)
            for n in ("ra", "ri"):
                w[q + n], w[q + n + ".b"] = r(nb, wb, wb, s=2.0 * wb ** -0.5), r(nb, wb, s=0.5)
            w[q + "lam"], w[q + "o"] = bf(r(R) - 3.0 - slow), r(W, R, s=R ** -0.5)
        f = ly.get("mlp")
        if f:
            q = p + "mlp."
            w[p + "norm2"] = gain(W)
            if f["kind"] == "dense":
                w[q + "up"], w[q + "down"] = r(f["ff"], W, s=W ** -0.5), r(W, f["ff"], s=f["ff"] ** -0.5)
            else:
                ff = f["expert"]["ff"]
                w[q + "router"] = r(f["router"]["experts"], W, s=1.5 * W ** -0.5)
                for e in range(f["router"]["experts"]):
                    w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = r(ff, W, s=W ** -0.5), r(ff, W, s=W ** -0.5), r(W, ff, s=ff ** -0.5)
    return w
