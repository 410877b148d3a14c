"""Helpers of the Nagosun tests: small random models (config dict + weights under the design's tensor names)."""
import math

import torch


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=12, size=24, softcap=6.0, scale=None, mlp="default"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.5 / math.sqrt(dim)}
    if softcap:
        m["softcap"] = softcap
    if size:
        m["mask"] = {"size": size}
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "default" else mlp}


def latent_layer(heads=3, dim=12, rot_dim=8, vdim=20, kv_rank=24, base=300.0, size=24, scale=None, mlp="default"):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim),
         "rot": {"dims": rot_dim, "base": base}}
    if size:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": dense() if mlp == "default" else mlp}


def make_config(layers, vocab=83, width=44, eps=1e-5, groups=2, mult=0.7, logit_scale=1.75):
    return {"architecture": "Nagosun", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "residual_mult": mult,
            "logit_scale": logit_scale, "layers": layers}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random weights, rounded to bfloat16 values (held as float32) so that every dtype sees the same numbers.  `sharp` scales the query
    projections: large values make the softmax maps peaked, so that a key wrongly seen or missed moves the output."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    bf = lambda t: t.to(torch.bfloat16).to(torch.float32)
    r = lambda *shape, s=1.0: bf(torch.randn(*shape, generator=g) * s)
    gain = lambda n: bf(1.0 + 0.3 * torch.randn(n, generator=g))
    w = {"embed": r(cfg["vocab"], W, s=0.2), "embed.norm": gain(W), "head": r(cfg["vocab"], W, s=2.0 * W ** -0.5), "final.norm": gain(W)}
    for i, ly in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", ly["mixer"]
        w[p + "norm1"], w[p + "norm1b"] = gain(W), gain(W)
        w[p + "rg1"], w[p + "rg1.b"] = r(W, W, s=1.5 * W ** -0.5), r(W, s=0.5)
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        if ly["type"] == "latent_attention":
            R, K = m["rot_dim"], m["kv_rank"]
            w[q + "q"] = r(H * (D + R), W, s=sharp * 2.0 * W ** -0.5)
            w[q + "dkv"], w[q + "dkv.norm"] = r(K + R, W, s=W ** -0.5), gain(K)
            w[q + "uk"], w[q + "uv"] = r(H * D, K, s=2.0 * K ** -0.5), r(H * Dv, K, s=K ** -0.5)
        else:
            G = m["kv_heads"]
            w[q + "q"], w[q + "q.b"] = r(H * D, W, s=sharp * W ** -0.5), r(H * D, s=0.3)
            w[q + "k"], w[q + "k.b"] = r(G * D, W, s=W ** -0.5), r(G * D, s=0.3)
            w[q + "v"], w[q + "v.b"] = r(G * Dv, W, s=W ** -0.5), r(G * Dv, s=0.3)
            w[q + "g"], w[q + "o.b"] = r(H * Dv, W, s=2.0 * W ** -0.5), r(W, s=0.3)
        w[q + "o"] = r(W, H * Dv, s=(H * Dv) ** -0.5)
        f = ly.get("mlp")
        if f:
            q = p + "mlp."
            w[p + "norm2"], w[p + "norm2b"] = gain(W), gain(W)
            w[p + "rg2"], w[p + "rg2.b"] = r(W, W, s=1.5 * W ** -0.5), r(W, s=0.5)
            w[q + "gate"], w[q + "up"], w[q + "down"] = r(f["ff"], W, s=2.0 * W ** -0.5), r(f["ff"], W, s=W ** -0.5), r(W, f["ff"], s=f["ff"] ** -0.5)
    return w
