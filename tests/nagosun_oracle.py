"""Plain float64 restatement of the Nagosun family, one function per mechanism, for the tests.  Whole sequences only: no cache, no batching --
the engine's paged / chunked / batched results are compared against this.

Notation: n tokens at positions 0 .. n-1, h the [n, width] input of a sublayer, weights under the design's tensor names (a mixer sees them
without the "<layer>.mix." prefix).  Linear weights are [out, in]."""
import math

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, gain, groups, eps):
    """Every one of `groups` equal runs of neighbouring entries is brought to unit RMS by itself; then the gain, entry by entry."""
    runs = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return unit_rms(runs, eps).reshape(x.shape) * gain


def silu(z):
    return z / (1.0 + torch.exp(-z))


def logistic(z):
    return 1.0 / (1.0 + torch.exp(-z))


def turn_neighbours(x, base, dims):
    """x [n, ..., d] at positions 0 .. n-1: entries (2i, 2i+1) of the first `dims`, read as a complex number, are turned by
    position * base^(-2i / dims); the rest passes."""
    n = x.shape[0]
    rate = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    angle = (torch.arange(n, dtype=F64)[:, None] * rate).reshape(n, *([1] * (x.dim() - 2)), dims // 2)
    z = torch.complex(x[..., 0:dims:2], x[..., 1:dims:2]) * torch.polar(torch.ones_like(angle), angle)
    out = x.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = z.real, z.imag
    return out


def in_window(n, size):
    """[query, key] table: the key is not later than the query and fewer than `size` positions before it (size 0: any number)."""
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) & ((back < size) if size else (back >= 0))


def cap_scores(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def softmax_plus_one(s, seen):
    """Softmax over the seen keys of each row whose denominator has one more term exp(0) that weighs nothing."""
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    top = s.max(-1, keepdim=True).values.clamp_min(0.0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def attention(h, m, w, eps):
    """Grouped heads with unit-RMS values, capped scores less a distance penalty, a sliding window, a spare term in the softmax, a gate per
    output number; biases on the q / k / v / output projections."""
    n, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).reshape(n, H, D)
    k = (h @ w["k"].T + w["k.b"]).reshape(n, G, D)
    v = unit_rms((h @ w["v"].T + w["v.b"]).reshape(n, G, Dv), eps)
    seen = in_window(n, (m.get("mask") or {}).get("size", 0))
    far = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).to(F64)
    heads = []
    for i in range(H):
        g = i // (H // G)
        s = cap_scores(q[:, i] @ k[:, g].T * m["scale"], m.get("softcap")) - slope(i, H) * far
        heads.append(softmax_plus_one(s, seen) @ v[:, g])
    out = torch.cat(heads, 1) * logistic(h @ w["g"].T)
    return out @ w["o"].T + w["o.b"]


def latent_attention(h, m, w, eps):
    """Every head's keys and values are linear images of one small normed latent per position; a second, turned key part is shared by the
    heads.  Plain softmax over a sliding window."""
    n, H, D, R, Dv, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).reshape(n, H, D + R)
    down = h @ w["dkv"].T
    c = unit_rms(down[:, :K], eps) * w["dkv.norm"]
    k_shared, q_turned = down[:, K:], q[:, :, D:]
    if m.get("rot"):
        k_shared = turn_neighbours(k_shared, m["rot"]["base"], m["rot"]["dims"])
        q_turned = turn_neighbours(q_turned, m["rot"]["base"], m["rot"]["dims"])
    keys, values = (c @ w["uk"].T).reshape(n, H, D), (c @ w["uv"].T).reshape(n, H, Dv)
    seen = in_window(n, (m.get("mask") or {}).get("size", 0))
    heads = []
    for i in range(H):
        s = (q[:, i, :D] @ keys[:, i].T + q_turned[:, i] @ k_shared.T) * m["scale"]
        heads.append(torch.softmax(torch.where(seen, s, torch.full_like(s, -math.inf)), -1) @ values[:, i])
    return torch.cat(heads, 1) @ w["o"].T


def feed_forward(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def residual_gate(h, w, b):
    return logistic(h @ w.T + b)


MIXERS = {"latent_attention": latent_attention, "attention": attention}


# ---------------------------------------------------------------------------------------------------------------------------------
# the stack: a sublayer reads the normed stream; its output, gated by the same input, is normed again, weighed and added
# ---------------------------------------------------------------------------------------------------------------------------------
def forward(cfg, weights, tokens, taps=None):
    """Logits [n, vocab] (float64) of a whole sequence.  taps: a list that receives the stream after every layer."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps, groups, mult = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
    norm = lambda x, name: grouped_norm(x, w[name], groups, eps)
    x = norm(w["embed"][torch.tensor(tokens)], "embed.norm")
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        sub = lambda kind: {k[len(p) + len(kind) + 1:]: v for k, v in w.items() if k.startswith(p + kind + ".")}
        h = norm(x, p + "norm1")
        y = MIXERS[ly["type"]](h, ly["mixer"], sub("mix"), eps)
        x = x + mult * norm(y * residual_gate(h, w[p + "rg1"], w[p + "rg1.b"]), p + "norm1b")
        if ly.get("mlp"):
            h = norm(x, p + "norm2")
            y = feed_forward(h, sub("mlp"))
            x = x + mult * norm(y * residual_gate(h, w[p + "rg2"], w[p + "rg2.b"]), p + "norm2b")
        if taps is not None:
            taps.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n_new):
    """n_new tokens by argmax, re-running the whole sequence every time."""
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(cfg, weights, toks)[-1])))
    return toks[len(prompt):]
