"""Plain float64 restatement of the Tumitar family, one function per mechanism, for the tests.  Whole sequences only: no cache, no batching --
the engine's paged / portioned / batched results are compared against this.

Notation: n tokens at positions 0 .. n-1, h the [n, width] input of a sublayer, weights under the design's tensor names (a mixer sees them
without the "<layer>.mix." prefix, a feed-forward without "<layer>.mlp.").  Linear weights are [out, in]."""
import math

import torch

F64 = torch.float64


def rms_norm(x, gain, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def logistic(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * logistic(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp_min(0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(x, taps, bias):
    """x [n, channels]: every channel's weighted sum of its own latest values, the last column of `taps` for the current one."""
    n, k = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, x.shape[1], dtype=F64), x])
    return sum(padded[j:j + n] * taps[:, j] for j in range(k)) + bias


def query_temperature(n, coef, every):
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(n)], dtype=F64)


def softmax_plus_one(s):
    """Causal softmax of a square score table whose denominators have one more term exp(0) that weighs nothing."""
    n = s.shape[0]
    s = torch.where(torch.tril(torch.ones(n, n, dtype=torch.bool)), s, torch.full_like(s, -math.inf))
    top = s.max(-1, keepdim=True).values.clamp_min(0.0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def attention(h, m, w, eps):
    """Grouped heads without positions in the scores: biased projections, q and k normed over the whole projection, queries that grow with the
    position, one spare term in the softmax."""
    n, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w["q"].T + w["q.b"], w["q.norm"], eps) * query_temperature(n, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
    k = rms_norm(h @ w["k"].T + w["k.b"], w["k.norm"], eps)
    v = h @ w["v"].T + w["v.b"]
    q, k, v = q.reshape(n, H, D), k.reshape(n, G, D), v.reshape(n, G, Dv)
    heads = []
    for i in range(H):
        g = i // (H // G)
        heads.append(softmax_plus_one(q[:, i] @ k[:, g].T * m["scale"]) @ v[:, g])
    return torch.cat(heads, 1) @ w["o"].T


def state_space(h, m, w, eps):
    """Per head a [state, vdim] matrix that forgets by one number per token and takes a scaled outer product."""
    n, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = (h @ w["in"].T).split([inner, inner + 2 * G * N, H], 1)
    x, B, C = silu(short_conv(xbc, w["conv"], w["conv.b"])).split([inner, G * N, G * N], 1)
    x, B, C = x.reshape(n, H, P), B.reshape(n, G, N), C.reshape(n, G, N)
    dt = softplus(dt + w["dt_bias"])
    y = torch.zeros(n, H, P, dtype=F64)
    for i in range(H):
        g = i // (H // G)
        S = torch.zeros(N, P, dtype=F64)
        for t in range(n):
            S = torch.exp(-torch.exp(w["A_log"][i]) * dt[t, i]) * S + dt[t, i] * torch.outer(B[t, g], x[t, i])
            y[t, i] = S.T @ C[t, g] + w["D"][i] * x[t, i]
    y = y.reshape(n, inner) * silu(z)
    parts = y.reshape(n, m["norm_groups"], inner // m["norm_groups"])
    return (rms_norm(parts, 1.0, eps).reshape(n, inner) * w["norm"]) @ w["o"].T


def side_by_side(h, m, w, eps):
    sub = lambda side: {k[len(side) + 1:]: t for k, t in w.items() if k.startswith(side + ".")}
    return m["left_scale"] * attention(h, m["left"], sub("left"), eps) + m["right_scale"] * state_space(h, m["right"], sub("right"), eps)


def gated_linear_unit(h, m, w, eps):
    """A diagonal recurrence whose decay and input gate are logistic functions of the convolved input, beside a gelu branch."""
    n, nb = h.shape[0], m["blocks"]
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = short_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    parts = u.reshape(n, nb, -1)
    gate = lambda name: logistic(torch.einsum("nbi,boi->nbo", parts, w[name]) + w[name + ".b"].reshape(nb, -1)).reshape(n, -1)
    r, i = gate("ra"), gate("ri")
    a = torch.exp(-8.0 * r * softplus(w["lam"]))
    S, out = torch.zeros_like(u[0]), []
    for t in range(n):
        S = a[t] * S + torch.sqrt(1.0 - a[t] ** 2) * i[t] * u[t]
        out.append(S)
    return (torch.stack(out) * y) @ w["o"].T


MIXERS = {"parallel": side_by_side, "rglru": gated_linear_unit}


def dense_ff(h, w):
    return (h @ w["up"].T).clamp_min(0.0) ** 2 @ w["down"].T


def experts_ff(h, c, w):
    top, scale = c["router"]["top"], c["router"]["scale"]
    s = logistic(h @ w["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.argsort(s[t], descending=True, stable=True)[:top].tolist():
            out[t] += scale * s[t, e] * (w[f"e{e}.down"] @ (silu(w[f"e{e}.gate"] @ h[t]) * (w[f"e{e}.up"] @ h[t])))
    return out


def layer_runs(cfg):
    """(layer, whether the embedding output joins the stream ahead of it) of every layer run."""
    n, lp = len(cfg["layers"]), cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    span = list(range(lp["start"], lp["stop"]))
    looped = [(i, p > 0 and i == lp["start"]) for p in range(lp["times"]) for i in span]
    return [(i, False) for i in range(lp["start"])] + looped + [(i, False) for i in range(lp["stop"], n)]


def forward(cfg, weights, tokens, taps=None):
    """Logits [n, vocab] (float64) of a whole sequence.  taps: a list that receives the stream after every layer run."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = start = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, again in layer_runs(cfg):
        p, ly = f"l{i}.", cfg["layers"][i]
        sub = lambda kind: {k[len(p) + len(kind) + 1:]: v for k, v in w.items() if k.startswith(p + kind + ".")}
        if again:
            x = x + start
        x = x + MIXERS[ly["type"]](rms_norm(x, w[p + "norm1"], eps), ly["mixer"], sub("mix"), eps)
        if ly.get("mlp"):
            h = rms_norm(x, w[p + "norm2"], eps)
            x = x + (dense_ff(h, sub("mlp")) if ly["mlp"]["kind"] == "dense" else experts_ff(h, ly["mlp"], sub("mlp")))
        if taps is not None:
            taps.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, weights, prompt, n_new):
    """n_new tokens by argmax, re-running the whole sequence every time."""
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(cfg, weights, toks)[-1])))
    return toks[len(prompt):]
