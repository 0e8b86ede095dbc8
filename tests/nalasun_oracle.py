"""Plain, slow float64 restatement of the Nalasun decoder: one function per mechanism, whole sequences only, no cache. It shares no code
with the package; the tests compare the engine with it.

``cfg`` is the checkpoint's config.json as a dict, ``w`` maps tensor names to tensors."""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def embed(tokens, w):
    """Token row plus the row of the position."""
    return w["embed"][torch.tensor(tokens)] + w["pos"][: len(tokens)]


def causal_conv(x, taps, bias=None):
    """x [T, C], taps [C, n]: every channel's last n values weighted, the last tap being the current one; zeros ahead of the sequence."""
    n = taps.shape[1]
    out = torch.zeros_like(x) if bias is None else bias.expand_as(x).clone()
    for back in range(min(n, x.shape[0])):
        out[back:] += taps[:, n - 1 - back] * x[: x.shape[0] - back]
    return out


def temperature(T, coef, every, dtype=F64):
    return 1.0 + coef * torch.log(torch.div(torch.arange(T) + 1, every, rounding_mode="floor").to(dtype) + 1.0)


def distance_penalty(T, r1, r2):
    """[heads, T, T]: what is taken off the score of a key at distance row - column."""
    d = (torch.arange(T).view(-1, 1) - torch.arange(T).view(1, -1)).clamp(min=0).to(r1.dtype)
    return r1.view(-1, 1, 1) * torch.log(1.0 + r2.view(-1, 1, 1) * d)


def softmax_weights(s):
    T = s.shape[-1]
    s = s.masked_fill(torch.arange(T).view(1, -1) > torch.arange(T).view(-1, 1), -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def talk(a, mix):
    """Weights a [heads, T, T] -> sums over the heads with mix [to, from]."""
    return torch.einsum("hg,gij->hij", mix, a)


def attention(h, w, p, mx, eps):
    T, H, G, D = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q = h @ w[p + "q"].T + w[p + "q.b"]
    k = h @ w[p + "k"].T + w[p + "k.b"]
    v = k.view(T, G, D)
    q = (rms(q, eps) * w[p + "q.norm"]).view(T, H, D)
    k = (rms(k, eps) * w[p + "k.norm"]).view(T, G, D)
    if mx.get("q_temp"):
        q = q * temperature(T, mx["q_temp"]["coef"], mx["q_temp"]["every"], q.dtype).view(-1, 1, 1)
    own = [n // (H // G) for n in range(H)]
    s = torch.einsum("ihd,jhd->hij", q, k[:, own]) * mx["scale"] - distance_penalty(T, w[p + "r1"], w[p + "r2"])
    a = talk(softmax_weights(s), w[p + "talk"])
    return torch.einsum("hij,jhd->ihd", a, v[:, own]).reshape(T, H * D) @ w[p + "o"].T


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_steps(q, k, v, g, beta):
    """q, k, g [T, H, D], v [T, H, V], beta [T, H] -> o [T, H, V]; the matrix [D, V] of a head starts at zero."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = S * g[t].unsqueeze(-1)
        u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t].unsqueeze(-1) * u.unsqueeze(-2)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def channel_decay(h, w, p, H):
    a = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    return torch.exp(-torch.exp(w[p + "A_log"]).view(1, H, 1) * softplus(a).view(h.shape[0], H, -1))


def channel_delta(h, w, p, mx, eps):
    T, H, G, D, V = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    conv = lambda n: silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"]))
    own = [n // (H // G) for n in range(H)]
    q = unit(conv("q").view(T, G, D))[:, own] * D ** -0.5
    k = unit(conv("k").view(T, G, D))[:, own]
    v = conv("v").view(T, H, V)
    o = delta_steps(q, k, v, channel_decay(h, w, p, H), torch.sigmoid(h @ w[p + "b"].T))
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, V)
    return (rms(o, eps) * w[p + "norm"] * gate).reshape(T, H * V) @ w[p + "o"].T


def ssm_steps(x, B, C, dt, A_log, D):
    """x [T, H, V], B, C [T, H, N], dt [T, H] -> y [T, H, V]; the state [N, V] of a head starts at zero."""
    T, H, V = x.shape
    S = torch.zeros(H, B.shape[-1], V, dtype=x.dtype)
    out = []
    for t in range(T):
        S = S * torch.exp(-torch.exp(A_log) * dt[t]).view(H, 1, 1) + dt[t].view(H, 1, 1) * B[t].unsqueeze(-1) * x[t].unsqueeze(-2)
        out.append(torch.einsum("hnv,hn->hv", S, C[t]) + D.view(H, 1) * x[t])
    return torch.stack(out)


def mamba2(h, w, p, mx, eps):
    T, H, V, N, G = h.shape[0], mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * V
    z, xbc, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], -1)
    x, B, C = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])).split([inner, G * N, G * N], -1)
    own = [n // (H // G) for n in range(H)]
    y = ssm_steps(x.reshape(T, H, V), B.reshape(T, G, N)[:, own], C.reshape(T, G, N)[:, own], softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, mx["norm_groups"], -1), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def gated(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, router, top, scale):
    """[T, experts]: the factor of every expert, zero where it is not chosen."""
    s = torch.sigmoid(h @ router.T)
    out = torch.zeros_like(s)
    for t in range(h.shape[0]):
        for e in sorted(range(s.shape[1]), key=lambda e: -float(s[t, e]))[:top]:
            out[t, e] = s[t, e] * scale
    return out


def experts(h, w, p, mlp):
    r = mlp["router"]
    factor = route(h, w[p + "router"], r["top"], r["scale"])
    out = sum(factor[:, e: e + 1] * gated(h, w, f"{p}e{e}.") for e in range(r["experts"]))
    return out + gated(h, w, p + "shared.") if mlp.get("shared") else out


MIXERS = {"attention": attention, "channel_delta": channel_delta, "mamba2": mamba2}


def layer(x, w, i, lc, eps):
    p = f"l{i}."
    h = rms(x, eps) * w[p + "norm1"]
    h = h + causal_conv(h, w[p + "canon1"])
    x = x + MIXERS[lc["type"]](h, w, p + "mix.", lc["mixer"], eps)
    if lc.get("mlp"):
        x = x + experts(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", lc["mlp"])
    return x


def forward(cfg, w, tokens, dtype=F64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps, stream = cfg["norm"]["eps"], []
    x = embed(list(tokens), w)
    for i, lc in enumerate(cfg["layers"]):
        x = layer(x, w, i, lc, eps)
        stream.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T, torch.stack(stream)


def greedy(cfg, w, tokens, n):
    toks = list(tokens)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(tokens):]
