"""Plain, slow float64 restatement of the Sepirax decoder: one function per mechanism, whole sequences only, no cache. It shares no code
with the package; the tests compare the engine with it.

``cfg`` is the checkpoint's config.json as a dict, ``w`` maps tensor names to tensors."""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def yarn_frequencies(dims, base, scaling):
    """Rotary frequencies and the factor on cos and sin. Slow pairs are divided by ``factor``, fast ones stay, with a linear ramp between
    the pairs that turn ``fast`` and ``slow`` times within the original context."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=F64), 1.0
    turns = lambda t: dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / scaling["factor"] * r + v * (1 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, pos, rot):
    """x [..., T, n]: pairs (i, i + dims/2) of the first ``dims`` elements turn with the position; the rest pass."""
    d = rot["dims"]
    f, m = yarn_frequencies(d, rot["base"], rot.get("scaling"))
    a = pos.double().view(-1, 1) * f
    c, s = (torch.cos(a) * m).to(x.dtype), (torch.sin(a) * m).to(x.dtype)
    u, v = x[..., : d // 2], x[..., d // 2: d]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., d:]], -1)


def causal_softmax(s):
    T = s.shape[-1]
    s = s.masked_fill(~torch.tril(torch.ones(T, T, dtype=torch.bool)), -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_attention(h, w, p, mx, eps):
    T = h.shape[0]
    H, D, R, V, L = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = torch.arange(T)
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, D + R).permute(1, 0, 2)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :L], eps) * w[p + "dkv.norm"]
    kr = rotate(down[:, L:], pos, mx["rot"])
    qn, qr = q[..., :D], rotate(q[..., D:], pos, mx["rot"])
    k = (c @ w[p + "uk"].T).view(T, H, D).permute(1, 0, 2)
    v = (c @ w[p + "uv"].T).view(T, H, V).permute(1, 0, 2)
    s = (qn @ k.transpose(1, 2) + qr @ kr.T) * mx["scale"]
    o = (causal_softmax(s) @ v).permute(1, 0, 2).reshape(T, H * V)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mlstm_cell(q, k, v, i, f, state=None):
    """q, k [T, heads, dim], v [T, heads, vdim], log gates i, f [T, heads]. Returns the outputs and the (S, n, m) that follow."""
    T, H, D = q.shape
    z = lambda *s: torch.zeros(*s, dtype=q.dtype)
    S, n, m = state if state is not None else (z(H, D, v.shape[2]), z(H, D), z(H))
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new).view(H, 1), torch.exp(i[t] - new).view(H, 1)
        S = keep.unsqueeze(-1) * S + (put * k[t]).unsqueeze(-1) * v[t].unsqueeze(1)
        n = keep * n + put * k[t]
        m = new
        dot = (n * q[t]).sum(-1)
        out.append((S * q[t].unsqueeze(-1)).sum(1) / (torch.maximum(dot.abs(), torch.exp(-m)) + 1e-6).view(H, 1))
    return torch.stack(out), (S, n, m)


def log_gates(h, w, p, cap):
    """Log input gate and log forget gate [T, heads]."""
    cut = lambda z: cap * torch.tanh(z / cap)
    fz = cut(h @ w[p + "f"].T + w[p + "f.b"])
    return cut(h @ w[p + "i"].T + w[p + "i.b"]), -torch.log1p(torch.exp(-fz))


def mlstm(h, w, p, mx, eps):
    T = h.shape[0]
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    i, f = log_gates(h, w, p, mx["gate_cap"])
    o = rms(mlstm_cell(q, k, v, i, f)[0], eps).reshape(T, H * V)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def choose_experts(z, router):
    """Router logits [T, experts] -> for every token the list of (expert, weight)."""
    out, E = [], router["experts"]
    g = router.get("groups") or dict(count=1, keep=1)
    size = E // g["count"]
    for row in torch.softmax(z, -1):
        s = row.tolist()
        best = sorted(range(g["count"]), key=lambda a: -max(s[a * size:(a + 1) * size]))[: g["keep"]]
        cand = [e for e in range(E) if e // size in best]
        top = sorted(cand, key=lambda e: -s[e])[: router["top"]]
        total = sum(s[e] for e in top) + 1e-20
        out.append([(e, s[e] / total) for e in top])
    return out


def experts(h, w, p, mlp):
    picks = choose_experts(h @ w[p + "router"].T, mlp["router"])
    weight = torch.zeros(h.shape[0], mlp["router"]["experts"], dtype=h.dtype)
    for t, row in enumerate(picks):
        for e, a in row:
            weight[t, e] = a
    out = torch.zeros_like(h)
    for e in range(weight.shape[1]):
        n = f"{p}e{e}."
        out = out + weight[:, e:e + 1] * ((silu(h @ w[n + "gate"].T) * (h @ w[n + "up"].T)) @ w[n + "down"].T)
    return out


MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm}


def layer(x, w, i, lc, cfg):
    p, m = f"l{i}.", cfg["residual_mult"]
    norm = lambda name: dynamic_tanh(x, w[p + name + ".alpha"], w[p + name], w[p + name + ".b"])
    x = x + m * MIXERS[lc["type"]](norm("norm1"), w, p + "mix.", lc["mixer"], cfg["norm"]["eps"])
    if lc.get("mlp"):
        x = x + m * experts(dynamic_tanh(x, w[p + "norm2.alpha"], w[p + "norm2"], w[p + "norm2.b"]), w, p + "mlp.", lc["mlp"])
    return x


def forward(cfg, w, tokens, dtype=F64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: v.to(dtype) for k, v in w.items()}
    x, stream = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"], []
    for i, lc in enumerate(cfg["layers"]):
        x = layer(x, w, i, lc, cfg)
        stream.append(x)
    lg = dynamic_tanh(x, w["final.norm.alpha"], w["final.norm"], w["final.norm.b"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return (cap * torch.tanh(lg / cap) if cap else lg), torch.stack(stream)


def greedy(cfg, w, tokens, n):
    toks = list(tokens)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(tokens):]
