"""Plain, slow float64 restatement of the Gabisun decoder: one function per mechanism, whole sequences only, no cache. It shares no code
with the package; the tests compare the engine with it.

``cfg`` is the checkpoint's config.json as a dict, ``w`` maps tensor names to tensors."""
import math
from fractions import Fraction

import torch

F64 = torch.float64


def layer_norm(x, w, b, eps):
    m = x.mean(-1, keepdim=True)
    d = x - m
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def distance_bucket(n, buckets, max_dist):
    """Bucket of distance ``n``: exact up to half of the buckets, then logarithmic up to ``max_dist``. The floor of the logarithm's ratio
    is taken exactly: the largest m with (max_dist/half)^m <= (n/half)^(buckets-half)."""
    half = buckets // 2
    if n < half:
        return n
    top = Fraction(n, half) ** (buckets - half)
    m = 0
    while half + m < buckets - 1 and Fraction(max_dist, half) ** (m + 1) <= top:
        m += 1
    return min(buckets - 1, half + m)


def visible(i, j, mask):
    """Whether position i sees position j: causal, inside the window or among the kept first tokens."""
    if j > i:
        return False
    if not mask:
        return True
    return i - j < mask["size"] or j < mask.get("keep_first", 0)


def visibility(T, mask):
    return torch.tensor([[visible(i, j, mask) for j in range(T)] for i in range(T)])


def bias_matrix(T, rel, max_dist):
    """[heads, T, T]: the learned bias of each causal pair."""
    B = rel.shape[0]
    idx = torch.tensor([distance_bucket(n, B, max_dist) for n in range(T)])
    per = rel[idx]                                       # [T (distance), heads]
    i = torch.arange(T).view(T, 1)
    j = torch.arange(T).view(1, T)
    return per[(i - j).clamp(min=0)].permute(2, 0, 1)


def sink_softmax(s, sink):
    """Softmax of ``s`` [heads, q, k] whose denominator also holds exp(sink) of the head."""
    m = torch.maximum(s.max(-1, keepdim=True).values, sink.view(-1, 1, 1))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink.view(-1, 1, 1) - m))


def attention(h, w, p, mx):
    """The mixer: values are the keys, learned distance bias, window with kept first tokens, sink, one sigmoid gate per head."""
    T = h.shape[0]
    H, G, D = mx["heads"], mx["kv_heads"], mx["dim"]
    q = (h @ w[p + "q"].T).view(T, H, D).permute(1, 0, 2)
    k = (h @ w[p + "k"].T).view(T, G, D).permute(1, 0, 2).repeat_interleave(H // G, 0)
    s = q @ k.transpose(1, 2) * mx["scale"] + bias_matrix(T, w[p + "rel"], mx["bias_max"])
    s = s.masked_fill(~visibility(T, mx.get("mask")), -math.inf)
    o = sink_softmax(s, w[p + "sink"]) @ k
    o = o * torch.sigmoid(h @ w[p + "g"].T).T.unsqueeze(-1)
    return o.permute(1, 0, 2).reshape(T, H * D) @ w[p + "o"].T


def feed_forward(h, w, p):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def layer(x, w, i, lc, eps):
    p = f"l{i}."
    norm = lambda name, v: layer_norm(v, w[p + name], w[p + name + ".b"], eps)
    x = x + w[p + "ls1"] * norm("norm1b", attention(norm("norm1", x), w, p + "mix.", lc["mixer"]))
    if lc.get("mlp"):
        x = x + w[p + "ls2"] * norm("norm2b", feed_forward(norm("norm2", x), w, p + "mlp."))
    return x


def layer_runs(cfg):
    """(layer, pass or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)] + [(i, None) for i in range(b, n)]


def enter_pass(x, x0, w, t):
    """What happens ahead of a pass of the looped layers."""
    return torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, w, tokens, dtype=F64):
    """Logits [T, vocab] and the residual stream after every layer run [runs, T, width]."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens)]
    x, stream = x0, []
    for i, t in layer_runs(cfg):
        if t is not None and i == cfg["loop"]["start"]:
            x = enter_pass(x, x0, w, t)
        x = layer(x, w, i, cfg["layers"][i], eps)
        stream.append(x)
    y = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    return y @ w["embed"].T, torch.stack(stream)


def greedy(cfg, w, tokens, n):
    toks = list(tokens)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(tokens):]
