"""Plain, slow float64 restatement of the Lodevik decoder: one function per mechanism, whole sequences only, no cache. It shares no code
with the package; the tests compare the engine with it.

``cfg`` is the checkpoint's config.json as a dict, ``w`` maps tensor names to tensors."""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(tokens, bigram):
    """Row of the bigram table for every token: a hash of (previous token, token); the row past the hashed ones for a first token."""
    rows = [bigram["buckets"]]
    for before, now in zip(tokens, tokens[1:]):
        rows.append((before * bigram["mul_prev"] + now * bigram["mul_cur"]) % bigram["buckets"])
    return rows


def embed(tokens, w, emb):
    return w["embed"][torch.tensor(tokens)] * emb["scale"] + w["bigram"][torch.tensor(bigram_rows(tokens, emb["bigram"]))]


def rotate(x, pos, rot):
    """x [..., T, n]: neighbours (2i, 2i + 1) among the first ``dims`` elements turn with the position; the rest pass."""
    out = x.clone()
    for i in range(rot["dims"] // 2):
        a = pos.double() * rot["base"] ** (-2.0 * i / rot["dims"])
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def sees(T, chunk=None):
    """[T, T]: whether a position (row) sees another one. ``chunk``: only inside its own chunk of that many positions."""
    i = torch.arange(T)
    ok = i.view(1, -1) <= i.view(-1, 1)
    return ok if chunk is None else ok & ((i.view(1, -1) // chunk) == (i.view(-1, 1) // chunk))


def weights(s, ok, sink=None):
    """Softmax over the visible keys of s [heads, T, T]; ``sink`` [heads] joins the denominator only."""
    s = s.masked_fill(~ok, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink.view(-1, 1, 1))
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    return e / (den if sink is None else den + torch.exp(sink.view(-1, 1, 1) - top))


def difference_factor(w, p, diff):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def differential(q, k, v, mx, lam, eps):
    """Rotated q [H, 2, T, dim], k [G, 2, T, dim], v [G, T, vdim] -> [H, T, vdim]: the two maps' outputs over the same values, the second
    one subtracted ``lam`` times, normalised per head and scaled."""
    H, T, share = q.shape[0], q.shape[2], q.shape[0] // k.shape[0]
    ok = sees(T, (mx.get("mask") or {}).get("size"))
    out = []
    for h in range(H):
        maps = []
        for m in range(2):
            s = (q[h, m] @ k[h // share, m].T) * mx["scale"]
            if mx.get("softcap"):
                s = mx["softcap"] * torch.tanh(s / mx["softcap"])
            maps.append(weights(s.unsqueeze(0), ok)[0] @ v[h // share])
        out.append(rms(maps[0] - lam * maps[1], eps) * (1 - mx["diff"]))
    return torch.stack(out)


def attention(h, w, p, mx, eps):
    T, H, G, D, V = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    pos = torch.arange(T)
    heads = lambda name, n: (h @ w[p + name].T).view(T, n, 2, D).permute(1, 2, 0, 3)
    q = rotate(rms(heads("q", H), eps) * w[p + "q.norm"], pos, mx["rot"])
    k = rotate(rms(heads("k", G), eps) * w[p + "k.norm"], pos, mx["rot"])
    v = (h @ w[p + "v"].T).view(T, G, V).permute(1, 0, 2)
    o = differential(q, k, v, mx, difference_factor(w, p, mx["diff"]), eps)
    return o.permute(1, 0, 2).reshape(T, H * V) @ w[p + "o"].T


def latent_attention(h, w, p, mx, eps):
    T = h.shape[0]
    H, D, R, V, L = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T).view(T, H, D + R).permute(1, 0, 2)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :L], eps) * w[p + "dkv.norm"]
    kr = rotate(down[:, L:], pos, mx["rot"])
    qn, qr = q[..., :D], rotate(q[..., D:], pos, mx["rot"])
    k = (c @ w[p + "uk"].T).view(T, H, D).permute(1, 0, 2)
    v = (c @ w[p + "uv"].T).view(T, H, V).permute(1, 0, 2)
    s = (qn @ k.transpose(1, 2) + qr @ kr.T) * mx["scale"]
    o = weights(s, sees(T), w[p + "sink"]) @ v * torch.sigmoid(h @ w[p + "g"].T).T.unsqueeze(-1)
    return o.permute(1, 0, 2).reshape(T, H * V) @ w[p + "o"].T


def feed_forward(h, w, p):
    return (gelu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"latent_attention": latent_attention, "attention": attention}


def layer(x, w, i, lc, eps):
    p = f"l{i}."
    x = x + rms(MIXERS[lc["type"]](x, w, p + "mix.", lc["mixer"], eps), eps) * w[p + "norm1"] * w[p + "ls1"]
    if lc.get("mlp"):
        x = x + rms(feed_forward(x, w, p + "mlp."), eps) * w[p + "norm2"] * w[p + "ls2"]
    return x


def forward(cfg, w, tokens, dtype=F64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps, stream = cfg["norm"]["eps"], []
    x = embed(list(tokens), w, cfg["embedding"])
    for i, lc in enumerate(cfg["layers"]):
        x = layer(x, w, i, lc, eps)
        stream.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T * cfg["logit_scale"], torch.stack(stream)


def greedy(cfg, w, tokens, n):
    toks = list(tokens)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(tokens):]
