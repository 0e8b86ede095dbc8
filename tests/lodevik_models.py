"""Small random Lodevik checkpoints for the tests (not a test file)."""
import torch

from gabisun_models import save  # noqa: F401  (same checkpoint layout)


def attn(heads, kv, dim, vdim, rot, chunk, ff, cap=15.0, diff=0.4, scale=None, base=700.0):
    return dict(type="attention", mlp=dict(kind="dense", ff=ff) if ff else None, mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, diff=diff,
                rot=dict(base=base, dims=rot), scale=scale or 1.2 * dim ** -0.5, softcap=cap, mask=dict(size=chunk) if chunk else None))


def latent(heads, dim, rot_dim, vdim, kv_rank, ff, scale=None, base=3000.0):
    return dict(type="latent_attention", mlp=dict(kind="dense", ff=ff) if ff else None, mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim,
                kv_rank=kv_rank, scale=scale or 1.1 * (dim + rot_dim) ** -0.5, rot=dict(base=base, dims=rot_dim)))


def config(width, vocab, layers, scale=2.0, buckets=97, muls=(31, 7), logit_scale=0.8, eps=1e-5):
    return dict(architecture="Lodevik", width=width, vocab=vocab, layers=layers, norm=dict(eps=eps), logit_scale=logit_scale,
                embedding=dict(scale=scale, bigram=dict(buckets=buckets, mul_prev=muls[0], mul_cur=muls[1])))


# unlike layers, orders and sizes: head, value, latent and feed-forward sizes that are no multiples of the kernels' tiles, one to eight query
# heads per key head, rotations of all, a part and none of a map, chunks of one position up to longer than every sequence and none at all,
# layers without a feed-forward, factors of 1, one kind of mixer only, rows too wide for the tensor-core kernels
CONFIGS = {
    "mixed": config(128, 210, [attn(6, 3, 16, 24, 4, 37, 160, cap=6.0, diff=0.3), latent(4, 24, 8, 16, 40, None), latent(2, 32, 16, 48, 64, 72),
                               attn(2, 1, 48, 96, 48, 100, None, diff=0.8)], buckets=301, muls=(1009, 613)),
    "odd": config(100, 133, [attn(5, 5, 18, 22, 6, 1, 44, diff=0.1), latent(3, 20, 6, 10, 36, 52, base=50.0), attn(3, 1, 140, 300, 10, 70, None, cap=30.0),
                             attn(4, 2, 9, 15, 8, 24, 20)], scale=1.0, buckets=2, muls=(1, 1), logit_scale=1.0, eps=1e-3),
    "wide": config(192, 301, [attn(8, 1, 64, 128, 32, 64, 256), attn(4, 4, 128, 200, 0, 129, 320, cap=50.0), latent(16, 64, 64, 64, 256, 192),
                              attn(6, 2, 32, 40, 32, None, 64, cap=None)], scale=5.0, buckets=5003, muls=(70001, 90001)),
    "chunks": config(96, 90, [attn(4, 2, 32, 64, 16, 30, 100, cap=8.0), attn(3, 3, 24, 32, 8, 50, None, diff=0.6)]),
    "latents": config(96, 75, [latent(2, 40, 10, 16, 512, None), latent(7, 8, 2, 8, 12, 90)], logit_scale=2.0),
}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random bf16 weights. Norm weights, layer scales, sinks, gates and the numbers of lambda are far from their neutral values; ``sharp``
    scales queries and keys, so that single keys stand out."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).bfloat16()
    W, V, emb = cfg["width"], cfg["vocab"], cfg["embedding"]
    w = {"embed": n(V, W, std=1.0 / emb["scale"]), "bigram": n(emb["bigram"]["buckets"] + 1, W, std=0.7), "final.norm": n(W, std=0.2, mean=1.0)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        H, D, U = m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "ls1"] = n(W, std=0.2, mean=1.0), n(W, std=0.3, mean=0.7)
        if l["type"] == "latent_attention":
            R, L = m["rot_dim"], m["kv_rank"]
            w[p + "mix.q"], w[p + "mix.dkv"] = n(H * (D + R), W, std=sharp * W ** -0.5), n(L + R, W, std=sharp * W ** -0.5)
            w[p + "mix.dkv.norm"], w[p + "mix.sink"], w[p + "mix.g"] = n(L, std=0.2, mean=1.0), n(H, std=1.5), n(H, W, std=W ** -0.5)
            w[p + "mix.uk"], w[p + "mix.uv"] = n(H * D, L, std=sharp * L ** -0.5), n(H * U, L, std=L ** -0.5)
        else:
            G = m["kv_heads"]
            w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"] = (n(r, W, std=W ** -0.5) for r in (H * 2 * D, G * 2 * D, G * U))
            w[p + "mix.q.norm"], w[p + "mix.k.norm"] = n(D, std=0.3 * sharp, mean=sharp), n(D, std=0.3 * sharp, mean=sharp)
            for x in ("lq1", "lk1", "lq2", "lk2"):
                w[p + "mix." + x] = n(D, std=0.6 * D ** -0.25)
        w[p + "mix.o"] = n(W, H * U, std=(H * U) ** -0.5)
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            w[p + "norm2"], w[p + "ls2"] = n(W, std=0.2, mean=1.0), n(W, std=0.3, mean=0.7)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = n(ff, W, std=W ** -0.5), n(ff, W, std=W ** -0.5), n(W, ff, std=ff ** -0.5)
    return w
