"""Small random Sepirax checkpoints for the tests (not a test file)."""
import json
import os

import torch
from safetensors.torch import save_file


def moe(experts, top, ff, count=1, keep=1):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, groups=dict(count=count, keep=keep)))


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, mlp=None, scale=None, base=1000.0, factor=2.5, original=64, fast=8.0, slow=0.5):
    rot = dict(base=base, dims=rot_dim, scaling=dict(factor=factor, original=original, fast=fast, slow=slow) if factor else None)
    return dict(type="latent_attention", mlp=mlp, mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank,
                scale=scale or 1.1 * (dim + rot_dim) ** -0.5, rot=rot))


def mlstm(heads, dim, vdim, mlp=None, cap=12.0):
    return dict(type="mlstm", mlp=mlp, mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap))


def config(width, vocab, layers, mult=0.6, scale=3.0, cap=20.0, eps=1e-5):
    return dict(architecture="Sepirax", width=width, vocab=vocab, layers=layers, norm=dict(eps=eps), residual_mult=mult, embedding=dict(scale=scale),
                logit_softcap=cap)


# unlike layers, orders and sizes: head, latent and value sizes that are no multiples of the kernels' tiles, one group and many, every
# expert used and one of them, layers without a feed-forward, a residual factor and an embedding scale of 1, one kind of mixer only
CONFIGS = {
    "mixed": config(128, 210, [mlstm(2, 24, 40, moe(6, 2, 48, 3, 2)), latent(4, 16, 8, 24, 40, 56, moe(12, 3, 32, 4, 1)), mlstm(3, 64, 32, None, cap=5.0),
                               latent(2, 32, 16, 48, 64, 32, None, factor=8.0, original=32, fast=4.0, slow=1.0)]),
    "odd": config(100, 133, [latent(3, 20, 6, 10, 36, 30, moe(5, 5, 20), base=50.0), mlstm(5, 9, 21, moe(7, 1, 36, 7, 3)), mlstm(1, 130, 70, moe(4, 2, 8, 2, 2))],
                  mult=1.0, scale=1.0, cap=7.0, eps=1e-3),
    "wide": config(192, 301, [mlstm(2, 128, 256, moe(40, 6, 64, 8, 3)), latent(16, 64, 32, 64, 256, 96, moe(32, 4, 128, 4, 2)),
                              latent(5, 48, 64, 32, 130, 64, moe(64, 8, 32, 1, 1), factor=None)], mult=0.3, scale=8.0),
    "latents": config(96, 90, [latent(2, 40, 10, 16, 512, 24, None), latent(7, 8, 2, 8, 12, 16, moe(3, 2, 16, 3, 3))]),
    "memories": config(64, 75, [mlstm(4, 16, 16, moe(4, 2, 24, 2, 1), cap=30.0), mlstm(2, 256, 320, None)], cap=50.0),
}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random bf16 weights. Norm weights, biases and gates are far from their neutral values; the forget gates of different heads keep
    from a few to thousands of tokens; ``sharp`` scales queries and keys, so that single keys stand out."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).bfloat16()
    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": n(V, W, std=1.0 / cfg["embedding"]["scale"]), "head": n(V, W, std=1.5 * W ** -0.5)}

    def norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = n(W, std=0.2, mean=1.0), n(W, std=0.2), (0.5 + torch.rand((), generator=g)).bfloat16()
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        norm(p + "norm1")
        H, D, U = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "latent_attention":
            R, L, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            w[p + "mix.dq"], w[p + "mix.dq.norm"] = n(Q, W, std=W ** -0.5), n(Q, std=0.2, mean=1.0)
            w[p + "mix.uq"] = n(H * (D + R), Q, std=sharp * Q ** -0.5)
            w[p + "mix.dkv"], w[p + "mix.dkv.norm"] = n(L + R, W, std=sharp * W ** -0.5), n(L, std=0.2, mean=1.0)
            w[p + "mix.uk"], w[p + "mix.uv"] = n(H * D, L, std=sharp * L ** -0.5), n(H * U, L, std=L ** -0.5)
        else:
            for x, r in (("q", D), ("k", D), ("v", U)):
                w[p + "mix." + x] = n(H * r, W, std=W ** -0.5)
            w[p + "mix.norm"] = n(H * U, std=0.2, mean=1.0)
            w[p + "mix.i"], w[p + "mix.i.b"] = n(H, W, std=W ** -0.5), n(H)
            w[p + "mix.f"], w[p + "mix.f.b"] = n(H, W, std=W ** -0.5), torch.linspace(1.0, 8.0, H).bfloat16()
        w[p + "mix.g"], w[p + "mix.o"] = n(H * U, W, std=W ** -0.5), n(W, H * U, std=1.5 * (H * U) ** -0.5)
        if l["mlp"]:
            norm(p + "norm2")
            ff, E = l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"]
            w[p + "mlp.router"] = n(E, W, std=3 * W ** -0.5)
            for e in range(E):
                w[f"{p}mlp.e{e}.gate"], w[f"{p}mlp.e{e}.up"] = n(ff, W, std=W ** -0.5), n(ff, W, std=W ** -0.5)
                w[f"{p}mlp.e{e}.down"] = n(W, ff, std=2 * ff ** -0.5)
    return w


def save(cfg, w, path):
    os.makedirs(path, exist_ok=True)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return str(path)
