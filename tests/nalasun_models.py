"""Small random Nalasun checkpoints for the tests (not a test file)."""
import torch

from gabisun_models import save  # noqa: F401  (same checkpoint layout)


def moe(experts, top, ff, shared, scale=1.3):
    return dict(kind="moe", expert=dict(ff=ff), shared=dict(ff=shared), router=dict(experts=experts, top=top, scale=scale))


def attn(heads, kv, dim, mlp, coef=0.25, every=37, scale=None):
    return dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale or 1.1 * dim ** -0.5, q_temp=dict(coef=coef, every=every)))


def delta(heads, kv, dim, vdim, mlp, conv=3):
    return dict(type="channel_delta", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv))


def mamba(heads, vdim, state, groups, norm_groups, mlp, conv=4):
    return dict(type="mamba2", mlp=mlp, mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv))


def config(width, vocab, layers, taps=3, eps=1e-5, positions=400, ranks=(10, 14)):
    return dict(architecture="Nalasun", width=width, vocab=vocab, layers=layers, max_positions=positions, norm=dict(eps=eps), canon=dict(taps=taps)), ranks


# Unlike layers, orders and sizes: head, value, state and feed-forward sizes that are no multiples of the kernels' tiles, one to sixteen query heads per
# key head, convolutions of one to seven taps, norm groups that are not the state's groups, layers without a feed-forward, one kind of mixer only.
# Every token takes every expert, so that no close call of a router separates bf16 from float64; "routed" is for fp32.
CONFIGS = {
    "mixed": config(128, 210, [attn(6, 3, 40, moe(3, 3, 48, 56)), delta(4, 2, 24, 40, None), mamba(6, 16, 24, 2, 3, moe(2, 2, 72, 20, 0.7)), attn(4, 1, 64, None)]),
    "odd": config(100, 133, [mamba(3, 10, 18, 1, 1, moe(1, 1, 20, 12), conv=2), delta(3, 3, 9, 15, moe(2, 2, 36, 44, 1.0), conv=5), attn(5, 5, 12, moe(3, 3, 28, 52), 0.6, 1),
                             attn(3, 1, 150, None)], taps=5, eps=1e-3, ranks=(5, 3)),
    "wide": config(192, 301, [attn(16, 1, 32, moe(2, 2, 64, 128)), mamba(8, 64, 64, 4, 2, None), delta(2, 1, 128, 64, moe(2, 2, 128, 64)), attn(8, 8, 64, None, 0.1, 100)],
                   taps=2, ranks=(64, 32)),
    "states": config(96, 90, [delta(2, 2, 64, 96, None), mamba(2, 48, 128, 1, 2, moe(2, 2, 40, 40))], taps=7),
    "heads": config(96, 75, [attn(12, 2, 20, None, 0.4, 64), attn(33, 11, 8, moe(1, 1, 90, 30))], taps=1),
    "routed": config(64, 80, [attn(2, 1, 32, moe(12, 3, 24, 16, 1.7)), delta(2, 1, 16, 16, moe(7, 2, 16, 8)), mamba(2, 16, 16, 1, 1, moe(5, 1, 20, 4))], taps=4),
}
RANKS = {k: r for k, (_, r) in CONFIGS.items()}
CONFIGS = {k: c for k, (c, _) in CONFIGS.items()}


def make_weights(cfg, seed=0, ranks=(10, 14), sharp=1.0):
    """Random bf16 weights, norms, biases and mixes far from their neutral values; ``sharp`` scales queries, so that single keys stand out."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).bfloat16()
    u = lambda *s, lo, hi: (torch.rand(*s, generator=g) * (hi - lo) + lo).bfloat16()
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    lin = lambda o, i: n(o, i, std=i ** -0.5)
    w = {"embed": n(V, W), "pos": n(cfg["max_positions"], W, std=0.5), "final.norm": n(W, std=0.2, mean=1.0)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        q = p + "mix."
        H = m["heads"]
        w[p + "norm1"], w[p + "canon1"] = n(W, std=0.2, mean=1.0), n(W, taps, std=0.5 * taps ** -0.5)
        if l["type"] == "attention":
            G, D = m["kv_heads"], m["dim"]
            w.update({q + "q": lin(H * D, W), q + "k": lin(G * D, W), q + "q.b": n(H * D, std=0.3), q + "k.b": n(G * D, std=0.3),
                      q + "q.norm": n(H * D, std=0.3 * sharp, mean=sharp), q + "k.norm": n(G * D, std=0.3, mean=1.0), q + "r1": u(H, lo=0.1, hi=0.8),
                      q + "r2": u(H, lo=0.05, hi=2.0), q + "talk": (torch.eye(H) * 0.7 + torch.randn(H, H, generator=g) * 0.4 * H ** -0.5).bfloat16(), q + "o": lin(W, H * D)})
        elif l["type"] == "channel_delta":
            G, D, U = m["kv_heads"], m["dim"], m["vdim"]
            for name, rows in (("q", G * D), ("k", G * D), ("v", H * U)):
                w[q + name], w[f"{q}{name}.conv"] = lin(rows, W), n(rows, m["conv"], std=m["conv"] ** -0.5)
            w.update({q + "b": lin(H, W), q + "A_log": u(H, lo=-1.0, hi=1.5), q + "norm": n(U, std=0.3, mean=1.0), q + "a1": lin(ranks[0], W), q + "a2": lin(H * D, ranks[0]),
                      q + "dt_bias": n(H * D, std=1.0, mean=-2.0), q + "g1": lin(ranks[1], W), q + "g2": n(H * U, ranks[1], std=1.5 * ranks[1] ** -0.5), q + "o": lin(W, H * U)})
        else:
            U, N, G = m["vdim"], m["state"], m["groups"]
            C = H * U + 2 * G * N
            w.update({q + "in": lin(2 * H * U + 2 * G * N + H, W), q + "conv": n(C, m["conv"], std=m["conv"] ** -0.5), q + "conv.b": n(C, std=0.3),
                      q + "dt_bias": n(H, std=0.8, mean=-1.0), q + "A_log": u(H, lo=-1.5, hi=1.0), q + "D": n(H), q + "norm": n(H * U, std=0.3, mean=1.0), q + "o": lin(W, H * U)})
        if l["mlp"]:
            e, f, s = l["mlp"]["router"]["experts"], l["mlp"]["expert"]["ff"], l["mlp"]["shared"]["ff"]
            w[p + "norm2"], w[p + "mlp.router"] = n(W, std=0.2, mean=1.0), lin(e, W)
            for name, ff in [(f"e{k}", f) for k in range(e)] + [("shared", s)]:
                w[f"{p}mlp.{name}.gate"], w[f"{p}mlp.{name}.up"], w[f"{p}mlp.{name}.down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    return w
