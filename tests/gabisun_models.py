"""Small random Gabisun checkpoints for the tests (not a test file)."""
import json
import os

import torch
from safetensors.torch import save_file


def layer(heads, kv, dim, size, keep, ff, scale=None, bias_max=40, buckets=8):
    return dict(type="attention", _buckets=buckets, mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale or 1.3 * dim ** -0.5, bias_max=bias_max,
                mask=dict(size=size, keep_first=keep)), mlp=dict(kind="dense", ff=ff) if ff else None)


def config(width, vocab, layers, loop=None, eps=1e-5):
    return dict(architecture="Gabisun", width=width, vocab=vocab, norm=dict(eps=eps), layers=layers, loop=dict(zip(("start", "stop", "times"), loop)) if loop else None)


# unlike layers, loops at either end or none, layers without a feed-forward, widths and head sizes that are no multiples of the kernels'
# tiles, windows from one token to longer than every sequence, no kept tokens, kept tokens that reach into the window
CONFIGS = {
    "mixed": config(128, 210, [layer(4, 2, 32, 24, 3, 160), layer(6, 3, 16, 70, 0, None, buckets=6), layer(8, 1, 64, 17, 9, 200, bias_max=96, buckets=12),
                               layer(2, 2, 48, 300, 1, 72)], loop=(1, 3, 3)),
    "plain": config(96, 133, [layer(3, 3, 80, 33, 5, 130, bias_max=128, buckets=32), layer(3, 1, 80, 64, 64, 130, bias_max=64, buckets=16)], eps=3e-4),
    "loop_all": config(160, 96, [layer(8, 2, 128, 1, 2, 96, bias_max=10, buckets=4), layer(5, 5, 24, 50, 70, 256, bias_max=200)], loop=(0, 2, 2)),
    "wide_heads": config(192, 301, [layer(4, 1, 256, 100, 20, 192), layer(16, 1, 64, 129, 0, 320, bias_max=33, buckets=10),
                                    layer(2, 1, 96, 40, 4, 64)], loop=(1, 2, 1)),
}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random bf16 weights. Layer scales, norms, gates, sinks and biases are far from their neutral values; ``sharp`` scales queries and
    keys, so that single keys stand out and a lost or an extra one shows in the logits."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean).bfloat16()
    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": n(V, W), "final.norm": n(W, std=0.2, mean=1.0), "final.norm.b": n(W, std=0.2)}
    if cfg.get("loop"):
        w["loop.in"] = n(W, 2 * W, std=(2 * W) ** -0.5)
        w["loop.step"] = n(cfg["loop"]["times"], W, std=0.5)
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if l["mlp"] else ()):
            w[p + name] = n(W, std=0.2, mean=1.0)
            w[p + name + ".b"] = n(W, std=0.2)
        w[p + "mix.q"] = n(H * D, W, std=sharp * W ** -0.5)
        w[p + "mix.k"] = n(G * D, W, std=sharp * W ** -0.5)
        w[p + "mix.g"] = n(H, W, std=W ** -0.5)
        w[p + "mix.o"] = n(W, H * D, std=(H * D) ** -0.5)
        w[p + "mix.rel"] = n(l["_buckets"], H)
        w[p + "mix.sink"] = n(H, std=1.5)
        w[p + "ls1"] = n(W, std=0.3, mean=0.7)
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            w[p + "mlp.up"] = n(ff, W, std=W ** -0.5)
            w[p + "mlp.down"] = n(W, ff, std=ff ** -0.5)
            w[p + "ls2"] = n(W, std=0.3, mean=0.7)
    return w


def save(cfg, w, path):
    os.makedirs(path, exist_ok=True)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return str(path)


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def replay(run, seqs, portions, want_all=True, end=True):
    """Feed the sequences (name -> tokens) in steps given as lists of (name, count); returns name -> logits of every token [n, vocab]."""
    done, out = {k: 0 for k in seqs}, {k: [] for k in seqs}
    for step in portions:
        entries, ends = [], []
        for name, n in step:
            a = done[name]
            n = min(n, len(seqs[name]) - a)
            if n <= 0:
                continue
            entries.append(dict(id=name, tokens=seqs[name][a:a + n], want=list(range(n)) if want_all else []))
            done[name] = a + n
            if end and done[name] == len(seqs[name]):
                ends.append(name)
        lg = run.step(entries, ends)
        o = 0
        for e in entries:
            out[e["id"]].append(lg[o:o + len(e["want"])])
            o += len(e["want"])
    assert all(done[k] == len(seqs[k]) for k in seqs)
    return {k: torch.cat(v) for k, v in out.items()}


def error(got, want):
    """Largest root-mean-square difference of a position's logits (mean taken off), in units of the logits' spread."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.double().std()).max().item()
