"""Lodevik's kernels on a B200: each against a plain float64 computation, then the engine (paged cache, CUDA graphs, mixed batches) in bf16
and fp32 against the float64 restatement."""
import pytest
import torch

import lodevik_models as M
import lodevik_oracle as O
from gabisun_models import error, replay, tokens

pytestmark = pytest.mark.gpu
DEV = "cuda"
# differences of the logits in units of their spread: bf16 products against float64, and true fp32 against float64
TOL = {"bfloat16": 0.08, "float32": 1e-4}
DTYPES = [torch.bfloat16, torch.float32]


class Meta:
    """Metadata of a batch of (new tokens, context length) requests; ``bt`` [R, pages]."""

    def __init__(self, lens, bt=None):
        q = [a for a, _ in lens]
        self.query_start_loc = torch.tensor([0] + q, dtype=torch.int32).cumsum(0, dtype=torch.int32).to(DEV)
        self.query_lens_cpu, self.seq_lens_cpu, self.num_reqs = q, [s for _, s in lens], len(q)
        self.seq_lens, self.block_table = torch.tensor(self.seq_lens_cpu, dtype=torch.int32, device=DEV), bt
        self.max_query_len, self.max_seq_len = max(q), max(self.seq_lens_cpu)
        self.positions = torch.cat([torch.arange(s - n, s) for n, s in lens]).to(torch.int32).to(DEV)


def pages(lens, bs, seed):
    """Block table [R, pages] of shuffled pages, their number."""
    nbs = [-(-s // bs) for _, s in lens]
    perm = torch.randperm(sum(nbs) + 4, generator=torch.Generator().manual_seed(seed)).tolist()
    bt = torch.zeros(len(lens), max(nbs), dtype=torch.int32)
    for r, n in enumerate(nbs):
        bt[r, :n] = torch.tensor([perm.pop() for _ in range(n)])
    return bt, sum(nbs) + 4


LENS = [[(200, 200), (1, 400), (3, 77), (64, 300), (1, 1)], [(1, 1500), (1, 16), (1, 17), (1, 640)], [(2, 2), (33, 65), (130, 513)], [(1, 129)] * 40]


# ------------------------------------------------------------------------------------------------ differential attention
def width_of(dim, vdim, dtype):
    need = max(2 * dim, vdim + vdim % 2)
    return next((d for d in (64, 128, 256) if d >= need), need) if dtype == torch.bfloat16 else need


def diff_cache(ks, vs, bt, n, G, D, dtype, bs):
    """Rows k [S, G, 2, dim], v [S, G, vdim] of each request in their pages; everything else holds what earlier owners left."""
    cache = torch.full((n, 2, G, bs, D), 3.0, dtype=dtype)
    for r, (k, v) in enumerate(zip(ks, vs)):
        S, dim = k.shape[0], k.shape[3]
        row = torch.zeros(S, 2, G, D, dtype=dtype)
        row[:, 0, :, :dim], row[:, 0, :, D // 2: D // 2 + dim], row[:, 1, :, : v.shape[2]] = k[:, :, 0], k[:, :, 1], v
        pos = torch.arange(S)
        cache[bt[r].long()[pos // bs], :, :, pos % bs] = row
    return cache.to(DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 4, 24, 40), (6, 2, 64, 128), (8, 1, 64, 100), (3, 3, 100, 256), (16, 1, 40, 56), (5, 5, 9, 15), (2, 1, 140, 300),
                                          (32, 1, 32, 64), (33, 1, 16, 32), (6, 2, 128, 64)])
@pytest.mark.parametrize("cap,chunk", [(5.0, 100), (0.0, 0), (1.5, 64), (40.0, 1), (8.0, 333)])
def test_differential_attention_kernels(H, G, dim, vdim, cap, chunk, dtype):
    from onecat_vllm.ops import cuda as K
    g = torch.Generator().manual_seed(H * dim + chunk)
    D, bs, eps, lam, mx = width_of(dim, vdim, dtype), 16, 1e-4, 0.6, dict(scale=1.5 * dim ** -0.5, softcap=cap, mask=dict(size=chunk) if chunk else None, diff=0.3)
    lamt = torch.tensor([lam], device=DEV)
    for lens in LENS:
        bt, n = pages(lens, bs, len(lens))
        ks = [torch.randn(s, G, 2, dim, generator=g).to(dtype) for _, s in lens]
        vs = [torch.randn(s, G, vdim, generator=g).to(dtype) for _, s in lens]
        qs = [torch.randn(a, H, 2, dim, generator=g).mul(1.5).to(dtype) for a, _ in lens]
        cache = diff_cache(ks, vs, bt, n, G, D, dtype, bs)
        q = torch.nn.functional.pad(torch.cat(qs), (0, D // 2 - dim)).reshape(-1, 2 * H, D // 2).to(DEV)
        got = K.diff_attention(q, cache, Meta(lens, bt.to(DEV)), mx["scale"], lamt, 1 - mx["diff"], eps, vdim, cap, chunk).cpu().double()
        assert K.check_status() == 0
        o, seen = 0, set()
        for (a, s), qq, k, v in zip(lens, qs, ks, vs):
            if (a, s) not in seen or o == 0:
                seen.add((a, s))
                full = torch.zeros(s, H, 2, dim, dtype=torch.float64)
                full[s - a:] = qq.double()
                want = reference(full, k.double(), v.double(), mx, lam, eps, a)
                d = (got[o:o + a] - want).abs()
                # where the maps' difference nearly vanishes its normalised form has no digits: the mean says more than the largest one
                assert d.max() < (0.15 if dtype == torch.bfloat16 else 2e-3) and d.mean() < (4e-3 if dtype == torch.bfloat16 else 3e-6), (a, s, d.max(), d.mean())
            o += a


def reference(q, k, v, mx, lam, eps, last):
    """The restatement's differential attention for the last rows only (its loops run over heads; rows are cut to bound the time)."""
    H, G, S = q.shape[1], k.shape[1], k.shape[0]
    ok, out = O.sees(S, (mx["mask"] or {}).get("size"))[S - last:], []
    for h in range(H):
        maps = []
        for m in range(2):
            s = (q[S - last:, h, m] @ k[:, h * G // H, m].T) * mx["scale"]
            if mx["softcap"]:
                s = mx["softcap"] * torch.tanh(s / mx["softcap"])
            maps.append(O.weights(s.unsqueeze(0), ok)[0] @ v[:, h * G // H])
        out.append(O.rms(maps[0] - lam * maps[1], eps) * (1 - mx["diff"]))
    return torch.stack(out, 1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [0, 1])
def test_one_key_stands_out_at_page_tile_and_chunk_edges(m, dtype):
    """A query of one map that matches exactly one cached key of that map finds it inside its chunk, decoded alone and as the last token of a
    portion; one position outside it does not."""
    from onecat_vllm.ops import cuda as K
    dim, U, bs, chunk = 32, 64, 16, 150
    g = torch.Generator().manual_seed(3)
    lam = torch.tensor([0.0 if m == 0 else 50.0], device=DEV)   # the first map alone, or almost only the second
    for i in (0, 15, 63, 64, 149, 150, 151, 299, 300, 900, 1049):
        lo = i - i % chunk
        for j in sorted({lo - 1, lo, lo + 1, i - 64, i - 16, i - 1, i, 0} & set(range(i + 1))):
            k, v = (torch.randn(i + 1, 1, 2, dim, generator=g) * 0.1).to(dtype), torch.randn(i + 1, 1, U, generator=g).to(dtype)
            k[j, 0, m] = (torch.randn(dim, generator=g) * 2).to(dtype)
            for n in {1, min(i + 1, 40)}:
                bt, total = pages([(n, i + 1)], bs, j)
                q = torch.zeros(n, 2, dim)
                q[-1, m] = k[j, 0, m].float() * 2
                o = K.diff_attention(q.to(DEV, dtype), diff_cache([k], [v], bt, total, 1, 64, dtype, bs), Meta([(n, i + 1)], bt.to(DEV)), 1.0, lam, 1.0, 1e-6, U,
                                     0.0, chunk)[-1, 0].float().cpu()
                like = torch.cosine_similarity(o * (1 if m == 0 else -1), v[j, 0].float(), dim=0)
                assert bool(like > 0.97) == (j >= lo), (i, j, n, like)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,Hkv,D", [(4, 2, 64), (6, 1, 128), (3, 3, 256)])
@pytest.mark.parametrize("cap,chunk,window", [(0.0, 100, 0), (3.0, 77, 0), (9.0, 200, 50)])
def test_chunks_and_soft_cap_of_ordinary_attention(Hq, Hkv, D, cap, chunk, window, dtype):
    """The chunk mask is an option of ordinary attention as well; with a window the nearer edge counts."""
    from onecat_vllm.ops import cuda as K
    g, bs = torch.Generator().manual_seed(D + chunk), 16
    for lens in LENS[:3]:
        bt, n = pages(lens, bs, D)
        ks, vs = ([torch.randn(s, Hkv, D, generator=g).to(dtype) for _, s in lens] for _ in range(2))
        cache = torch.full((n, 2, Hkv, bs, D), 3.0, dtype=dtype)
        for r, (k, v) in enumerate(zip(ks, vs)):
            pos = torch.arange(k.shape[0])
            cache[bt[r].long()[pos // bs], :, :, pos % bs] = torch.stack([k, v], 1)
        q = torch.randn(sum(a for a, _ in lens), Hq, D, generator=g).to(dtype)
        got = K.paged_attention(q.to(DEV), cache.to(DEV), Meta(lens, bt.to(DEV)), 1.3 * D ** -0.5, chunk=chunk, softcap=cap, window=window).cpu().double()
        o = 0
        for (a, s), k, v in zip(lens, ks, vs):
            i = torch.arange(s)
            ok = O.sees(s, chunk) & (i.view(1, -1) > i.view(-1, 1) - window if window else torch.ones(s, s, dtype=torch.bool))
            for h in range(Hq):
                sc = (q[o:o + a, h].double() @ k[:, h * Hkv // Hq].double().T) * 1.3 * D ** -0.5
                sc = cap * torch.tanh(sc / cap) if cap else sc
                want = O.weights(sc.unsqueeze(0), ok[s - a:])[0] @ v[:, h * Hkv // Hq].double()
                assert (got[o:o + a, h] - want).abs().max() < (0.02 if dtype == torch.bfloat16 else 3e-5), (a, s, h)
            o += a


def test_both_prefill_kernels_agree():
    """The tcgen05 form (long portions) and the mma.sync form of one prompt: beyond the output's rounding they agree; scores well past the cap."""
    from onecat_vllm.ops import cuda as K
    g, bs, H, G, dim, U = torch.Generator().manual_seed(8), 32, 6, 2, 64, 128
    lens = [(300, 700), (257, 257)]
    bt, n = pages(lens, bs, 1)
    ks, vs = [torch.randn(s, G, 2, dim, generator=g).bfloat16() for _, s in lens], [torch.randn(s, G, U, generator=g).bfloat16() for _, s in lens]
    cache = diff_cache(ks, vs, bt, n, G, 128, torch.bfloat16, bs)
    q = (torch.randn(557, 2 * H, dim, generator=g) * 4).bfloat16().to(DEV)
    for cap, chunk in ((20.0, 200), (55.0, 0), (0.5, 64)):
        outs = []
        for least in (64, 10 ** 9):
            old, K.DIFF_PREFILL_MIN_LEN = K.DIFF_PREFILL_MIN_LEN, least
            try:
                outs.append(K.diff_attention(q, cache, Meta(lens, bt.to(DEV)), 1.0, torch.tensor([0.5], device=DEV), 0.6, 1e-5, U, cap, chunk).float().cpu())
            finally:
                K.DIFF_PREFILL_MIN_LEN = old
        assert K.check_status() == 0 and outs[0].isfinite().all()
        assert (outs[0] - outs[1]).abs().mean() < 1e-3 and (outs[0] - outs[1]).abs().max() < 0.1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,rot,interleaved", [(4, 4, 24, 40, 8, True), (6, 2, 64, 128, 64, True), (3, 1, 9, 15, 4, True), (2, 2, 100, 256, 30, False),
                                                          (2, 1, 140, 300, 10, True), (5, 5, 33, 64, 0, True), (4, 2, 31, 40, 6, False)])
def test_prepare_kernel(H, G, dim, vdim, rot, interleaved, dtype):
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops import ref
    g = torch.Generator().manual_seed(dim)
    T, bs, D, eps = 41, 16, width_of(dim, vdim, dtype), 1e-3
    x = torch.randn(T, 2 * (H + G) * dim + G * vdim + 2, generator=g).to(dtype)[:, :-2]
    qw, kw = torch.randn(dim, generator=g).to(dtype), torch.randn(dim, generator=g).to(dtype)
    slots = torch.randperm(64, generator=g)[:T].to(torch.int32)
    slots[5] = -1
    pos = torch.randint(0, 500, (T,), generator=g).to(torch.int32)
    table = ref.build_cos_sin_cache(rot, 512, 100.0)
    cache = torch.full((4, 2, G, bs, D), 3.0, dtype=dtype)
    dc = cache.to(DEV)
    q = ops.diff_prepare(x.to(DEV), qw.to(DEV), kw.to(DEV), eps, pos.to(DEV), table.to(DEV), dc, slots.to(DEV), H, G, dim, vdim, interleaved)
    assert K.check_status() == 0
    want, keep = cache.double(), slots >= 0
    full = torch.zeros(5, 2, G, bs, D, dtype=torch.float64)
    full[:4] = want
    wq = ref.diff_prepare(x.float(), qw.float(), kw.float(), eps, pos, table, (fc := full.float()), torch.where(keep, slots, 64), H, G, dim, vdim, interleaved)
    tol = dict(atol=0.02, rtol=0.01) if dtype == torch.bfloat16 else dict(atol=2e-5)
    assert torch.allclose(q.cpu().float(), wq, **tol) and torch.allclose(dc.cpu().float(), fc[:4], **tol)
    if interleaved:   # the fp32 form is itself compared with the restatement
        xq = x.double()[:, : 2 * H * dim].view(T, 2 * H, dim).transpose(0, 1)
        o = O.rotate(O.rms(xq, eps) * qw.double(), pos, dict(dims=rot, base=100.0)).transpose(0, 1)
        assert torch.allclose(wq[..., :dim].double(), o, atol=3e-4)   # angles are fp32


# ------------------------------------------------------------------------------------------------ latent attention: sink, gate
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,lora,rope", [(6, 64, 48), (5, 40, 6), (16, 512, 64), (7, 130, 64), (4, 600, 16)])
@pytest.mark.parametrize("lens", LENS[:3])
def test_latent_sink_and_gate(H, lora, rope, lens, dtype):
    from onecat_vllm.ops import cuda as K
    g = torch.Generator().manual_seed(H * lora)
    bs = 16
    lp, rp = K.mla_padded_sizes(lora, rope) if dtype == torch.bfloat16 else (lora, rope)
    bt, n = pages(lens, bs, H)
    lat = [torch.randn(s, lora + rope, generator=g).to(dtype) for _, s in lens]
    cache = torch.zeros(n, bs, lp + rp, dtype=dtype)
    for r, x in enumerate(lat):
        pos = torch.arange(x.shape[0])
        where = bt[r].long()[pos // bs], pos % bs
        row = torch.zeros(x.shape[0], lp + rp, dtype=dtype)
        row[:, :lora], row[:, lp: lp + rope] = x[:, :lora], x[:, lora:]
        cache[where] = row
    T = sum(a for a, _ in lens)
    q = torch.randn(T, H, lora + rope, generator=g).to(dtype)
    gate = torch.randn(T, H + 3, generator=g).to(dtype)
    sink = torch.linspace(-3.0, 8.0, H)
    q_abs = torch.nn.functional.pad(q[..., :lora], (0, lp - lora)).contiguous().to(DEV)
    scale = (lora + rope) ** -0.5
    got = K.mla_decode(q_abs, q[..., lora:].to(DEV), cache.to(DEV), Meta(lens, bt.to(DEV)), scale, lp, None, True, True, 0, sink.to(DEV),
                       gate.to(DEV)[:, 1: H + 1])[..., :lora].cpu().double()
    assert K.check_status() == 0
    o = 0
    for (a, s), x in zip(lens, lat):
        sc = torch.einsum("qhd,kd->hqk", q[o:o + a].double(), x.double()) * scale
        want = O.weights(sc, O.sees(s)[s - a:], sink.double()) @ x[:, :lora].double() * torch.sigmoid(gate[o:o + a, 1: H + 1].double()).T.unsqueeze(-1)
        assert (got[o:o + a] - want.permute(1, 0, 2)).abs().max() < (0.02 if dtype == torch.bfloat16 else 3e-5), (a, s)
        o += a


@pytest.mark.parametrize("H,nope,rope,vd,lora", [(4, 128, 64, 128, 512), (3, 32, 48, 32, 64), (5, 20, 6, 10, 36), (2, 64, 16, 100, 200)])
@pytest.mark.parametrize("lens", [[(200, 200), (1, 400), (3, 77), (64, 300), (130, 1000)], [(65, 65), (257, 513)]])
def test_expanded_prefill_sink_and_gate(H, nope, rope, vd, lora, lens):
    """The tcgen05 prefill kernel and the absorbed one share a layer: with the sink and the gate they agree with the restatement."""
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops import ref
    g, dt, bs = torch.Generator().manual_seed(nope + vd), torch.bfloat16, 16
    lp, rp = K.mla_padded_sizes(lora, rope)
    bt, n = pages(lens, bs, H)
    lat = [torch.randn(s, lora + rope, generator=g).to(dt) for _, s in lens]
    cache = torch.zeros(n, bs, lp + rp, dtype=dt)
    for r, x in enumerate(lat):
        pos = torch.arange(x.shape[0])
        row = torch.zeros(x.shape[0], lp + rp, dtype=dt)
        row[:, :lora], row[:, lp: lp + rope] = x[:, :lora], x[:, lora:]
        cache[bt[r].long()[pos // bs], pos % bs] = row
    T = sum(a for a, _ in lens)
    q, gate, sink = torch.randn(T, H, nope + rope, generator=g).to(dt), torch.randn(T, H, generator=g).to(dt), torch.linspace(-2.0, 7.0, H)
    wk, wv = (torch.randn(H, m, lora, generator=g).mul(lora ** -0.5).to(dt) for m in (nope, vd))
    pad = lambda w: torch.nn.functional.pad(w, (0, lp - lora, 0, -w.shape[1] % 64))
    wkv = torch.cat([pad(wk), pad(wv)], 1).reshape(-1, lp).to(DEV)
    md, table, scale = Meta(lens, bt.to(DEV)), ref.build_cos_sin_cache(rope, 2048, 300.0, DEV), 1.3 * (nope + rope) ** -0.5
    out = torch.full((T, H, vd), 7.0, dtype=dt, device=DEV)
    plan = K.mla_prefill_plan(md, H, nope, rope, vd, lp, torch.device(DEV))
    K.mla_prefill(plan, q.to(DEV), cache.to(DEV), md, lambda x: K.gemm_bf16(x, wkv), out, nope, rope, lp, scale, table, True, True, sink.to(DEV), gate.to(DEV))
    assert K.check_status() == 0
    got, o = out.cpu().double(), 0
    for (a, s), x in zip(lens, lat):
        if a >= 64:
            c = x[:, :lora].double()
            rot = dict(dims=rope, base=300.0)
            k, v = (torch.einsum("sl,hnl->hsn", c, w.double()).to(dt).double() for w in (wk, wv))
            qq = q[o:o + a].double().permute(1, 0, 2)
            sc = (qq[..., :nope] @ k.transpose(1, 2) + O.rotate(qq[..., nope:], torch.arange(s - a, s), rot).to(dt).double() @ x[:, lora:].double().T) * scale
            want = O.weights(sc, O.sees(s)[s - a:], sink.double()) @ v * torch.sigmoid(gate[o:o + a].double()).T.unsqueeze(-1)
            assert (got[o:o + a] - want.permute(1, 0, 2)).abs().max() < 0.02, (a, s)
        o += a


# ------------------------------------------------------------------------------------------------ embeddings, joins, feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,buckets,muls", [(192, 97, (31, 7)), (100, 2, (1, 1)), (77, 5003, (70001, 90001)), (4096, 311, (5, 9))])
def test_embedding_kernel(H, buckets, muls, dtype):
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(H)
    V, T = 70000 if H < 1000 else 500, 67
    emb = dict(scale=2.5, bigram=dict(buckets=buckets, mul_prev=muls[0], mul_cur=muls[1]))
    w = {"embed": torch.randn(V, H, generator=g).to(dtype), "bigram": torch.randn(buckets + 1, H, generator=g).to(dtype)}
    toks = torch.randint(V - 50, V, (T,), generator=g).tolist()
    ids, prev = torch.tensor(toks, dtype=torch.int32, device=DEV), torch.tensor([-1] + toks[:-1], dtype=torch.int32, device=DEV)
    x, y = ops.embed_stream(ids, w["embed"].to(DEV), 2.5, prev, w["bigram"].to(DEV), muls)
    want = O.embed(toks, {k: v.double() for k, v in w.items()}, emb)
    assert torch.allclose(x.cpu().double(), want, atol=2e-6) and y.dtype == dtype and torch.equal(y, x.to(dtype))
    z, _ = ops.embed_stream(ids, w["embed"].to(DEV)[ids.long()], 2.5, prev, w["bigram"].to(DEV), muls, gathered=True)
    assert torch.equal(x, z)


@pytest.mark.parametrize("H", [4096, 336, 100, 77])
@pytest.mark.parametrize("dtype", DTYPES)
def test_join_with_an_output_norm_only(H, dtype):
    from onecat_vllm import ops
    from onecat_vllm.layers.common import RMSNorm
    g = torch.Generator().manual_seed(H)
    part, x, scale = (torch.randn(29, H, generator=g) * 3).to(dtype), torch.randn(29, H, generator=g), torch.randn(H, generator=g).to(dtype)
    n = RMSNorm(H, 1e-3, dtype=dtype)
    n.weight.data.normal_(generator=g)
    want = x.double() + O.rms(part.double(), 1e-3) * n.weight.double() * scale.double()
    y = torch.empty(29, H, dtype=dtype, device=DEV)
    _, x1 = ops.stream_join(part.to(DEV), x.to(DEV), n.to(DEV), scale.to(DEV), None, out_dtype=dtype, copy_out=y)
    assert torch.allclose(x1.cpu().double(), want, atol=1e-5) and torch.equal(y, x1.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,ff", [(1, 192, 256), (37, 100, 44), (300, 128, 200), (3, 77, 20), (513, 512, 1024)])
def test_gated_gelu_of_any_size(T, H, ff, dtype):
    from onecat_vllm.layers.mlp import MLP
    g = torch.Generator().manual_seed(ff)
    m = MLP(H, ff, None, "m", dtype, act="gelu_tanh")
    w = {n: (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype) for n, s in (("gate", (ff, H)), ("up", (ff, H)), ("down", (H, ff)))}
    m.gate_up_proj.load_weight("weight", w["gate"], 0), m.gate_up_proj.load_weight("weight", w["up"], 1), m.down_proj.load_weight("weight", w["down"])
    m.to(DEV)
    for c in (m.gate_up_proj, m.down_proj):
        c.process_weights_after_loading()
    x = (torch.randn(T, H, generator=g) * 2).to(dtype)
    want = O.feed_forward(x.double(), {k: v.double() for k, v in w.items()}, "")
    assert torch.allclose(m(x.to(DEV)).cpu().double(), want, atol=0.04 if dtype == torch.bfloat16 else 1e-5, rtol=0.02 if dtype == torch.bfloat16 else 1e-5)


# ------------------------------------------------------------------------------------------------ the engine
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        w = M.make_weights(cfg, seed=len(name), sharp=1.1)
        out[name] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, dtype, max_tokens, **kw):
    from onecat_vllm.engine.replay import TraceReplay
    return TraceReplay(path, dtype, max_tokens, device="cuda", **kw)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_prompts_portions_and_decoding(models, name, dtype):
    cfg, w, path = models[name]
    toks = tokens(cfg, 330, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, dtype, 336)
    for sizes in ([330], [1] * 40 + [290], [2] * 20 + [100, 3, 130, 1, 1, 55], [250] + [1] * 80, [64, 64, 64, 64, 64, 10], [37] * 9):
        got = replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert error(got, want) < TOL[dtype], (sizes[:4], error(got, want))
    if dtype == "bfloat16":
        assert run.core.executor.worker.runner.graphs.hits > 0   # single tokens ran as CUDA graphs
    run.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", ["mixed", "wide", "chunks"])
def test_mixed_batches_reuse_pages(models, name, dtype):
    cfg, w, path = models[name]
    seqs = {f"r{i}": tokens(cfg, n, 10 + i) for i, n in enumerate((130, 1, 47, 64, 16, 99, 33, 130))}
    run = engine(path, dtype, 336)
    steps = [[("r0", 40), ("r1", 1), ("r2", 2)], [("r2", 1), ("r3", 63)], [("r0", 1), ("r3", 1), ("r2", 44), ("r4", 3)], [("r4", 1), ("r0", 17)],
             [("r5", 50), ("r4", 12), ("r0", 1)]] + [[("r0", 2), ("r5", 3)]] * 15 + [[("r0", 99), ("r5", 99), ("r6", 5)], [("r6", 28), ("r7", 2)]] + \
            [[("r7", 1)]] * 60 + [[("r7", 68)]]
    got = replay(run, seqs, steps)
    for k, t in seqs.items():
        assert error(got[k], O.forward(cfg, w, t)[0]) < TOL[dtype], k
    run.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_long_decoding(tmp_path, dtype):
    """Decoding across many chunks and several context buckets: every new bucket captures its graphs in the middle of live sequences."""
    cfg = M.config(64, 50, [M.attn(2, 1, 16, 32, 8, 90, 64), M.latent(2, 32, 16, 16, 64, None), M.attn(4, 2, 32, 40, 32, 700, None)])
    w = M.make_weights(cfg, 5, sharp=1.1)
    run = engine(M.save(cfg, w, tmp_path), dtype, 2048)
    seqs = {"a": tokens(cfg, 1100), "b": tokens(cfg, 700, 1)}
    got = replay(run, seqs, [[("a", 400)], [("b", 5)]] + [[("a", 1), ("b", 1)]] * 695 + [[("a", 1)]] * 5)
    for k, t in seqs.items():
        assert error(got[k], O.forward(cfg, w, t)[0]) < TOL[dtype], k
    run.close()


@pytest.mark.parametrize("dtype,name", [("float32", "mixed"), ("float32", "odd"), ("float32", "chunks"), ("bfloat16", "wide"), ("bfloat16", "latents")])
def test_greedy_generation_through_the_scheduler(models, name, dtype):
    """fp32: token for token. bf16: every chosen token's exact logit is within rounding of the best one along the engine's own path."""
    from onecat_vllm import LLM, SamplingParams
    cfg, w, path = models[name]
    llm = LLM(model=path, dtype=dtype, device="cuda", max_model_len=256, max_num_batched_tokens=96, max_num_seqs=4, kv_cache_memory_bytes=64 << 20)
    prompts = [tokens(cfg, n, 30 + n) for n in (50, 3, 1, 140, 41)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        ids = list(o.outputs[0].token_ids)
        lg = O.forward(cfg, w, p + ids)[0][len(p) - 1:-1]
        gap = lg.max(-1).values - lg[torch.arange(len(ids)), ids]
        assert gap.max() <= (0 if dtype == "float32" else 4 * TOL[dtype] * lg.std()), gap.max()
