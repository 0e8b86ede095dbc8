"""Sepirax's kernels on a B200: each against a plain float64 computation, then the engine (paged latents, state slots, CUDA graphs, mixed
batches) in bf16 and fp32 against the float64 restatement."""
import copy
import math

import pytest
import torch

import sepirax_models as M
import sepirax_oracle as O
from gabisun_models import error, replay, tokens

pytestmark = pytest.mark.gpu
DEV = "cuda"
# differences of the logits in units of their spread: bf16 products against float64, and true fp32 against float64
TOL = {"bfloat16": 0.04, "float32": 1e-4}


def tol(name, dtype):
    """"odd" rounds coarsely: its small products cancel, and the same model in bf16 on the CPU path is as far off."""
    return 0.25 if (name, dtype) == ("odd", "bfloat16") else TOL[dtype]


DTYPES = [torch.bfloat16, torch.float32]


class Meta:
    """Metadata of a batch of (new tokens, context length) requests; ``bt`` [R, pages]."""

    def __init__(self, lens, bt=None, slots=None, init=None):
        t = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        q = [a for a, _ in lens]
        self.query_start_loc = torch.tensor([0] + q, dtype=torch.int32).cumsum(0, dtype=torch.int32).to(DEV)
        self.query_lens_cpu, self.seq_lens_cpu, self.num_reqs = q, [s for _, s in lens], len(q)
        self.seq_lens, self.block_table = t(self.seq_lens_cpu), bt
        self.max_query_len, self.max_seq_len = max(q), max(self.seq_lens_cpu)
        if slots is not None:
            self.state_slots, self.has_initial_state = t(slots), t(init)


# ------------------------------------------------------------------------------------------------ latent attention
def latent_cache(lat, pad, width, dtype, bs=16):
    """Latent rows ``[S, lora + rope]`` of each request in shuffled pages; the key part sits at ``pad``, the padding is zero."""
    lora = pad[0]
    nbs = [-(-x.shape[0] // bs) for x in lat]
    total = sum(nbs) + 4
    perm = torch.randperm(total, generator=torch.Generator().manual_seed(total)).tolist()
    cache = torch.zeros(total, bs, width, dtype=dtype)
    cache[..., : lora] = 3.0
    bt = torch.zeros(len(lat), max(nbs), dtype=torch.int32)
    for r, x in enumerate(lat):
        pages = [perm.pop() for _ in range(nbs[r])]
        bt[r, : nbs[r]] = torch.tensor(pages)
        rows = torch.tensor([pages[i // bs] * bs + i % bs for i in range(x.shape[0])])
        flat = cache.view(-1, width)
        flat[rows, :lora] = x[:, :lora]
        flat[rows, pad[1]: pad[1] + x.shape[1] - lora] = x[:, lora:]
    return cache.to(DEV), bt.to(DEV)


LENS = [[(200, 200), (1, 400), (3, 77), (64, 300), (1, 1)], [(1, 1500), (1, 16), (1, 17), (1, 640)], [(2, 2), (33, 65), (130, 513)]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,lora,rope,fine", [(6, 64, 48, True), (5, 40, 6, True), (16, 512, 64, True), (16, 512, 64, False), (3, 200, 24, True), (7, 130, 64, False),
                                              (32, 320, 96, True), (1, 12, 2, True), (4, 600, 16, True)])
@pytest.mark.parametrize("lens", LENS)
def test_latent_attention_kernels(H, lora, rope, fine, lens, dtype):
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops import ref
    g = torch.Generator().manual_seed(H * lora)
    lat = [torch.randn(s, lora + rope, generator=g).to(dtype) for _, s in lens]
    T = sum(n for n, _ in lens)
    lp, rp = K.mla_padded_sizes(lora, rope) if dtype == torch.bfloat16 else (lora, rope)
    cache, bt = latent_cache(lat, (lora, lp), lp + rp, dtype)
    q = torch.randn(T, H, lora + rope + 3, generator=g).to(dtype)      # rows wider than what is used: strides
    q_abs = torch.nn.functional.pad(q[..., :lora], (0, lp - lora)).contiguous().to(DEV)
    rot = dict(dims=rope, base=300.0)
    table = ref.build_cos_sin_cache(rope, 2048, 300.0, DEV)
    scale = 1.2 * (lora + rope) ** -0.5
    got = K.mla_decode(q_abs, q.to(DEV)[..., lora: lora + rope], cache, Meta(lens, bt), scale, lp, table, False, fine)[..., :lora].cpu().double()
    assert K.check_status() == 0
    o = 0
    for (n, s), x in zip(lens, lat):
        pos = torch.arange(s - n, s)
        qq = q[o:o + n].double().permute(1, 0, 2)
        qr = O.rotate(qq[..., lora: lora + rope], pos, rot)
        if dtype == torch.bfloat16:
            qr = qr.bfloat16().double()
        sc = (torch.cat([qq[..., :lora], qr], -1) @ x.double().T) * scale
        sc = sc.masked_fill(torch.arange(s).view(1, 1, -1) > pos.view(1, -1, 1), -math.inf)
        want = (torch.softmax(sc, -1) @ x[:, :lora].double()).permute(1, 0, 2)
        assert (got[o:o + n] - want).abs().max() < (0.03 if dtype == torch.bfloat16 else 3e-5), (n, s)
        o += n


@pytest.mark.parametrize("fine", [True, False])
@pytest.mark.parametrize("H,nope,rope,vd,lora", [(4, 128, 64, 128, 512), (3, 32, 48, 32, 64), (5, 20, 6, 10, 36), (2, 64, 16, 100, 200), (2, 48, 70, 64, 130), (1, 100, 2, 128, 64)])
@pytest.mark.parametrize("lens", [[(200, 200), (1, 400), (3, 77), (64, 300), (130, 1000)], [(128, 128)], [(65, 65), (257, 513)], [(64, 64), (63, 63), (600, 601)]])
def test_expanded_prefill_kernel(H, nope, rope, vd, lora, lens, fine):
    """Portions of at least 64 tokens in the expanded form; the other requests' rows stay as they are."""
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops import ref
    g = torch.Generator().manual_seed(nope + vd)
    dt = torch.bfloat16
    lat = [torch.randn(s, lora + rope, generator=g).to(dt) for _, s in lens]
    T = sum(n for n, _ in lens)
    lp, rp = K.mla_padded_sizes(lora, rope)
    cache, bt = latent_cache(lat, (lora, lp), lp + rp, dt)
    q = torch.randn(T, H, nope + rope, generator=g).to(dt)
    wk, wv = (torch.randn(H, n, lora, generator=g).mul(lora ** -0.5).to(dt) for n in (nope, vd))
    pad = lambda w: torch.nn.functional.pad(w, (0, lp - lora, 0, -w.shape[1] % 64))
    wkv = torch.cat([pad(wk), pad(wv)], 1).reshape(-1, lp).to(DEV)
    md = Meta(lens, bt)
    md.positions = torch.cat([torch.arange(s - n, s) for n, s in lens]).to(torch.int32).to(DEV)
    table = ref.build_cos_sin_cache(rope, 2048, 300.0, DEV)
    scale = 1.3 * (nope + rope) ** -0.5
    out = torch.full((T, H, vd), 7.0, dtype=dt, device=DEV)
    plan = K.mla_prefill_plan(md, H, nope, rope, vd, lp, torch.device(DEV))
    assert plan[1] == sum(n >= 64 for n, _ in lens) and plan[-1] == any(n < 64 for n, _ in lens)
    K.mla_prefill(plan, q.to(DEV), cache, md, lambda x: K.gemm_bf16(x, wkv), out, nope, rope, lp, scale, table, False, fine)
    assert K.check_status() == 0
    got, o = out.cpu().double(), 0
    for (n, s), x in zip(lens, lat):
        if n < 64:
            assert (got[o:o + n] == 7.0).all()
        else:
            pos = torch.arange(s - n, s)
            c = x[:, :lora].double()
            k, v = (torch.einsum("sl,hnl->hsn", c, w.double()).to(dt).double() for w in (wk, wv))
            qq = q[o:o + n].double().permute(1, 0, 2)
            qr = O.rotate(qq[..., nope:], pos, dict(dims=rope, base=300.0)).to(dt).double()
            sc = (qq[..., :nope] @ k.transpose(1, 2) + qr @ x[:, lora:].double().T) * scale
            sc = sc.masked_fill(torch.arange(s).view(1, 1, -1) > pos.view(1, -1, 1), -math.inf)
            want = (torch.softmax(sc, -1) @ v).permute(1, 0, 2)
            assert (got[o:o + n] - want).abs().max() < (0.02 if fine else 0.03), (n, s)
        o += n


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_latent_stands_out_everywhere(dtype):
    """A query that matches exactly one cached key, at page and tile borders, at the start and far away: found when it is visible, decoded
    alone and as the last token of a portion."""
    from onecat_vllm.ops import cuda as K
    L, R = 64, 16
    g = torch.Generator().manual_seed(3)
    for i in (0, 15, 16, 63, 64, 65, 127, 128, 1000):
        for j in sorted({0, 1, 15, 16, 63, 64, i - 65, i - 64, i - 1, i} & set(range(i + 1))):
            x = torch.randn(i + 1, L + R, generator=g) * 0.1
            x[j] = torch.randn(L + R, generator=g) * 2
            x = x.to(dtype)
            cache, bt = latent_cache([x], (L, L), L + R, dtype)
            for n in (1, min(i + 1, 40)):
                q = torch.zeros(n, 1, L + R)
                q[-1] = x[j].float() * 2
                q = q.to(DEV, dtype)
                o = K.mla_decode(q[..., :L].contiguous(), q[..., L:], cache, Meta([(n, i + 1)], bt), 1.0, L, None, False, True)[-1, 0].float().cpu()
                assert torch.cosine_similarity(o, x[j, :L].float(), dim=0) > 0.99, (i, j, n)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,lora,rope,interleaved", [(80, 64, 48, False), (30, 36, 6, False), (0, 512, 64, True), (1536, 512, 64, True)])
def test_latent_prepare_kernel(nq, lora, rope, interleaved, dtype):
    from onecat_vllm import ops
    from onecat_vllm.layers.common import RMSNorm
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops import ref
    g = torch.Generator().manual_seed(lora)
    T = 37
    x = torch.randn(T, nq + lora + rope + 5, generator=g).to(dtype)
    qn, kn = RMSNorm(max(nq, 1), 1e-3, dtype=dtype), RMSNorm(lora, 1e-3, dtype=dtype)
    qn.weight.data.normal_(generator=g), kn.weight.data.normal_(generator=g)
    lp, rp = K.mla_padded_sizes(lora, rope) if dtype == torch.bfloat16 else (lora, rope)
    slots = torch.randperm(64, generator=g)[:T].to(torch.int32)
    slots[5] = -1
    pos = torch.randint(0, 500, (T,), generator=g).to(torch.int32)
    table = ref.build_cos_sin_cache(rope, 512, 100.0)
    cache = torch.zeros(4, 16, lp + rp, dtype=dtype)
    args = lambda d: (x.to(d)[:, :nq] if nq else None, x.to(d)[:, nq: nq + lora + rope], qn.to(d) if nq else None, kn.to(d), pos.to(d), table.to(d))
    ref_cache = cache.double().clone()
    dc = cache.to(DEV)
    out = ops.mla_prepare(*args(DEV), dc, slots.to(DEV), lora, lp, interleaved)
    kv = x[:, nq: nq + lora + rope].double()
    tol = dict(atol=0.03, rtol=0.01) if dtype == torch.bfloat16 else dict(atol=3e-5)
    if nq:
        assert torch.allclose(out.cpu().double(), O.rms(x[:, :nq].double(), 1e-3) * qn.weight.cpu().double(), **tol)
    rows = ref_cache.view(-1, lp + rp)
    for t in range(T):
        if slots[t] >= 0:
            rows[slots[t], :lora] = O.rms(kv[t, :lora], 1e-3) * kn.weight.cpu().double()
            rows[slots[t], lp: lp + rope] = ref.rope_rows(kv[t:t + 1, lora:].view(1, 1, -1), pos[t:t + 1], table.double(), interleaved).view(-1) \
                if interleaved else O.rotate(kv[t:t + 1, lora:], pos[t:t + 1], dict(dims=rope, base=100.0))[0]
    assert torch.allclose(dc.cpu().double(), ref_cache, **tol)


# ------------------------------------------------------------------------------------------------ mLSTM
def mlstm_inputs(g, T, H, D, V, dtype):
    r = lambda *s: torch.randn(*s, generator=g)
    return r(T, 2 * H * (D + V)).to(dtype), r(T, 2 * H) * 2, r(H), torch.linspace(0.0, 9.0, H), r(H * V).to(dtype)


def mlstm_want(x, gates, bi, bf, nw, eps, cap, H, D, V, state):
    q, k, v, z = x.double().split([H * D, H * D, H * V, H * V], 1)
    cut = lambda a: cap * torch.tanh(a / cap)
    li = cut(gates[:, :H].double() + bi.double())
    lf = -torch.log1p(torch.exp(-cut(gates[:, H:].double() + bf.double())))
    T = x.shape[0]
    o, st = O.mlstm_cell(q.view(T, H, D) * D ** -0.5, k.view(T, H, D), v.view(T, H, V), li, lf, state)
    return O.rms(o, eps).reshape(T, H * V) * nw.double() * torch.sigmoid(z), st


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V", [(4, 56, 64), (3, 20, 72), (2, 128, 128), (1, 256, 512), (2, 9, 21), (1, 130, 200), (1, 512, 64), (2, 64, 300)])
def test_mlstm_kernels(H, D, V, dtype, monkeypatch):
    """Prompts, portions and single tokens in one batch over shuffled slots, then the same sequences go on: outputs and states equal the
    token-by-token float64 recurrence of each sequence alone."""
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    monkeypatch.setattr(K, "CHUNK_SEGMENT_BYTES", 8 * 8 * H * D * V)   # several segments a step
    g = torch.Generator().manual_seed(D + V)
    eps, cap = 1e-5, 9.0
    # how many tokens each of five sequences brings, step by step
    plan = [[700, 1, 63, 64, 0], [1, 65, 1, 2, 130], [64, 1, 1, 128, 7], [3, 200, 0, 0, 1]]
    total = [sum(s[a] for s in plan) for a in range(5)]
    full = [mlstm_inputs(g, n, H, D, V, dtype) for n in total]
    _, _, bi, bf, nw = full[0]
    slots = [4, 0, 6, 2, 5]
    fill = lambda *s: torch.randn(*s, generator=g).to(DEV)     # what earlier owners of the slots left
    state = (fill(7, H, D, V), fill(7, H, D), fill(7, H))
    spare = [t[1].clone() for t in state]
    done, got = [0] * 5, [[] for _ in range(5)]
    for step in plan:
        who = [a for a in range(5) if step[a]]
        part = lambda k: torch.cat([full[a][k][done[a]: done[a] + step[a]] for a in who]).to(DEV)
        md = Meta([(step[a], done[a] + step[a]) for a in who], slots=[slots[a] for a in who], init=[int(done[a] > 0) for a in who])
        y = ops.mlstm(part(0), part(1), bi.to(DEV), bf.to(DEV), nw.to(DEV), eps, cap, H, D, V, state, md).cpu()
        o = 0
        for a in who:
            got[a].append(y[o:o + step[a]])
            o += step[a]
            done[a] += step[a]
    assert K.check_status() == 0 and all(torch.equal(t[1], s) for t, s in zip(state, spare))
    for a in range(5):
        want, st = mlstm_want(full[a][0], full[a][1], bi, bf, nw, eps, cap, H, D, V, None)
        d = (torch.cat(got[a]).double() - want).abs()
        # where |n . q| is small beside its terms the quotient has no digits: such rows are normalised noise in any precision
        assert d.max() < (0.05 if dtype == torch.bfloat16 else 2e-3) and d.mean() < (4e-3 if dtype == torch.bfloat16 else 1e-5), (a, d.max(), d.mean())
        for t, s in zip(state, st):
            t = t[slots[a]].cpu().double()
            assert ((t - s).abs().max() / s.abs().max()) < 2e-4, (a, s.shape)


def test_mlstm_chunks_and_recurrence_agree():
    """The chunked kernels on a bf16 prompt against the recurrent kernel on the same numbers: beyond the output's rounding they agree."""
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    H, D, V, T = 3, 64, 96, 517
    g = torch.Generator().manual_seed(9)
    x, gates, bi, bf, nw = mlstm_inputs(g, T, H, D, V, torch.bfloat16)
    outs, states = [], []
    for least in (64, 10 ** 9):
        old, K.CHUNK_MIN_LEN = K.CHUNK_MIN_LEN, least
        try:
            state = tuple(torch.zeros(2, *s, device=DEV) for s in ((H, D, V), (H, D), (H,)))
            md = Meta([(T, T)], slots=[1], init=[0])
            outs.append(ops.mlstm(x.to(DEV), gates.to(DEV), bi.to(DEV), bf.to(DEV), nw.to(DEV), 1e-5, 9.0, H, D, V, state, md).float().cpu())
            states.append([t[1].cpu() for t in state])
        finally:
            K.CHUNK_MIN_LEN = old
    assert (outs[0] - outs[1]).abs().mean() < 1e-3
    assert all((a - b).abs().max() <= 1e-4 * b.abs().max() for a, b in zip(*states))


# ------------------------------------------------------------------------------------------------ small kernels
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,n,off", [(5, 64, 0), (33, 100, 3), (700, 2048, 64), (1, 7, 1)])
def test_sigmoid_mul_kernel(T, n, off, dtype):
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(n)
    x, z = torch.randn(T, n, generator=g).to(dtype), torch.randn(T, n + off + 2, generator=g).to(dtype)
    got = ops.sigmoid_mul(x.to(DEV), z.to(DEV)[:, off: off + n]).cpu().double()
    assert torch.allclose(got, x.double() * torch.sigmoid(z[:, off: off + n].double()), atol=1e-6, rtol=5e-3 if dtype == torch.bfloat16 else 1e-6)


@pytest.mark.parametrize("H", [4096, 336, 100, 77])
@pytest.mark.parametrize("dtype", DTYPES)
def test_dynamic_tanh_join_kernel(H, dtype):
    from onecat_vllm import ops
    from onecat_vllm.layers.common import DynamicTanh
    g = torch.Generator().manual_seed(H)
    T = 29
    part, x = (torch.randn(T, H, generator=g) * 3).to(dtype), torch.randn(T, H, generator=g)
    n = DynamicTanh(H, dtype)
    n.weight.data.normal_(generator=g), n.bias.data.normal_(generator=g), n.alpha.data.fill_(0.7)
    w, b, al = n.weight.double(), n.bias.double(), n.alpha.double()
    y, x1 = ops.stream_join(part.to(DEV), x.to(DEV), None, None, n.to(DEV), out_dtype=dtype, mul=0.35)
    want = x.double() + 0.35 * part.double()
    assert torch.allclose(x1.cpu().double(), want, atol=2e-6)
    assert torch.allclose(y.cpu().double(), O.dynamic_tanh(want, al, w, b), atol=1e-5 if dtype == torch.float32 else 0.03, rtol=1e-2 if dtype == torch.bfloat16 else 0)


@pytest.mark.parametrize("E,top,count,keep", [(10, 4, 5, 3), (12, 3, 4, 1), (6, 2, 3, 2), (7, 2, 7, 3), (5, 5, 1, 1), (64, 6, 8, 3), (256, 8, 8, 4), (40, 6, 8, 3), (500, 16, 50, 7)])
def test_router_kernel(E, top, count, keep):
    from types import SimpleNamespace
    from onecat_vllm.ops import cuda as K
    z = torch.randn(67, E, generator=torch.Generator().manual_seed(E)) * 2
    c = SimpleNamespace(num_experts_per_tok=top, n_group=count, topk_group=keep, scoring_func="softmax", norm_topk_prob=True, routed_scaling_factor=1.0)
    w, ids = K.route(z.to(DEV), c, None)
    for t, picks in enumerate(O.choose_experts(z.double(), dict(experts=E, top=top, groups=dict(count=count, keep=keep)))):
        assert ids[t].tolist() == [e for e, _ in picks]
        assert torch.allclose(w[t].cpu().double(), torch.tensor([a for _, a in picks], dtype=torch.float64), atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,top,H,I", [(1, 10, 4, 336, 48), (37, 5, 2, 100, 20), (300, 12, 3, 128, 96), (70, 4, 4, 77, 33), (513, 16, 4, 512, 256)])
def test_experts_of_any_size(T, E, top, H, I, dtype):
    from onecat_vllm.config import ModelConfig
    from onecat_vllm.layers.moe import FusedMoE
    g = torch.Generator().manual_seed(H + I)
    m = FusedMoE(ModelConfig(hidden_size=H, num_experts=E, num_experts_per_tok=top, moe_intermediate_size=I, dtype=dtype), "t")
    w = {}
    for e in range(E):
        for name, s in (("gate", (I, H)), ("up", (I, H)), ("down", (H, I))):
            w[f"e{e}.{name}"] = (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype)
            m.load_expert_weight(e, name + "_proj", "weight", w[f"e{e}.{name}"])
    m.to(DEV)
    m.process_weights_after_loading()
    x = torch.randn(T, H, generator=g).to(dtype)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)])
    a = torch.rand(T, top, generator=g)
    got = m(x.to(DEV), a.to(DEV), ids.to(torch.int32).to(DEV)).cpu().double()
    want = torch.zeros(T, H, dtype=torch.float64)
    for e in range(E):
        share = (a.double() * (ids == e)).sum(-1, keepdim=True)
        gate, up, down = (w[f"e{e}.{n}"].double() for n in ("gate", "up", "down"))
        want += share * ((O.silu(x.double() @ gate.T) * (x.double() @ up.T)) @ down.T)
    assert torch.allclose(got, want, atol=0.03 if dtype == torch.bfloat16 else 1e-5)


# ------------------------------------------------------------------------------------------------ the engine
def every_expert(cfg):
    """The same model with every expert chosen for every token: no close call of the router between bf16 and float64."""
    cfg = copy.deepcopy(cfg)
    for l in cfg["layers"]:
        if l["mlp"]:
            r = l["mlp"]["router"]
            r["top"], r["groups"]["keep"] = min(r["experts"], 16), r["groups"]["count"]
            if r["experts"] > 16:
                r["experts"], r["groups"] = 16, dict(count=1, keep=1)
    return cfg


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for dtype in ("float32", "bfloat16"):
        for name, cfg in M.CONFIGS.items():
            cfg = every_expert(cfg) if dtype == "bfloat16" else cfg
            w = M.make_weights(cfg, seed=len(name), sharp=1.1)
            out[name, dtype] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, dtype, max_tokens, **kw):
    from onecat_vllm.engine.replay import TraceReplay
    return TraceReplay(path, dtype, max_tokens, device="cuda", **kw)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_prompts_portions_and_decoding(models, name, dtype):
    cfg, w, path = models[name, dtype]
    toks = tokens(cfg, 330, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, dtype, 336)
    for sizes in ([330], [1] * 40 + [290], [2] * 20 + [100, 3, 130, 1, 1, 55], [250] + [1] * 80, [64, 64, 64, 64, 64, 10]):
        got = replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert error(got, want) < tol(name, dtype), sizes[:4]
    if dtype == "bfloat16":
        assert run.core.executor.worker.runner.graphs.hits > 0   # single tokens ran as CUDA graphs
    run.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", ["mixed", "wide", "memories"])
def test_mixed_batches_reuse_pages_and_slots(models, name, dtype):
    cfg, w, path = models[name, dtype]
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
    """Decoding across several context buckets: every new bucket captures its graphs in the middle of live sequences."""
    cfg = M.config(64, 50, [M.mlstm(2, 16, 24, None), M.latent(16, 32, 16, 16, 64, 32, None, base=10000.0), M.mlstm(1, 32, 32, M.moe(4, 4, 32))])
    w = M.make_weights(cfg, 5, sharp=1.1)
    run = engine(M.save(cfg, w, tmp_path), dtype, 2048)
    seqs = {"a": tokens(cfg, 1100), "b": tokens(cfg, 700, 1)}
    got = replay(run, seqs, [[("a", 400)], [("b", 5)]] + [[("a", 1), ("b", 1)]] * 695 + [[("a", 1)]] * 5)
    for k, t in seqs.items():
        assert error(got[k], O.forward(cfg, w, t)[0]) < TOL[dtype], k
    run.close()


@pytest.mark.parametrize("dtype,name", [("float32", "mixed"), ("float32", "odd"), ("float32", "memories"), ("bfloat16", "wide"), ("bfloat16", "latents")])
def test_greedy_generation_through_the_scheduler(models, name, dtype):
    """fp32: token for token. bf16: every chosen token's exact logit is within rounding of the best one along the engine's own path."""
    from onecat_vllm import LLM, SamplingParams
    cfg, w, path = models[name, dtype]
    llm = LLM(model=path, dtype=dtype, device="cuda", max_model_len=256, max_num_batched_tokens=96, max_num_seqs=4, kv_cache_memory_bytes=64 << 20)
    prompts = [tokens(cfg, n, 30 + n) for n in (50, 3, 1, 140, 41)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        ids = list(o.outputs[0].token_ids)
        lg = O.forward(cfg, w, p + ids)[0][len(p) - 1:-1]
        gap = lg.max(-1).values - lg[torch.arange(len(ids)), ids]
        assert gap.max() <= (0 if dtype == "float32" else 4 * TOL[dtype] * lg.std()), gap.max()
