"""Gabisun's kernels on a B200: each against a plain computation, then the engine (paged cache, CUDA graphs, mixed batches) in bf16 and
fp32 against the float64 restatement."""
import pytest
import torch

import gabisun_models as M
import gabisun_oracle as O

pytestmark = pytest.mark.gpu
DEV = "cuda"
# differences of the logits in units of their spread: bf16 products against float64, and true fp32 against float64
TOL = {"bfloat16": 0.09, "float32": 1e-4}


class Meta:
    """Metadata of a batch of (new tokens, context length) requests over a paged cache."""

    def __init__(self, lens, bt):
        q = [a for a, _ in lens]
        self.query_start_loc = torch.tensor([0] + q, dtype=torch.int32).cumsum(0, dtype=torch.int32).to(DEV)
        self.seq_lens = torch.tensor([s for _, s in lens], dtype=torch.int32, device=DEV)
        self.block_table, self.query_lens_cpu, self.seq_lens_cpu = bt, q, [s for _, s in lens]
        self.max_query_len, self.max_seq_len = max(q), max(self.seq_lens_cpu)


def paged_batch(keys, dtype, bs=16):
    """Keys of each request ``[S, G, D]`` inserted into shuffled pages of one cache with one tensor per page."""
    from onecat_vllm import ops
    G, D = keys[0].shape[1:]
    nbs = [-(-k.shape[0] // bs) for k in keys]
    total = sum(nbs) + 5
    perm = torch.randperm(total, generator=torch.Generator().manual_seed(total)).tolist()
    cache = torch.full((total, 1, G, bs, D), 2.0, dtype=dtype, device=DEV)
    bt = torch.zeros(len(keys), max(nbs), dtype=torch.int32)
    for r, k in enumerate(keys):
        pages = [perm.pop() for _ in range(nbs[r])]
        bt[r, : nbs[r]] = torch.tensor(pages)
        slots = torch.tensor([pages[i // bs] * bs + i % bs for i in range(k.shape[0])], dtype=torch.int32, device=DEV)
        ops.kv_insert(k.to(DEV, dtype), cache, slots)
    return cache, bt.to(DEV)


def attention_oracle(q, k, scale, mask, rel, top, sink, gate):
    """Outputs of the last ``q.shape[0]`` positions of one request, float64."""
    nq, H, D = q.shape
    S, G = k.shape[0], k.shape[1]
    kk = k.double().permute(1, 0, 2).repeat_interleave(H // G, 0)
    s = q.double().permute(1, 0, 2) @ kk.transpose(1, 2) * scale
    if rel is not None:
        s = s + O.bias_matrix(S, rel.double(), top)[:, S - nq:]
    i, j = torch.arange(S - nq, S).view(-1, 1), torch.arange(S).view(1, -1)
    seen = (j <= i) & ((i - j < mask["size"]) | (j < mask["keep_first"])) if mask else j <= i
    p = O.sink_softmax(s.masked_fill(~seen, -torch.inf), sink.double() if sink is not None else torch.full((H,), -torch.inf, dtype=torch.float64))
    o = p @ kk
    if gate is not None:
        o = o * torch.sigmoid(gate.double()).T.unsqueeze(-1)
    return o.permute(1, 0, 2)


CASES = [  # heads, kv heads, head size, window, keep, (new tokens, context) of each request
    (6, 2, 64, 150, 37, [(200, 200), (1, 400), (3, 77), (64, 300), (1, 1)]),
    (8, 2, 128, 100, 130, [(1, 1000), (1, 99), (2, 131), (8, 640)]),
    (8, 8, 128, 64, 0, [(33, 33), (1, 64), (1, 65), (130, 513)]),
    (6, 2, 64, 1, 1, [(70, 70), (1, 129), (2, 66)]),
    (16, 1, 64, 300, 64, [(150, 700), (1, 2000), (2, 500)]),
    (40, 1, 64, 70, 9, [(50, 50), (1, 333), (2, 90)]),
    (4, 1, 256, 129, 3, [(90, 400), (1, 1025), (4, 200)]),
    (2, 2, 256, 5000, 10, [(1, 3000), (65, 65)]),
]


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,G,D,size,keep,lens", CASES)
@pytest.mark.parametrize("opts", ["all", "keep", "bias", "gate", "plain"])
def test_attention_kernels(H, G, D, size, keep, lens, opts, dtype):
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops import ref
    g = torch.Generator().manual_seed(H * D + size)
    B, top = 12, 90
    every = opts == "all"
    mask = dict(size=size, keep_first=keep if every or opts == "keep" else 0)
    rel = torch.randn(B, H, generator=g) if every or opts == "bias" else None
    sink = torch.randn(H, generator=g) if every else None
    keys = [torch.randn(s, G, D, generator=g).to(dtype) for _, s in lens]
    T = sum(n for n, _ in lens)
    qkg = torch.randn(T, -(-(H * D + H) // 8) * 8, generator=g).to(dtype)
    q, gate = qkg[:, : H * D].view(T, H, D), qkg[:, H * D: H * D + H] if every or opts == "gate" else None
    cache, bt = paged_batch(keys, dtype)
    dq = qkg.to(DEV)
    table = rel[torch.tensor(ref.distance_buckets(B, top))].t().contiguous().to(DEV) if rel is not None else None
    scale = 1.5 * D ** -0.5
    got = ops.paged_attention(dq[:, : H * D].view(T, H, D), cache, Meta(lens, bt), scale, window=size, sinks=sink.to(DEV) if every else None,
                              keep=mask["keep_first"], bias_table=table, gate=dq[:, H * D: H * D + H] if gate is not None else None).cpu()
    assert K.check_status() == 0
    o = 0
    for (n, s), k in zip(lens, keys):
        want = attention_oracle(q[o:o + n], k, scale, mask, rel, top, sink, gate[o:o + n] if gate is not None else None)
        d = (got[o:o + n].double() - want).abs().max().item()
        assert d < (0.02 if dtype == torch.bfloat16 else 2e-5), ((n, s), d)
        o += n


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_one_key_stands_out_at_every_edge(dtype):
    """A query that matches exactly one key, which lies just inside or outside the window, the kept tokens, a page or a key tile: the
    output is that key exactly when the rule says it is visible. Decoded alone and as the last of a portion."""
    from onecat_vllm import ops
    size, keep, D = 100, 70, 64
    g = torch.Generator().manual_seed(5)
    for i in (99, 100, 169, 170, 171, 300, 319, 320, 500):
        for j in sorted({0, 15, 16, 63, 64, 69, 70, 71, i - size - 1, i - size, i - size + 1, i - 64, i - 1, i}):
            if not 0 <= j <= i:
                continue
            k = torch.randn(i + 1, 1, D, generator=g) * 0.1
            k[j] = torch.randn(1, D, generator=g) * 2
            cache, bt = paged_batch([k], dtype)
            for n in (1, 50):
                q = torch.zeros(n, 1, D)
                q[-1] = k[j] * 2
                o = ops.paged_attention(q.to(DEV, dtype), cache, Meta([(n, i + 1)], bt), 1.0, window=size, keep=keep)[-1, 0].float().cpu()
                seen = torch.cosine_similarity(o, k[j, 0], dim=0) > 0.99
                assert bool(seen) == O.visible(i, j, dict(size=size, keep_first=keep)), (i, j, n)


class Norm:
    def __init__(self, w, b, eps, kind):
        self.weight, self.bias, self.eps, self.plain, self.gemma = w, b, eps, kind == 2, False


@pytest.mark.parametrize("H", [4096, 256, 96, 1000, 77, 8192])
@pytest.mark.parametrize("dtype,part_dtype", [(torch.bfloat16, torch.bfloat16), (torch.bfloat16, torch.float32), (torch.float32, torch.float32)])
def test_stream_join_kernel(H, dtype, part_dtype):
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(H)
    r = lambda *s: torch.randn(*s, generator=g)
    T = 37
    part, x = (r(T, H) * 3 + 1).to(part_dtype), r(T, H)
    w1, b1, w2, b2, ls, add = (r(H).to(dtype) for _ in range(6))
    c = lambda t: t.to(DEV)
    both = torch.zeros(T, 2 * H, dtype=dtype, device=DEV)
    xd = c(x)
    y, x1 = ops.stream_join(c(part), xd, Norm(c(w1), c(b1), 1e-5, 2), c(ls), Norm(c(w2), c(b2), 1e-5, 2), out_dtype=dtype, add=c(add), copy_out=both[:, :H])
    want = x.double() + ls.double() * O.layer_norm(part.double(), w1.double(), b1.double(), 1e-5) + add.double()
    assert x1.data_ptr() == xd.data_ptr() and torch.allclose(x1.cpu().double(), want, atol=2e-5)
    assert torch.equal(both[:, :H], x1.to(dtype)) and not both[:, H:].any()
    wy = O.layer_norm(want, w2.double(), b2.double(), 1e-5)
    assert torch.allclose(y.cpu().double(), wy, atol=2e-5 if dtype == torch.float32 else 0.05, rtol=1e-2 if dtype == torch.bfloat16 else 1e-5)
    y, x1 = ops.stream_join(c(part), None, None, None, Norm(c(w2), None, 1e-3, 1), out_dtype=dtype)
    wy = part.double() / torch.sqrt(part.double().pow(2).mean(-1, keepdim=True) + 1e-3) * w2.double()
    assert torch.equal(x1.cpu(), part.float()) and torch.allclose(y.cpu().double(), wy, atol=1e-4, rtol=1e-2 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("T,N,Kd", [(1, 300, 256), (4, 64, 96), (33, 1000, 512), (200, 260, 128), (700, 384, 320), (64, 4096, 4096), (5, 7, 160)])
def test_gemm_epilogues(T, N, Kd):
    from onecat_vllm.layers.linear import ReplicatedLinear
    from onecat_vllm.ops import cuda as K
    g = torch.Generator().manual_seed(N)
    x, w = torch.randn(T, Kd, generator=g).bfloat16(), (torch.randn(N, Kd, generator=g) * Kd ** -0.5).bfloat16()
    want = x.double() @ w.double().T
    f32 = K.gemm_bf16(x.to(DEV), w.to(DEV), out_dtype=torch.float32)
    assert f32.dtype == torch.float32 and torch.allclose(f32.cpu().double(), want, atol=2e-5)
    for kw in (dict(fuse_gelu_tanh=True), dict(out_dtype=torch.float32), dict()):
        lin = ReplicatedLinear(Kd, N, quant=None, prefix="t", dtype=torch.bfloat16, **kw).to(DEV)
        lin.load_weight("weight", w.to(DEV))
        lin.process_weights_after_loading()
        y = lin(x.to(DEV)).cpu().double()
        ref = O.gelu_tanh(want) if "fuse_gelu_tanh" in kw else want
        assert torch.allclose(y, ref, atol=2e-5 if "out_dtype" in kw else 0.004, rtol=0 if "out_dtype" in kw else 0.01), kw
    assert K.check_status() == 0


# ------------------------------------------------------------------------------------------------ the engine
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        w = M.make_weights(cfg, seed=len(name), sharp=1.2)
        out[name] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, dtype, max_tokens, **kw):
    from onecat_vllm.engine.replay import TraceReplay
    return TraceReplay(path, dtype, max_tokens, device="cuda", **kw)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_prompts_portions_and_decoding(models, name, dtype):
    cfg, w, path = models[name]
    toks = M.tokens(cfg, 330, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, dtype, 336)
    for sizes in ([330], [1] * 40 + [290], [2] * 20 + [100, 3, 130, 1, 1, 55], [250] + [1] * 80, [64, 64, 64, 64, 64, 10]):
        got = M.replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert M.error(got, want) < TOL[dtype], sizes[:4]
    if dtype == "bfloat16":
        assert run.core.executor.worker.runner.graphs.hits > 0   # single tokens ran as CUDA graphs
    run.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", ["mixed", "wide_heads"])
def test_mixed_batches_reuse_pages(models, name, dtype):
    cfg, w, path = models[name]
    seqs = {f"r{i}": M.tokens(cfg, n, 10 + i) for i, n in enumerate((130, 1, 47, 64, 16, 99, 33, 130))}
    run = engine(path, dtype, 336)
    steps = [[("r0", 40), ("r1", 1), ("r2", 2)], [("r2", 1), ("r3", 63)], [("r0", 1), ("r3", 1), ("r2", 44), ("r4", 3)], [("r4", 1), ("r0", 17)],
             [("r5", 50), ("r4", 12), ("r0", 1)]] + [[("r0", 2), ("r5", 3)]] * 15 + [[("r0", 99), ("r5", 99), ("r6", 5)], [("r6", 28), ("r7", 2)]] + \
            [[("r7", 1)]] * 60 + [[("r7", 68)]]
    got = M.replay(run, seqs, steps)
    for k, t in seqs.items():
        assert M.error(got[k], O.forward(cfg, w, t)[0]) < TOL[dtype], k
    run.close()


def test_long_decoding_in_a_small_pool(tmp_path):
    cfg = M.config(64, 50, [M.layer(2, 1, 64, 40, 5, 64), M.layer(2, 2, 16, 70, 3, 32)], loop=(0, 2, 2))
    w = M.make_weights(cfg, 5, sharp=1.2)
    run = engine(M.save(cfg, w, tmp_path), "bfloat16", 1024)
    toks = M.tokens(cfg, 900)
    got = M.replay(run, {"a": toks}, [[("a", 300)]] + [[("a", 1)]] * 600)["a"]
    assert M.error(got, O.forward(cfg, w, toks)[0]) < TOL["bfloat16"]
    run.close()


@pytest.mark.parametrize("dtype,name", [("float32", "mixed"), ("float32", "loop_all"), ("bfloat16", "wide_heads")])
def test_greedy_generation_through_the_scheduler(models, name, dtype):
    """fp32: token for token. bf16: every chosen token's exact logit is within rounding of the best one along the engine's own path."""
    from onecat_vllm import LLM, SamplingParams
    cfg, w, path = models[name]
    llm = LLM(model=path, dtype=dtype, device="cuda", max_model_len=256, max_num_batched_tokens=64, max_num_seqs=4, kv_cache_memory_bytes=64 << 20)
    prompts = [M.tokens(cfg, n, 30 + n) for n in (50, 3, 1, 140, 41)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        ids = list(o.outputs[0].token_ids)
        lg = O.forward(cfg, w, p + ids)[0][len(p) - 1:-1]
        gap = lg.max(-1).values - lg[torch.arange(len(ids)), ids]
        assert gap.max() <= (0 if dtype == "float32" else 4 * TOL[dtype] * lg.std()), gap.max()
