"""Nalasun's kernels on a B200: each against a plain float64 computation, then the engine (paged cache, state slots, CUDA graphs, mixed batches) in
bf16 and fp32 against the float64 restatement."""
import pytest
import torch

import nalasun_models as M
import nalasun_oracle as O
from gabisun_models import error, replay, tokens

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.bfloat16, torch.float32]
# differences of the logits in units of their spread: bf16 products against float64, and true fp32 against float64
TOL = {"bfloat16": 0.08, "float32": 1e-4}


class Meta:
    """Metadata of a batch of (new tokens, context length) requests; ``bt`` [R, pages]."""

    def __init__(self, lens, bt=None, slots=None):
        q = [a for a, _ in lens]
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
        self.query_start_loc = torch.tensor([0] + q, dtype=torch.int32).cumsum(0, dtype=torch.int32).to(DEV)
        self.query_lens_cpu, self.seq_lens_cpu, self.num_reqs = q, [s for _, s in lens], len(q)
        self.seq_lens, self.block_table = i32(self.seq_lens_cpu), bt
        self.max_query_len, self.max_seq_len = max(q), max(self.seq_lens_cpu)
        self.positions = torch.cat([torch.arange(s - n, s) for n, s in lens]).to(torch.int32).to(DEV)
        self.state_slots, self.has_initial_state = i32(slots or list(range(len(q)))), i32([int(s > n) for n, s in lens])


def portions(plan, slots, run):
    """``plan``: steps of token counts per sequence. ``run(md, who, ranges)`` gets one step's metadata and (first, last) of every sequence in it and
    returns the rows of the step; comes back with the rows of every sequence."""
    n = len(slots)
    done, got = [0] * n, [[] for _ in range(n)]
    for step in plan:
        who = [a for a in range(n) if step[a]]
        md = Meta([(step[a], done[a] + step[a]) for a in who], slots=[slots[a] for a in who])
        y, o = run(md, who, [(done[a], done[a] + step[a]) for a in who]), 0
        for a in who:
            got[a].append(y[o:o + step[a]].cpu())
            o += step[a]
            done[a] += step[a]
    return [torch.cat(x) for x in got]


PLAN = [[700, 1, 63, 64, 0], [1, 65, 1, 2, 130], [64, 1, 1, 128, 7], [3, 200, 0, 0, 1]]
SLOTS = [4, 0, 6, 2, 5]
TOTAL = [sum(s[a] for s in PLAN) for a in range(5)]


def rel(got, want):
    return ((got.double() - want).abs().max() / want.abs().max()).item()


# ------------------------------------------------------------------------------------------------ short convolutions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps,bias,silu,residual", [(192, 4, False, False, True), (256, 4, True, True, False), (77, 3, True, True, False),
                                                       (64, 2, False, True, True), (40, 1, True, False, False), (24, 7, False, True, False),
                                                       (4104, 4, False, False, True), (96, 3, False, False, True)])
def test_causal_convolution(C, taps, bias, silu, residual, dtype):
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(C + taps)
    plan = PLAN + [[2, 1, 2, 1, 3], [1, 2, 1, 3, 1], [2500, 0, 2, 0, 5]]
    total = [sum(s[a] for s in plan) for a in range(5)]
    full = [torch.randn(n, C + 16, generator=g).to(dtype) for n in total]
    w, b = torch.randn(C, taps, generator=g).to(dtype), torch.randn(C, generator=g).to(dtype) if bias else None
    state = torch.randn(7, *ops.conv_state_shape(C, taps), generator=g).to(dtype).to(DEV)   # what earlier owners of the slots left
    spare = state[1].clone()

    def run(md, who, ranges):
        x = torch.cat([full[a][i:j] for a, (i, j) in zip(who, ranges)]).to(DEV)[:, 8: 8 + C]   # a column slice
        return ops.causal_conv(x, w.to(DEV), None if b is None else b.to(DEV), state, md, silu, residual)
    got = portions(plan, SLOTS, run)
    assert torch.equal(state[1], spare)
    for a in range(5):
        x = full[a][:, 8: 8 + C].double()
        y = O.causal_conv(x, w.double(), None if b is None else b.double())
        y = O.silu(y) if silu else y
        assert rel(got[a], x + y if residual else y) < (6e-3 if dtype == torch.bfloat16 else 1e-6)


# ------------------------------------------------------------------------------------------------ matrix-state recurrences
def delta_case(g, n, Hk, H, D, V, dtype, strong):
    qkv = torch.randn(n, 2 * Hk * D + H * V + 8, generator=g).to(dtype)
    a = torch.randn(n, H * D, generator=g) * (4.0 if strong else 1.0) - (0.0 if strong else 3.0)
    return qkv, a, torch.randn(n, H, generator=g).to(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hk,H,D,V,strong", [(4, 4, 64, 32, False), (2, 6, 128, 128, False), (1, 2, 32, 64, True), (3, 3, 20, 72, True), (2, 2, 100, 40, False),
                                             (1, 1, 256, 48, False), (2, 4, 9, 21, True), (1, 3, 128, 200, True), (2, 2, 16, 33, False)])
def test_channel_delta_kernels(Hk, H, D, V, strong, dtype, monkeypatch):
    """Prompts, portions and single tokens in one batch over shuffled slots, then the same sequences go on: outputs and states equal the
    token-by-token float64 recurrence of each sequence alone. ``strong``: decays that forget within a token or two beside some near one."""
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    monkeypatch.setattr(K, "CHUNK_SEGMENT_BYTES", 8 * H * K._C.delta_chunk_bytes(D, V) if D <= 128 else 1)   # several segments a step
    g = torch.Generator().manual_seed(D + V)
    A_log, dt_bias = torch.rand(H, generator=g) * 2 - (1.0 if not strong else 0.0), torch.randn(H * D, generator=g)
    full = [delta_case(g, n, Hk, H, D, V, dtype, strong) for n in TOTAL]
    state = torch.randn(7, H, D, V, generator=g).to(DEV)
    spare = state[1].clone()

    def run(md, who, ranges):
        qkv, a, b = (torch.cat([full[x][k][i:j] for x, (i, j) in zip(who, ranges)]).to(DEV) for k in range(3))
        return ops.channel_delta(qkv[:, : 2 * Hk * D + H * V], a, b, A_log.to(DEV), dt_bias.to(DEV), state, md, Hk, H, D, V)
    got = portions(PLAN, SLOTS, run)
    assert torch.equal(state[1], spare)
    own = [h // (H // Hk) for h in range(H)]
    for x in range(5):
        qkv, a, b = full[x]
        n = qkv.shape[0]
        q, k, v = qkv[:, : 2 * Hk * D + H * V].double().split([Hk * D, Hk * D, H * V], 1)
        gate = torch.exp(-torch.exp(A_log.double()).view(1, H, 1) * O.softplus(a.double() + dt_bias.double()).view(n, H, D))
        want = O.delta_steps(O.unit(q.view(n, Hk, D))[:, own] * D ** -0.5, O.unit(k.view(n, Hk, D))[:, own], v.view(n, H, V), gate,
                             torch.sigmoid(b.double())).reshape(n, H * V)
        assert rel(got[x], want) < (6e-3 if dtype == torch.bfloat16 else 2e-5), (x, rel(got[x], want))
        err = (got[x].double() - want).abs().mean() / want.abs().mean()
        assert err < (3e-3 if dtype == torch.bfloat16 else 2e-6), (x, err)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("G,H,N,V,limit", [(2, 4, 32, 32, (0.0, float("inf"))), (1, 8, 128, 64, (0.0, float("inf"))), (3, 3, 20, 72, (0.05, 0.9)),
                                           (2, 4, 9, 21, (0.0, float("inf"))), (1, 2, 256, 40, (0.0, float("inf"))), (4, 4, 64, 100, (0.0, 0.5))])
def test_mamba2_kernels(G, H, N, V, limit, dtype):
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(N + V)
    A_log, dt_bias, skip = torch.rand(H, generator=g) * 3 - 2, torch.randn(H, generator=g) - 1, torch.randn(H, generator=g)
    full = [(torch.randn(n, H * V + 2 * G * N, generator=g).mul(0.7).to(dtype), torch.randn(n, H + 3, generator=g).to(dtype)) for n in TOTAL]
    state = torch.randn(7, H, N, V, generator=g).to(DEV)
    spare = state[1].clone()

    def run(md, who, ranges):
        xbc, dt = (torch.cat([full[x][k][i:j] for x, (i, j) in zip(who, ranges)]).to(DEV) for k in range(2))
        return ops.mamba2(xbc, dt[:, 3:], A_log.to(DEV), dt_bias.to(DEV), skip.to(DEV), state, md, H, G, N, V, limit)
    got = portions(PLAN, SLOTS, run)
    assert torch.equal(state[1], spare)
    own = [h // (H // G) for h in range(H)]
    for a in range(5):
        xbc, dt = full[a]
        n = xbc.shape[0]
        x, B, Cc = xbc.double().split([H * V, G * N, G * N], 1)
        want = O.ssm_steps(x.reshape(n, H, V), B.reshape(n, G, N)[:, own], Cc.reshape(n, G, N)[:, own],
                           O.softplus(dt[:, 3:].double() + dt_bias.double()).clamp(*limit), A_log.double(), skip.double()).reshape(n, H * V)
        assert rel(got[a], want) < (6e-3 if dtype == torch.bfloat16 else 2e-5), (a, rel(got[a], want))
        err = (got[a].double() - want).abs().mean() / want.abs().mean()
        assert err < (3e-3 if dtype == torch.bfloat16 else 2e-6), (a, err)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,n,groups,shared", [(33, 128, 4, True), (5, 4096, 2, False), (64, 300, 3, False), (7, 21, 1, True), (129, 2048, 16, True), (3, 8192, 1, False)])
@pytest.mark.parametrize("gate_first", [True, False])
def test_gated_norm(T, n, groups, shared, gate_first, dtype):
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(n)
    x, z = (torch.randn(T, n + 8, generator=g).to(dtype) for _ in range(2))
    w = torch.randn(n // groups if shared else n, generator=g).to(dtype)
    got = ops.gated_norm(x.to(DEV)[:, :n], z.to(DEV)[:, 8:], w.to(DEV), 1e-3, groups, gate_first).cpu()
    v, zz = x[:, :n].double(), z[:, 8:].double()
    v = v * O.silu(zz) if gate_first else v
    v = O.rms(v.view(T, groups, -1), 1e-3) * w.double().view(-1, n // groups)
    want = v.reshape(T, n) if gate_first else v.reshape(T, n) * torch.sigmoid(zz)
    assert rel(got, want) < (6e-3 if dtype == torch.bfloat16 else 2e-6)


# ------------------------------------------------------------------------------------------------ talking-heads attention
def pages(lens, bs, seed):
    """Block table [R, pages] of shuffled pages, their number."""
    nbs = [-(-s // bs) for _, s in lens]
    perm = torch.randperm(sum(nbs) + 4, generator=torch.Generator().manual_seed(seed)).tolist()
    bt = torch.zeros(len(lens), max(nbs), dtype=torch.int32)
    for r, n in enumerate(nbs):
        bt[r, :n] = torch.tensor([perm.pop() for _ in range(n)])
    return bt, sum(nbs) + 4


LENS = [[(200, 200), (1, 400), (3, 77), (64, 300), (1, 1)], [(1, 1500), (1, 16), (1, 17), (1, 640)], [(2, 2), (33, 65), (130, 513)], [(1, 129)] * 40,
        [(300, 1100)]]


def attend(q, k, f, bias, mix):
    """q [n, H, D] (the last rows of the sequence), k [S, G, D], f [S] -> [n, H, D], all float64."""
    n, H, _ = q.shape
    S, G, _ = k.shape
    kk = k[:, [h // (H // G) for h in range(H)]]
    s = torch.einsum("ihd,jhd->hij", q, kk) * f - O.distance_penalty(S, bias[0], bias[1])[:, S - n:]
    s = s.masked_fill(torch.arange(S).view(1, -1) > torch.arange(S - n, S).view(-1, 1), -float("inf"))
    return torch.einsum("hij,jhd->ihd", O.talk(torch.softmax(s, -1), mix), kk)


def talk_case(g, lens, H, G, dim, dtype, bs=16, sharp=1.0):
    """The step's q|k rows, the cache with everything ahead of them, and what the kernels need beside them."""
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    row = K.talk_row(H, G, dim) if dtype == torch.bfloat16 else dim
    bt, n = pages(lens, bs, len(lens) + H)
    cache, fac = torch.full((n, 1, G, bs, row), 3.0, dtype=dtype, device=DEV), torch.full((n, bs), 9.0, device=DEV)   # what earlier owners left
    seqs = [torch.randn(s, (H + G) * dim, generator=g).to(dtype) for _, s in lens]
    gain = (torch.randn(H * dim, generator=g) * 0.3 + 1.0) * sharp * 2 * dim ** -0.5
    bias = torch.stack([torch.rand(H, generator=g) * 0.8 + 0.1, torch.rand(H, generator=g) * 2 + 0.05])
    mix = (torch.eye(H) * 0.6 + torch.randn(H, H, generator=g) * 0.4).to(dtype)

    def insert(rows, md, a, b):   # positions a .. b - 1 of every request
        slot = torch.cat([bt[r].long()[torch.arange(i, j) // bs] * bs + torch.arange(i, j) % bs for r, (i, j) in enumerate(zip(a, b))])
        return ops.talk_prepare(rows.to(DEV), gain.to(DEV), 1e-4, (0.3, 50), md.positions, cache, fac, slot.to(torch.int32).to(DEV), H, G, dim)
    ahead = [s - q for q, s in lens]
    if any(ahead):
        insert(torch.cat([x[:n] for x, n in zip(seqs, ahead)]), Meta([(n, n) for n in ahead if n]), [0] * len(lens), ahead)
    md = Meta(lens, bt.to(DEV))
    q = insert(torch.cat([x[n:] for x, n in zip(seqs, ahead)]), md, ahead, [s for _, s in lens])
    return md, q, cache, fac, seqs, gain, bias, mix


SIZES = [(8, 2, 64), (16, 4, 128), (32, 8, 128), (6, 3, 40), (4, 4, 64), (12, 2, 96), (16, 1, 128), (5, 5, 20), (7, 1, 33), (1, 1, 64), (24, 8, 64), (18, 1, 32),
         (2, 1, 128), (16, 16, 128), (3, 1, 200), (33, 1, 16), (40, 8, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim", SIZES)
def test_talking_heads_kernels(H, G, dim, dtype):
    """Prompts, portions and single tokens in one batch over shuffled pages against float64 on the same cached numbers."""
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    g = torch.Generator().manual_seed(H * dim + G)
    for lens in LENS:
        md, q, cache, fac, seqs, gain, bias, mix = talk_case(g, lens, H, G, dim, dtype)
        rows = q[:, :, :dim].cpu().double()
        got = ops.talk_attention(q, cache, fac, md, bias.to(DEV), mix.to(DEV), dim).cpu().double()
        assert K.check_status() == 0
        o, seen = 0, set()
        for (n, s), x in zip(lens, seqs):
            k = x[:, H * dim:].double()
            want_q = O.rms(x[s - n:, : H * dim].double(), 1e-4) * gain.double() * O.temperature(s, 0.3, 50)[s - n:].view(-1, 1)
            assert rel(rows[o:o + n].reshape(n, -1), want_q) < (5e-3 if dtype == torch.bfloat16 else 1e-6)
            if (n, s) not in seen or o == 0:
                f = 1 / torch.sqrt((k * k).mean(-1) + 1e-4)
                want = attend(rows[o:o + n], k.view(s, G, dim), f, bias.double(), mix.double())
                assert rel(got[o:o + n], want) < (5e-3 if dtype == torch.bfloat16 else 1e-5), (n, s, rel(got[o:o + n], want))
            seen.add((n, s))
            o += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim", [(8, 2, 64), (6, 3, 40), (16, 1, 128)])
def test_one_key_stands_out_at_page_and_tile_edges(H, G, dim, dtype):
    """One head's query fits one far key, whose value is large: heads read it through the mix, in a prompt and decoded alone."""
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(dim)
    S = 700
    for at in (0, 15, 16, 31, 32, 63, 64, 127, 128, 511, 698):
        for lens in ([(40, S)], [(1, S)]):
            md, q, cache, fac, seqs, gain, bias, mix = talk_case(g, lens, H, G, dim, dtype)
            k = seqs[0][:, H * dim:].double().view(S, G, dim)
            h = H - 1
            q[:, h, :dim] = (k[at, G - 1] * 20 * dim ** -0.5).to(dtype).to(DEV)
            f = 1 / torch.sqrt((k.reshape(S, -1) ** 2).mean(-1) + 1e-4)
            qq = q[:, :, :dim].cpu().double()
            want = attend(qq, k, f, bias.double() * 0.1, mix.double())
            got = ops.talk_attention(q, cache, fac, md, bias.to(DEV) * 0.1, mix.to(DEV), dim).cpu()
            assert rel(got, want) < (5e-3 if dtype == torch.bfloat16 else 1e-5), (at, lens)
            assert (want[-1, h] - k[at, G - 1] * mix[h, h].double()).abs().max() < 3 * want[-1].abs().max()


def test_results_do_not_depend_on_splits_and_segments(monkeypatch):
    from onecat_vllm import ops
    from onecat_vllm.ops import cuda as K
    g = torch.Generator().manual_seed(3)
    md, q, cache, fac, _, _, bias, mix = talk_case(g, [(1, 900), (370, 1300), (1, 33), (2, 5)], 16, 4, 64, torch.bfloat16)
    outs = []
    for n in (1, 2, 5, 16):
        monkeypatch.setattr(K, "TALK_WS_BYTES", n * 4 * 128 * 16 * 4 * 64)
        md._talk_plan = (n, 4)
        outs.append(ops.talk_attention(q, cache, fac, md, bias.to(DEV), mix.to(DEV), 64).float())
    assert all(torch.isfinite(o).all() and (o - outs[0]).abs().max() < 0.01 * outs[0].abs().max() for o in outs)


@pytest.mark.parametrize("H,G,dim", [(4, 2, 64), (2, 1, 128)])
@pytest.mark.parametrize("order", ["rising", "falling", "alternating"])
def test_scores_that_move_the_reference(H, G, dim, order):
    """Scores that grow by many powers of two towards old keys (or new ones, or swing) make every tile rescale what earlier ones left."""
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(dim)
    S = 900
    for lens in ([(333, S)], [(1, S)]):
        md, q, cache, fac, seqs, gain, bias, mix = talk_case(g, lens, H, G, dim, torch.bfloat16)
        pos = torch.arange(S).double()
        lift = {"rising": (S - pos) / 10, "falling": pos / 10, "alternating": 40 * torch.sin(pos / 60)}[order]
        k = torch.randn(S, G, dim, generator=g).double()
        k[:, :, 0] = lift.view(-1, 1)
        k = k.bfloat16()
        bs, bt = 16, md.block_table[0].cpu().long()
        rows = torch.zeros(S, G, cache.shape[4], dtype=torch.bfloat16)
        rows[:, :, :dim] = k
        at = torch.arange(S)
        cache[bt[at // bs], 0, :, at % bs] = rows.to(DEV)
        fac[bt[at // bs], at % bs] = 1.0
        q[:, :, 0] = 1.0
        want = attend(q[:, :, :dim].cpu().double(), k.double(), torch.ones(S).double(), bias.double(), mix.double())
        got = ops.talk_attention(q, cache, fac, md, bias.to(DEV), mix.to(DEV), dim).cpu()
        assert rel(got, want) < 5e-3, (lens, rel(got, want))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,rows", [(192, 50), (100, 7), (77, 3), (2048, 300)])
def test_embedding_with_positions(H, rows, dtype):
    from onecat_vllm import ops
    g = torch.Generator().manual_seed(H)
    table, pos = torch.randn(90, H, generator=g).to(dtype), torch.randn(rows, H, generator=g).to(dtype)
    ids, p = torch.randint(0, 90, (41,), generator=g), torch.randint(0, rows, (41,), generator=g)
    x, _ = ops.embed_stream(ids.int().to(DEV), table.to(DEV), 1.0, rows=pos.to(DEV), positions=p.int().to(DEV))
    assert x.dtype == torch.float32 and (x.cpu().double() - table[ids].double() - pos[p].double()).abs().max() < 1e-6


@pytest.mark.parametrize("E,top,scale", [(12, 3, 1.5), (1, 1, 0.5), (64, 6, 2.0), (5, 5, 1.0)])
def test_sigmoid_router(E, top, scale):
    from types import SimpleNamespace
    from onecat_vllm.ops import cuda as K
    g = torch.Generator().manual_seed(E)
    h, router = torch.randn(77, 24, generator=g), torch.randn(E, 24, generator=g) * 0.3
    c = SimpleNamespace(num_experts_per_tok=top, n_group=1, topk_group=1, scoring_func="sigmoid", norm_topk_prob=False, routed_scaling_factor=scale)
    w, ids = K.route((h @ router.T).to(DEV), c, torch.zeros(E, device=DEV))
    got = torch.zeros(77, E).scatter_(1, ids.cpu().long(), w.cpu().float())
    assert (got.double() - O.route(h.double(), router.double(), top, scale)).abs().max() < 1e-5


# ------------------------------------------------------------------------------------------------ the engine
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        w = M.make_weights(cfg, len(name), M.RANKS[name], sharp=1.2)
        out[name] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, dtype, max_tokens, **kw):
    from onecat_vllm.engine.replay import TraceReplay
    return TraceReplay(path, dtype, max_tokens, device="cuda", **kw)


CASES = [(n, d) for n in M.CONFIGS for d in ("bfloat16", "float32") if not (n == "routed" and d == "bfloat16")]


@pytest.mark.parametrize("name,dtype", CASES)
def test_prompts_portions_and_decoding(models, name, dtype):
    cfg, w, path = models[name]
    toks = tokens(cfg, 330, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, dtype, 336)
    for sizes in ([330], [1] * 40 + [290], [2] * 20 + [100, 3, 130, 1, 1, 55], [250] + [1] * 80, [64, 64, 64, 64, 64, 10], [37] * 9):
        got = replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert error(got, want) < TOL[dtype], (sizes[:4], error(got, want))
    graphs = run.core.executor.worker.runner.graphs
    if dtype == "bfloat16":
        assert graphs.eligible and graphs.hits > 0   # single tokens ran as CUDA graphs
    run.close()


@pytest.mark.parametrize("name,dtype", [(n, d) for n, d in CASES if n in ("mixed", "wide", "states", "routed")])
def test_mixed_batches_reuse_pages_and_slots(models, name, dtype):
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
    """Decoding across several context buckets: every new bucket captures its graphs in the middle of live sequences, whose states must not move."""
    cfg, ranks = M.config(64, 50, [M.attn(4, 2, 16, M.moe(2, 2, 24, 16), 0.3, 90), M.delta(2, 1, 16, 24, None), M.mamba(2, 16, 24, 1, 2, M.moe(1, 1, 20, 16))], positions=1200)
    w = M.make_weights(cfg, 5, ranks, sharp=1.1)
    run = engine(M.save(cfg, w, tmp_path), dtype, 2048)
    seqs = {"a": tokens(cfg, 1100), "b": tokens(cfg, 700, 1)}
    got = replay(run, seqs, [[("a", 400)], [("b", 5)]] + [[("a", 1), ("b", 1)]] * 695 + [[("a", 1)]] * 5)
    for k, t in seqs.items():
        assert error(got[k], O.forward(cfg, w, t)[0]) < TOL[dtype], k
    run.close()


@pytest.mark.parametrize("dtype,name", [("float32", "mixed"), ("float32", "odd"), ("float32", "routed"), ("bfloat16", "wide"), ("bfloat16", "states"), ("bfloat16", "heads")])
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
