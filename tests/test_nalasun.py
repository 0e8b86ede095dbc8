"""Nalasun on the CPU path (fp32) against the plain float64 restatement in nalasun_oracle.py: each mechanism alone, whole prompts, decoding
through pages and state slots, portions, mixed batches, reuse of pages and slots, greedy generation through the scheduler."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import nalasun_models as M
import nalasun_oracle as O
from gabisun_models import error, replay, tokens
from onecat_vllm import LLM, SamplingParams, ops
from onecat_vllm.config import EngineArgs, ModelConfig
from onecat_vllm.engine.replay import TraceReplay
from onecat_vllm.loader.weights import nalasun_name

TOL = 3e-5
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, ignore_eos=True, detokenize=False)


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)   # tiny matrices
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        w = M.make_weights(cfg, len(name), M.RANKS[name], sharp=1.5)
        out[name] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, max_tokens, **kw):
    return TraceReplay(path, "float32", max_tokens, device="cpu", **kw)


class Meta:
    def __init__(self, lens, slots, bt=None):
        t = lambda v: torch.tensor(v, dtype=torch.int32)
        self.query_start_loc = t([0] + [n for n, _ in lens]).cumsum(0)
        self.seq_lens, self.state_slots, self.has_initial_state = t([s for _, s in lens]), t(slots), t([int(s > n) for n, s in lens])
        self.positions, self.block_table = torch.cat([torch.arange(s - n, s) for n, s in lens]), bt


CUTS = [[40], [1] * 40, [2, 2, 1, 30, 5], [3, 17, 2, 18]]


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("silu,residual,bias", [(True, False, True), (False, True, False)])
def test_causal_convolution(taps, silu, residual, bias):
    g = torch.Generator().manual_seed(taps)
    x, w, b = torch.randn(40, 12, generator=g), torch.randn(12, taps, generator=g), torch.randn(12, generator=g) if bias else None
    y = O.causal_conv(x.double(), w.double(), None if b is None else b.double())
    want = (O.silu(y) if silu else y) + (x if residual else 0)
    for cut in CUTS:
        state, done, got = torch.randn(3, *ops.conv_state_shape(12, taps), generator=g), 0, []
        for n in cut:
            got.append(ops.causal_conv(x[done:done + n], w, b, state, Meta([(n, done + n)], [2]), silu, residual))
            done += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5)


@pytest.mark.parametrize("Hk,H,D,V", [(2, 4, 6, 9), (3, 3, 5, 4), (1, 1, 8, 8)])
def test_delta_rule_with_channel_decays(Hk, H, D, V):
    g = torch.Generator().manual_seed(D)
    qkv, a, b = torch.randn(40, 2 * Hk * D + H * V, generator=g), torch.randn(40, H * D, generator=g) * 2, torch.randn(40, H, generator=g)
    A_log, dt = torch.randn(H, generator=g), torch.randn(H * D, generator=g)
    q, k, v = qkv.double().split([Hk * D, Hk * D, H * V], 1)
    own = [h // (H // Hk) for h in range(H)]
    decay = torch.exp(-torch.exp(A_log.double()).view(1, H, 1) * O.softplus(a.double() + dt.double()).view(40, H, D))
    want = O.delta_steps(O.unit(q.view(40, Hk, D))[:, own] * D ** -0.5, O.unit(k.view(40, Hk, D))[:, own], v.view(40, H, V), decay, torch.sigmoid(b.double()))
    for cut in CUTS:
        state, done, got = torch.randn(3, H, D, V, generator=g), 0, []
        for n in cut:
            s = slice(done, done + n)
            got.append(ops.channel_delta(qkv[s], a[s], b[s], A_log, dt, state, Meta([(n, done + n)], [1]), Hk, H, D, V))
            done += n
        assert torch.allclose(torch.cat(got).double(), want.reshape(40, H * V), atol=1e-5)


def test_a_write_is_seen_by_its_own_token():
    """One token: the read-out is beta (q . k) v, and the next token sees the state decayed before it writes."""
    D, V = 4, 3
    qkv = torch.randn(2, 2 * D + V, generator=torch.Generator().manual_seed(0))
    state = torch.zeros(1, 1, D, V)
    o = ops.channel_delta(qkv[:1], torch.zeros(1, D), torch.zeros(1, 1), torch.zeros(1), torch.zeros(D), state, Meta([(1, 1)], [0]), 1, 1, D, V)
    q, k, v = O.unit(qkv[0, :D].double()) * D ** -0.5, O.unit(qkv[0, D:2 * D].double()), qkv[0, 2 * D:].double()
    assert torch.allclose(o[0].double(), 0.5 * (q @ k) * v, atol=1e-6) and torch.allclose(state[0, 0].double(), 0.5 * k.view(-1, 1) * v, atol=1e-6)


@pytest.mark.parametrize("G,H,N,V", [(2, 4, 6, 9), (3, 3, 5, 4), (1, 2, 8, 8)])
def test_mamba2_state_space(G, H, N, V):
    g = torch.Generator().manual_seed(N)
    xbc, dt = torch.randn(40, H * V + 2 * G * N, generator=g), torch.randn(40, H, generator=g)
    A_log, bias, D = torch.randn(H, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g)
    x, B, C = xbc.double().split([H * V, G * N, G * N], 1)
    own = [h // (H // G) for h in range(H)]
    want = O.ssm_steps(x.reshape(40, H, V), B.reshape(40, G, N)[:, own], C.reshape(40, G, N)[:, own], O.softplus(dt.double() + bias.double()), A_log.double(), D.double())
    for cut in CUTS:
        state, done, got = torch.randn(3, H, N, V, generator=g), 0, []
        for n in cut:
            s = slice(done, done + n)
            got.append(ops.mamba2(xbc[s], dt[s], A_log, bias, D, state, Meta([(n, done + n)], [1]), H, G, N, V))
            done += n
        assert torch.allclose(torch.cat(got).double(), want.reshape(40, H * V), atol=2e-5)


@pytest.mark.parametrize("groups,first", [(1, True), (3, True), (4, False), (1, False)])
def test_gated_norm(groups, first):
    g = torch.Generator().manual_seed(groups)
    x, z, w = torch.randn(7, 24, generator=g), torch.randn(7, 24, generator=g), torch.randn(24 if first else 24 // groups, generator=g)
    v = (x * O.silu(z) if first else x).double()
    v = (O.rms(v.view(7, groups, -1), 1e-2) * w.double().view(-1, 24 // groups)).reshape(7, 24)
    assert torch.allclose(ops.gated_norm(x, z, w, 1e-2, groups, first).double(), v if first else v * torch.sigmoid(z.double()), atol=1e-6)


def talk_inputs(g, S, H, G, D, bs=16):
    qk, gain = torch.randn(S, (H + G) * D, generator=g), torch.randn(H * D, generator=g) * 0.4
    bias, mix = torch.stack([torch.rand(H, generator=g), torch.rand(H, generator=g) * 2]), torch.randn(H, H, generator=g)
    nb = -(-S // bs)
    bt = torch.randperm(nb + 2, generator=g)[:nb].view(1, -1)
    cache, fac = torch.full((nb + 2, 1, G, bs, D), 5.0), torch.full((nb + 2, bs), 7.0)
    slot = bt[0][torch.arange(S) // bs] * bs + torch.arange(S) % bs
    return qk, gain, bias, mix, bt, cache, fac, slot


def talk_want(qk, gain, bias, mix, H, G, D, coef, every, eps):
    S = qk.shape[0]
    q, k = qk.double().split([H * D, G * D], 1)
    v = k.view(S, G, D)
    q = (O.rms(q, eps) * gain.double()).view(S, H, D) * O.temperature(S, coef, every).view(-1, 1, 1)
    own = [h // (H // G) for h in range(H)]
    s = torch.einsum("ihd,jhd->hij", q, O.rms(k, eps).view(S, G, D)[:, own]) - O.distance_penalty(S, bias[0].double(), bias[1].double())
    return torch.einsum("hij,jhd->ihd", O.talk(O.softmax_weights(s), mix.double()), v[:, own])


@pytest.mark.parametrize("H,G,D", [(6, 3, 8), (4, 4, 5), (5, 1, 7)])
@pytest.mark.parametrize("coef,every", [(0.3, 10), (0.9, 1), (0.0, 5)])
def test_talking_heads(H, G, D, coef, every):
    """Norms over whole rows, temperature, distance bias, mixed weights and unnormalised keys as values, through shuffled pages and in portions."""
    g = torch.Generator().manual_seed(H * D)
    S = 70
    qk, gain, bias, mix, bt, cache, fac, slot = talk_inputs(g, S, H, G, D)
    want = talk_want(qk, gain, bias, mix, H, G, D, coef, every, 1e-4)
    for cut in ([70], [1] * 70, [2, 2, 12, 1, 20, 33]):
        done, got = 0, []
        for n in cut:
            md = Meta([(n, done + n)], [0], bt)
            q = ops.talk_prepare(qk[done:done + n], gain, 1e-4, (coef, every), md.positions, cache, fac, slot[done:done + n], H, G, D)
            got.append(ops.talk_attention(q, cache, fac, md, bias, mix, D))
            done += n
        assert torch.allclose(torch.cat(got).double(), want, atol=2e-5)


def test_one_far_key_is_read_through_the_mix():
    """One head's query fits one key that is far away or at a page's border; with a mix that only passes that head's weights on, every head returns
    its own key head's row of that token."""
    g = torch.Generator().manual_seed(4)
    H, G, D, S = 4, 2, 16, 100
    for at in (0, 1, 15, 16, 31, 32, 63, 64, 97, 98):
        qk, gain, bias, mix, bt, cache, fac, slot = talk_inputs(g, S, H, G, D)
        k = qk[:, H * D:].view(S, G, D)
        qk[-1, : H * D] = torch.randn(H * D, generator=g) * 0.01
        qk[-1, D: 2 * D] = k[at, 0]   # head 1 reads key head 0
        mix = torch.zeros(H, H)
        mix[:, 1] = torch.tensor([1.0, -2.0, 0.5, 3.0])
        md = Meta([(S, S)], [0], bt)
        q = ops.talk_prepare(qk, torch.full((H * D,), 30.0), 1e-4, None, md.positions, cache, fac, slot, H, G, D)
        o = ops.talk_attention(q, cache, fac, md, bias * 0.1, mix, D)[-1]
        want = torch.stack([mix[h, 1] * k[at, h // 2] for h in range(H)])
        assert torch.allclose(o, want, atol=1e-3), at


def test_position_rows():
    g = torch.Generator().manual_seed(1)
    table, rows, ids, pos = torch.randn(20, 6, generator=g), torch.randn(9, 6, generator=g), torch.tensor([3, 19, 3]), torch.tensor([0, 8, 4])
    x, _ = ops.embed_stream(ids, table, 1.0, rows=rows, positions=pos)
    assert torch.equal(x, table[ids] + rows[pos])
    x, _ = ops.embed_stream(ids, table[:3], 1.0, rows=rows, positions=pos, gathered=True)
    assert torch.equal(x, table[:3] + rows[pos])


@pytest.mark.parametrize("experts,top,scale", [(5, 2, 1.5), (3, 3, 1.0), (8, 1, 0.4)])
def test_router_weights_are_not_renormalised(experts, top, scale):
    from onecat_vllm.ops import ref
    g = torch.Generator().manual_seed(experts)
    h, router = torch.randn(9, 12, generator=g), torch.randn(experts, 12, generator=g)
    w, ids = ref.grouped_topk(h @ router.T, top, 1, 1, torch.zeros(experts), "sigmoid", False, scale)
    got = torch.zeros(9, experts).scatter_(1, ids.long(), w)
    assert torch.allclose(got.double(), O.route(h.double(), router.double(), top, scale), atol=1e-6)


# ------------------------------------------------------------------------------------------------ configuration and loading
def test_config_and_names(models):
    mc = ModelConfig.from_pretrained(models["mixed"][2])
    a, b, c, d = (mc.for_layer(i) for i in range(4))
    assert (a.num_attention_heads, a.num_key_value_heads, a.head_dim, a.attn_temperature, a.num_experts, a.num_experts_per_tok, a.moe_intermediate_size,
            a.shared_expert_intermediate_size, a.routed_scaling_factor, a.mixer_only_layers) == (6, 3, 40, (0.25, 37), 3, 3, 48, 56, 1.3, False)
    assert (b.linear_num_key_heads, b.linear_num_value_heads, b.linear_key_head_dim, b.linear_value_head_dim, b.linear_conv_kernel_dim, b.linear_decay_rank,
            b.linear_gate_rank, b.mixer_only_layers) == (2, 4, 24, 40, 3, 10, 14, True)
    assert (c.mamba_n_heads, c.mamba_d_head, c.mamba_d_state, c.mamba_n_groups, c.mamba_norm_groups, c.mamba_d_conv, c.routed_scaling_factor) == (6, 16, 24, 2, 3, 4, 0.7)
    assert d.mixer_only_layers and mc.layer_types == ["full_attention", "channel_delta", "mamba2", "full_attention"]
    assert (mc.position_rows, mc.input_conv, mc.rms_norm_eps, mc.is_hybrid, mc.norm_topk_prob, mc.scoring_func) == (400, 3, 1e-5, True, False, "sigmoid")
    assert ModelConfig.from_hf_dict(M.CONFIGS["heads"]).is_hybrid   # input convolutions need state slots
    kind = lambda i: mc.layer_types[i]
    assert nalasun_name("l0.mix.q.b", kind) == "model.layers.0.self_attn.q_proj.bias" and nalasun_name("l1.mix.v.conv", kind) == "model.layers.1.linear_attn.conv_v"
    assert nalasun_name("l2.mix.conv.b", kind) == "model.layers.2.linear_attn.conv_bias" and nalasun_name("l3.canon1", kind) == "model.layers.3.input_conv.weight"
    assert nalasun_name("l0.mlp.e11.up", kind) == "model.layers.0.mlp.experts.11.up_proj.weight" and nalasun_name("pos", kind) == "model.positions.weight"
    assert nalasun_name("l0.mlp.shared.down", kind) == "model.layers.0.mlp.shared_expert.down_proj.weight" and nalasun_name("l0.mix.conv", kind) == "l0.mix.conv"
    cfg = M.CONFIGS["mixed"]
    l0, l1, l2 = cfg["layers"][:3]
    for bad in (dict(l0, type="conv"), dict(l0, mlp=dict(kind="dense", ff=8)), dict(l0, mixer=dict(l0["mixer"], vdim=8)), dict(l0, mixer=dict(l0["mixer"], kv_heads=4)),
                dict(l1, mixer=dict(l1["mixer"], kv_heads=3)), dict(l2, mixer=dict(l2["mixer"], groups=4)), dict(l2, mixer=dict(l2["mixer"], norm_groups=7)),
                dict(l0, mlp=M.moe(2, 3, 8, 8))):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[bad]))


def test_every_tensor_of_a_checkpoint_is_used(models):
    from onecat_vllm.loader.weights import iter_safetensors, load_weights
    from onecat_vllm.models import build_model
    for name, (cfg, w, path) in models.items():
        mc = ModelConfig.from_pretrained(path, dtype=torch.float32)
        with torch.device("cpu"):
            m = build_model(mc)
        assert len(load_weights(m, iter_safetensors(path))) == len(w), name
        params = sum(p.numel() for n, p in m.named_parameters() if not n.endswith("e_score_correction_bias"))
        assert params == sum(v.numel() for v in w.values()) + (m.model.embed_tokens.padded - cfg["vocab"]) * cfg["width"], name


def test_caches_and_states(models):
    """Every layer has a slot for its input convolution; attention caches one row per token and key head and one number per token."""
    run = engine(models["mixed"][2], 64)
    caches = run.core.executor.worker.runner.kv_caches
    shapes = [tuple(tuple(t.shape[1:]) for t in c) for c in caches]
    conv = ((2, 128),)
    assert shapes == [conv, ((1, 3, 16, 40), (16,)), conv, ((2, 256), (4, 24, 40)), conv, ((3, 192), (6, 24, 16)), conv, ((1, 1, 16, 64), (16,))]
    run.close()


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_whole_prompt(models, name):
    cfg, w, path = models[name]
    toks = tokens(cfg, 150)
    run = engine(path, 160)
    got = replay(run, {"a": toks}, [[("a", 150)]])["a"]
    assert error(got, O.forward(cfg, w, toks)[0]) < TOL
    run.close()


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_portions_and_decoding(models, name):
    cfg, w, path = models[name]
    toks = tokens(cfg, 90, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, 96)
    for sizes in ([1] * 90, [2] * 45, [1, 2, 63, 24], [64, 26], [70] + [1] * 20, [17, 3, 2, 40, 1, 1, 26]):
        got = replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert error(got, want) < TOL, sizes[:4]
    run.close()


@pytest.mark.parametrize("name", ["mixed", "wide", "routed"])
def test_mixed_batches_reuse_pages_and_slots(models, name):
    cfg, w, path = models[name]
    seqs = {f"r{i}": tokens(cfg, n, 10 + i) for i, n in enumerate((70, 1, 33, 64, 16, 50, 20))}
    run = engine(path, 240)
    steps = [[("r0", 20), ("r1", 1), ("r2", 2)], [("r2", 1), ("r3", 63)], [("r0", 1), ("r3", 1), ("r2", 30), ("r4", 3)], [("r4", 1), ("r0", 17)],
             [("r5", 30), ("r4", 12), ("r0", 1)]] + [[("r0", 2), ("r5", 3)]] * 4 + [[("r0", 99), ("r5", 99), ("r6", 5)], [("r6", 2)], [("r6", 13)]]
    got = replay(run, seqs, steps)
    for k, t in seqs.items():
        assert error(got[k], O.forward(cfg, w, t)[0]) < TOL, k
    kv = run.core.scheduler.kv_cache_manager
    assert len(kv.free_state_slots) == 5 and not kv.req_to_state_slot
    run.close()


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_greedy_generation_through_the_scheduler(models, name):
    cfg, w, path = models[name]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, max_num_batched_tokens=32, max_num_seqs=3)
    prompts = [tokens(cfg, n, 30 + n) for n in (50, 3, 1, 41)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=12, **GREEDY))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 12)


@pytest.mark.parametrize("overlap", [True, False])
def test_preemption_and_overlapped_steps(models, overlap):
    """Few pages: requests are thrown out and recomputed from their first token, states included."""
    cfg, w, path = models["mixed"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=96, max_num_seqs=4, num_gpu_blocks_override=11, async_scheduling=overlap)
    prompts = [tokens(cfg, 20, 60 + i) for i in range(4)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=30, **GREEDY))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 30)


def test_trace_runner_program(models, tmp_path):
    cfg, w, path = models["odd"]
    toks = tokens(cfg, 30, 3)
    lines = [dict(step=0, entries=[dict(id="a", tokens=toks[:20], want=[3, 19]), dict(id="b", tokens=toks[:5], want=[])], end=["b"]),
             dict(step=1, entries=[dict(id="a", tokens=toks[20:29], want=[])], end=[]),
             dict(step=2, entries=[dict(id="b", tokens=toks[:1], want=[0]), dict(id="a", tokens=toks[29:], want=[0])], end=["a", "b"])]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens",
                        "128", "--device", "cpu"], input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    want = O.forward(cfg, w, toks)[0]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / n).read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    assert error(read("0.f32"), want[[3, 19]]) < TOL
    assert error(read("2.f32"), torch.stack([want[0], want[29]])) < TOL


def test_sequences_end_with_the_position_rows(models):
    """A pool for more tokens than a sequence may have; the last position's row is the table's last."""
    cfg, w, path = models["routed"]
    toks = tokens(cfg, 400, 2)
    run = engine(path, 900)
    got = replay(run, {"a": toks, "b": toks[:399]}, [[("a", 380), ("b", 399)], [("a", 20)]])
    want = O.forward(cfg, w, toks)[0]
    assert error(got["a"], want) < TOL and error(got["b"], want[:399]) < TOL
    run.close()
    assert EngineArgs(model=path, device="cpu", max_model_len=900).create_engine_config().model_config.max_model_len == 400


def test_random_weights_without_a_checkpoint():
    llm = LLM(hf_config=M.CONFIGS["mixed"], dtype="float32", device="cpu", max_model_len=64)
    o = llm.generate([{"prompt_token_ids": [1, 2, 3]}], SamplingParams(max_tokens=4, **GREEDY))
    assert len(o[0].outputs[0].token_ids) == 4


def test_prompt_given_as_vectors(models):
    """Vectors take the place of the token embeddings; the positions' rows join them."""
    from onecat_vllm.inputs import EmbedsPrompt
    cfg, w, path = models["states"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=64)
    p = tokens(cfg, 9, 2)
    got = llm.generate([EmbedsPrompt(prompt_embeds=w["embed"].float()[torch.tensor(p)])], SamplingParams(max_tokens=6, **GREEDY))[0].outputs[0].token_ids
    assert list(got) == O.greedy(cfg, w, p, 6)


# ------------------------------------------------------------------------------------------------ what the comparisons would catch
def _mutate(cfg, w, what):
    cfg, w = copy.deepcopy(cfg), {k: v.float() for k, v in w.items()}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        if what == "input convolution late":
            w[f"l{i}.canon1"] = w[f"l{i}.canon1"].roll(1, 1)
        if what == "router scale" and l["mlp"]:
            l["mlp"]["router"]["scale"] *= 1.05
        if what == "shared expert" and l["mlp"]:
            w[f"l{i}.mlp.shared.down"] *= 0.9
        if l["type"] == "attention":
            if what == "scale":
                m["scale"] *= 1.02
            if what == "temperature":
                m["q_temp"]["coef"] *= 1.1
            if what == "temperature step":
                m["q_temp"]["every"] += 1
            if what in ("r1", "r2"):
                w[p + what] *= 1.05
            if what == "mix transposed":
                w[p + "talk"] = w[p + "talk"].T.contiguous()
            if what == "no mix":
                w[p + "talk"] = torch.eye(m["heads"])
            if what == "key bias":
                w[p + "k.b"] *= 0.9
            if what == "key norm":
                w[p + "k.norm"] *= 1.05
        if l["type"] == "channel_delta":
            if what == "decay":
                w[p + "A_log"] += 0.1
            if what == "decay per head":
                w[p + "a2"] = w[p + "a2"].view(m["heads"], m["dim"], -1).mean(1, keepdim=True).expand(-1, m["dim"], -1).reshape(w[p + "a2"].shape)
            if what == "step size":
                w[p + "b"] *= 1.1
            if what == "output gate":
                w[p + "g2"] *= 1.1
            if what == "delta convolution late":
                w[p + "k.conv"] = w[p + "k.conv"].roll(1, 1)
        if l["type"] == "mamba2":
            if what == "skip":
                w[p + "D"] *= 1.05
            if what == "time step":
                w[p + "dt_bias"] += 0.05
            if what == "convolution bias":
                w[p + "conv.b"] *= 0.9
            if what == "norm groups":
                m["norm_groups"] = 1
            if what == "state decay":
                w[p + "A_log"] += 0.1
    if what == "positions":
        w["pos"] = w["pos"].roll(1, 0)
    if what == "eps":
        cfg["norm"]["eps"] *= 100
    return cfg, w


@pytest.mark.parametrize("what", ["input convolution late", "router scale", "shared expert", "scale", "temperature", "temperature step", "r1", "r2", "mix transposed", "no mix",
                                  "key bias", "key norm", "decay", "decay per head", "step size", "output gate", "delta convolution late", "skip", "time step",
                                  "convolution bias", "norm groups", "state decay", "positions", "eps"])
def test_mistakes_show_in_the_logits(models, what):
    """A mistake planted in the restatement moves the logits by far more than the tolerance, so the comparisons above would find the same
    mistake in the engine."""
    cfg, w, _ = models["mixed"]
    toks = tokens(cfg, 110, 7)
    assert error(O.forward(*_mutate(cfg, w, what), toks)[0], O.forward(cfg, w, toks)[0]) > (2 if what == "eps" else 50) * TOL


def test_combinations_that_are_not_served_are_refused(models):
    path = models["mixed"][2]
    for kw in (dict(pipeline_parallel_size=2), dict(tensor_parallel_size=2), dict(kv_cache_dtype="fp8"), dict(speculative_config=dict(method="mtp", num_speculative_tokens=1))):
        with pytest.raises((ValueError, RuntimeError)):
            LLM(model=path, dtype="float32", device="cpu", max_model_len=64, **kw)
    llm = LLM(model=models["states"][2], dtype="float32", device="cpu", max_model_len=64,
              speculative_config=dict(method="ngram", num_speculative_tokens=2, prompt_lookup_max=2, prompt_lookup_min=1))
    with pytest.raises(Exception):
        llm.generate([{"prompt_token_ids": [3, 4, 3, 4, 3, 4]}], SamplingParams(max_tokens=8, **GREEDY))
