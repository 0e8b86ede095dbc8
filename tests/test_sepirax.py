"""Sepirax on the CPU path (fp32) against the plain float64 restatement in sepirax_oracle.py: each mechanism alone, whole prompts, decoding
through the paged latents and the state slots, portions, mixed batches, reuse of pages and slots, greedy generation through the scheduler."""
import copy
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import sepirax_models as M
import sepirax_oracle as O
from gabisun_models import error, replay, tokens
from onecat_vllm import LLM, SamplingParams, ops
from onecat_vllm.config import ModelConfig
from onecat_vllm.engine.replay import TraceReplay
from onecat_vllm.layers.common import DynamicTanh, RMSNorm, get_rope
from onecat_vllm.loader.weights import sepirax_name
from onecat_vllm.ops import ref

TOL = 2e-5
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


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
        w = M.make_weights(cfg, seed=len(name), sharp=1.3)
        out[name] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, max_tokens, **kw):
    return TraceReplay(path, "float32", max_tokens, device="cpu", **kw)


# ------------------------------------------------------------------------------------------------ mechanisms
def test_dynamic_tanh_and_scaled_join():
    g = torch.Generator().manual_seed(0)
    part, x = torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g)
    n = DynamicTanh(24)
    n.load_weight("weight", torch.randn(24, generator=g))
    n.load_weight("bias", torch.randn(24, generator=g))
    n.load_weight("alpha", torch.tensor(0.8))
    want = x.double() + 0.3 * part.double()
    norm = lambda v: O.dynamic_tanh(v, 0.8, n.weight.double(), n.bias.double())
    y, x1 = ops.stream_join(part, x.clone(), None, None, n, out_dtype=torch.float32, mul=0.3)
    assert torch.allclose(x1.double(), want, atol=1e-6) and torch.allclose(y.double(), norm(want), atol=1e-6)
    y, x1 = ops.stream_join(part, None, None, None, n, out_dtype=torch.float32, mul=7.0)
    assert torch.allclose(x1, 7 * part) and torch.allclose(y.double(), norm(7 * part.double()), atol=1e-5)
    assert torch.allclose(n(part)[0].double(), norm(part.double()), atol=1e-6)


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(32, 20000.0, 5.0, 1024, 16.0, 1.0), (8, 50.0, 2.0, 64, 8.0, 0.5), (6, 1000.0, 1.0, 100, 3.0, 2.0),
                                                                 (64, 500000.0, 16.0, 8192, 32.0, 1.0), (4, 10.0, 3.0, 1000000, 4.0, 1.0), (16, 1e6, 2.5, 4, 3.0, 2.0)])
def test_yarn_table(dims, base, factor, original, fast, slow):
    sc = dict(factor=factor, original=original, fast=fast, slow=slow)
    f, m = O.yarn_frequencies(dims, base, sc)
    ours = dict(rope_type="yarn", factor=factor, original_max_position_embeddings=original, beta_fast=fast, beta_slow=slow)
    cs = ref.build_cos_sin_cache(dims, 300, base, "cpu", ours)
    a = torch.arange(300).double().view(-1, 1) * f
    assert m == pytest.approx(0.1 * math.log(factor) + 1.0)
    assert torch.allclose(cs.double(), torch.cat([torch.cos(a), torch.sin(a)], 1) * m, atol=5e-5)
    x = torch.randn(300, 2, dims, generator=torch.Generator().manual_seed(dims))
    want = O.rotate(x.transpose(0, 1).double(), torch.arange(300), dict(dims=dims, base=base, scaling=sc)).transpose(0, 1)
    assert torch.allclose(ref.rope_rows(x, torch.arange(300), cs, False).double(), want, atol=2e-4)


class Meta:
    def __init__(self, bt=None, qsl=(0,), seq=(0,), slots=(0,), init=(0,)):
        t = lambda v: torch.tensor(v, dtype=torch.int32)
        self.block_table, self.query_start_loc, self.seq_lens, self.state_slots, self.has_initial_state = bt, t(qsl), t(seq), t(slots), t(init)


@pytest.mark.parametrize("lora,lora_pad,width", [(12, 12, 20), (12, 16, 32)])
def test_latents_go_into_their_pages(lora, lora_pad, width):
    """Both latent norms, the rotated key part and the padded cache row; a token without a slot leaves every other row alone."""
    g = torch.Generator().manual_seed(lora_pad)
    T, rope, bs = 9, 8, 4
    kv, q = torch.randn(T, lora + rope, generator=g), torch.randn(T, 10, generator=g)
    qn, kn = RMSNorm(10, 1e-3), RMSNorm(lora, 1e-3)
    qn.weight.data.normal_(generator=g), kn.weight.data.normal_(generator=g)
    table = get_rope(rope, 64, 100.0, "cpu").cos_sin
    slots = torch.tensor([5, 23, 4, 22, 13, 7, -1, 8, 31])
    pos = torch.tensor([3, 0, 40, 41, 7, 7, 9, 63, 1])
    cache = torch.zeros(8, bs, width)
    out = ops.mla_prepare(q, kv, qn, kn, pos, table, cache, slots, lora, lora_pad, False)
    assert torch.allclose(out.double(), O.rms(q.double(), 1e-3) * qn.weight.double(), atol=1e-5)
    rows = cache.view(-1, width)
    rot = dict(dims=rope, base=100.0)
    for t in range(T):
        if slots[t] >= 0:
            assert torch.allclose(rows[slots[t], :lora].double(), O.rms(kv[t, :lora].double(), 1e-3) * kn.weight.double(), atol=1e-5)
            assert torch.allclose(rows[slots[t], lora_pad: lora_pad + rope].double(), O.rotate(kv[t, lora:].double().view(1, -1), pos[t:t + 1], rot)[0], atol=1e-5)
    used = set(slots.tolist()) | {0}
    assert not rows[[i for i in range(32) if i not in used]].any() and not rows[:, lora_pad + rope:].any()


@pytest.mark.parametrize("E,top,count,keep", [(10, 4, 5, 3), (8, 8, 1, 1), (12, 3, 4, 1), (6, 2, 3, 2), (7, 2, 7, 3), (5, 1, 1, 1), (64, 6, 8, 8)])
def test_router(E, top, count, keep):
    z = torch.randn(40, E, generator=torch.Generator().manual_seed(E)) * 2
    w, ids = ref.grouped_topk(z, top, count, keep, None, "softmax", True)
    for t, picks in enumerate(O.choose_experts(z.double(), dict(experts=E, top=top, groups=dict(count=count, keep=keep)))):
        assert ids[t].tolist() == [e for e, _ in picks]
        assert torch.allclose(w[t].double(), torch.tensor([a for _, a in picks], dtype=torch.float64), atol=1e-6)


def test_groups_are_ranked_by_their_best_expert():
    """Two good experts of one group lose against single better ones; the best expert of a dropped group is not chosen."""
    z = torch.log(torch.tensor([[0.2, 0.19, 0.25, 0.01, 0.3, 0.05]]))
    assert ref.grouped_topk(z, 3, 3, 2, None, "softmax", True)[1][0].tolist() == [4, 2, 5]


def mlstm_oracle(x, gates, bi, bf, nw, eps, cap, H, D, V, state=None):
    q, k, v, g = x.double().split([H * D, H * D, H * V, H * V], 1)
    li, lf = ref_gates(gates.double(), bi.double(), bf.double(), cap)
    T = x.shape[0]
    o, st = O.mlstm_cell(q.view(T, H, D) * D ** -0.5, k.view(T, H, D), v.view(T, H, V), li, lf, state)
    return O.rms(o, eps).reshape(T, H * V) * nw.double() * torch.sigmoid(g), st


def ref_gates(z, bi, bf, cap):
    H = z.shape[1] // 2
    cut = lambda a: cap * torch.tanh(a / cap)
    return cut(z[:, :H] + bi), -torch.log1p(torch.exp(-cut(z[:, H:] + bf)))


@pytest.mark.parametrize("H,D,V", [(2, 8, 12), (3, 5, 7), (1, 32, 16)])
def test_mlstm_op_batches_portions_and_slots(H, D, V):
    """Sequences in one batch, with and without a state, equal each alone; slots that no request of the batch uses keep their contents."""
    g = torch.Generator().manual_seed(D)
    r = lambda *s: torch.randn(*s, generator=g)
    T, cap, eps = 21, 6.0, 1e-4
    x, gates, bi, bf, nw = r(T, 2 * H * (D + V)), r(T, 2 * H) * 3, r(H), r(H) + 3, r(H * V)
    state = (r(5, H, D, V), r(5, H, D), r(5, H))
    before = tuple(t.clone() for t in state)
    qsl, slots, init = [0, 1, 9, 9, 21], [3, 1, 4, 0], [1, 0, 1, 1]
    y = ops.mlstm(x, gates, bi, bf, nw, eps, cap, H, D, V, state, Meta(None, qsl, slots=slots, init=init))
    for a in range(4):
        lo, hi, s = qsl[a], qsl[a + 1], slots[a]
        if lo == hi:
            assert all(torch.equal(n[s], o[s]) for n, o in zip(state, before))
            continue
        want, st = mlstm_oracle(x[lo:hi], gates[lo:hi], bi, bf, nw, eps, cap, H, D, V, tuple(t[s].double() for t in before) if init[a] else None)
        assert torch.allclose(y[lo:hi].double(), want, atol=2e-4)
        assert all(torch.allclose(n[s].double(), o, atol=1e-4) for n, o in zip(state, st))
    assert torch.equal(state[0][2], before[0][2])


def test_mlstm_maximum_starts_at_zero_and_bounds_the_denominator():
    """One token with a very negative input gate: the maximum stays near f (not at i), and e^-m, not |n . q|, divides."""
    D = V = 4
    x = torch.zeros(1, 16)
    x[0, 0], x[0, 4], x[0, 8] = 2.0, 1.0, 3.0
    state = (torch.zeros(1, 1, D, V), torch.zeros(1, 1, D), torch.zeros(1, 1))
    ops.mlstm(x, torch.tensor([[-4.0, 5.0]]), torch.zeros(1), torch.zeros(1), torch.ones(4), 1e-5, 100.0, 1, D, V, state, Meta(None, [0, 1]))
    f = -math.log1p(math.exp(-100 * math.tanh(0.05)))
    assert state[2].item() == pytest.approx(f, abs=1e-6)
    assert state[0][0, 0, 0, 0].item() == pytest.approx(3 * math.exp(100 * math.tanh(-0.04) - f), rel=1e-5)


def test_one_latent_stands_out_at_page_borders_and_far_away():
    """A query that matches exactly one cached key finds it wherever it lies (first token, either side of a page border, far away), and the
    key after the query's own position is not seen."""
    L, R, bs, S = 16, 4, 16, 700
    g = torch.Generator().manual_seed(3)
    for i in (0, 15, 16, 17, 63, 64, 650, 698):
        for j in sorted({0, 1, 15, 16, i - 1, i, i + 1} & set(range(i + 2))):
            lat = torch.randn(S, L + R, generator=g) * 0.1
            lat[j] = torch.randn(L + R, generator=g) * 3
            nb = -(-S // bs)
            perm = torch.randperm(nb + 2, generator=g)[:nb]
            cache = torch.full((nb + 2, bs, L + R), 5.0)
            cache.view(-1, L + R)[torch.tensor([int(perm[a // bs]) * bs + a % bs for a in range(S)])] = lat
            q = lat[j].view(1, 1, -1) * 4
            o = ref.mla_decode(q[..., :L], q[..., L:], cache, perm.view(1, -1).to(torch.int32), torch.tensor([0, 1]), torch.tensor([i + 1]), 1.0, L)[0, 0]
            assert bool(torch.cosine_similarity(o, lat[j, :L], dim=0) > 0.99) == (j <= i), (i, j)


# ------------------------------------------------------------------------------------------------ configuration and loading
def test_config_and_names():
    cfg = M.CONFIGS["mixed"]
    mc = ModelConfig.from_hf_dict(cfg)
    assert mc.is_hybrid and mc.use_mla and mc.layer_types == ["mlstm", "full_attention", "mlstm", "full_attention"]
    a, b = mc.for_layer(1), mc.for_layer(2)
    assert (a.num_attention_heads, a.kv_lora_rank, a.qk_rope_head_dim, a.v_head_dim, a.n_group, a.topk_group, a.num_experts, a.num_experts_per_tok) == \
        (4, 40, 8, 24, 4, 1, 12, 3)
    assert (b.mlstm_heads, b.mlstm_key_dim, b.mlstm_value_dim, b.mlstm_gate_cap, b.mixer_only_layers, b.use_mla) == (3, 64, 32, 5.0, True, False)
    assert (mc.embed_scale, mc.residual_multiplier, mc.final_softcap, mc.rms_norm_eps) == (3.0, 0.6, 20.0, 1e-5)
    kind = lambda i: "mlstm" if i in (0, 2) else "mla"
    assert sepirax_name("l12.norm2.alpha", lambda i: "mla") == "model.layers.12.post_attention_layernorm.alpha"
    assert sepirax_name("l0.mix.norm", kind) == "model.layers.0.linear_attn.norm_weight" and sepirax_name("l1.mix.g", kind) == "model.layers.1.self_attn.g_proj.weight"
    assert sepirax_name("l0.mix.g", kind) == "model.layers.0.linear_attn.in_proj_g.weight" and sepirax_name("l1.mix.uk", kind) == "model.layers.1.self_attn.uk"
    assert sepirax_name("l3.mlp.e11.down", kind) == "model.layers.3.mlp.experts.11.down_proj.weight" and sepirax_name("l1.mix.norm", kind) == "l1.mix.norm"
    l0, l1 = cfg["layers"][:2]
    for bad in (dict(l0, type="conv"), dict(l0, mlp=dict(l0["mlp"], kind="dense")), dict(l1, mixer=dict(l1["mixer"], rot_dim=16)),
                dict(l1, mlp=M.moe(12, 4, 32, 4, 1)), dict(l1, mlp=M.moe(10, 4, 32, 4, 2))):
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


def test_caches_hold_latents_and_states(models):
    cfg, w, path = models["mixed"]
    run = engine(path, 64)
    shapes = [tuple(tuple(t.shape[1:]) for t in c) if isinstance(c, tuple) else tuple(c.shape[1:]) for c in run.core.executor.worker.runner.kv_caches]
    assert shapes == [((2, 24, 40), (2, 24), (2,)), (16, 48), ((3, 64, 32), (3, 64), (3,)), (16, 80)]
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
    toks = tokens(cfg, 100, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, 112)
    for sizes in ([1] * 100, [2] * 50, [3, 60, 1, 1, 2, 33], [17] * 6, [64, 36], [70] + [1] * 30):
        got = replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert error(got, want) < TOL, sizes[:4]
    run.close()


@pytest.mark.parametrize("name", ["mixed", "memories"])
def test_mixed_batches_reuse_pages_and_slots(models, name):
    """Unequal requests together, each left out of some steps, in a pool and with slots for the live ones only: logits equal those alone."""
    cfg, w, path = models[name]
    seqs = {f"r{i}": tokens(cfg, n, 10 + i) for i, n in enumerate((90, 1, 47, 64, 16, 70, 33, 80))}
    run = engine(path, 256)
    steps = [[("r0", 40), ("r1", 1), ("r2", 2)], [("r2", 1), ("r3", 63)], [("r0", 1), ("r3", 1), ("r2", 44), ("r4", 3)], [("r4", 1), ("r0", 17)],
             [("r5", 50), ("r4", 12), ("r0", 1)]] + [[("r0", 2), ("r5", 1)]] * 15 + [[("r0", 99), ("r5", 99), ("r6", 5)], [("r6", 28), ("r7", 2)]] + \
            [[("r7", 1)]] * 30 + [[("r7", 68)]]
    got = replay(run, seqs, steps)
    for k, t in seqs.items():
        assert error(got[k], O.forward(cfg, w, t)[0]) < TOL, k
    m = run.core.scheduler.kv_cache_manager
    assert m.block_pool.get_num_free_blocks() == 256 // 16 and len(m.free_state_slots) == 5
    again = replay(run, {"r0": seqs["r5"]}, [[("r0", 30)], [("r0", 40)]])["r0"]   # the same ids may come back as new requests
    assert error(again, got["r5"]) < TOL
    run.close()


@pytest.mark.parametrize("name", ["mixed", "odd", "latents", "memories"])
def test_greedy_generation_through_the_scheduler(models, name):
    cfg, w, path = models[name]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, max_num_batched_tokens=32, max_num_seqs=3)
    prompts = [tokens(cfg, n, 30 + n) for n in (50, 3, 1, 41)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=16, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 16)


def test_preemption_recomputes_states_and_latents(models):
    cfg, w, path = models["mixed"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=96, max_num_seqs=4, num_gpu_blocks_override=11)
    prompts = [tokens(cfg, 20, 60 + i) for i in range(4)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 40)


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


def test_random_weights_without_a_checkpoint():
    llm = LLM(hf_config=M.CONFIGS["mixed"], dtype="float32", device="cpu", max_model_len=64)
    o = llm.generate([{"prompt_token_ids": [1, 2, 3]}], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True, detokenize=False))
    assert len(o[0].outputs[0].token_ids) == 4


def test_prompt_embeddings_are_those_of_the_tokens(models):
    """A prompt given as its (scaled) embeddings generates what the tokens generate; the model's own rows join unscaled twice nowhere."""
    from onecat_vllm.inputs import EmbedsPrompt
    cfg, w, path = models["mixed"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=64)
    p = tokens(cfg, 9, 2)
    emb = w["embed"][torch.tensor(p)].float() * cfg["embedding"]["scale"]
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True, detokenize=False)
    assert list(llm.generate([EmbedsPrompt(prompt_embeds=emb)], sp)[0].outputs[0].token_ids) == O.greedy(cfg, w, p, 6)


# ------------------------------------------------------------------------------------------------ what the comparisons would catch
def _mutate(cfg, w, what):
    cfg, w = copy.deepcopy(cfg), {k: v.clone() for k, v in w.items()}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        if what == "cap" and l["type"] == "mlstm":
            m["gate_cap"] *= 1.2
        if l["type"] == "latent_attention":
            if what == "scale":
                m["scale"] *= 1.02
            if what in ("factor", "fast", "slow", "original") and m["rot"]["scaling"]:
                m["rot"]["scaling"][what] *= {"fast": 0.125, "slow": 8}.get(what, 2)
            if what == "base":
                m["rot"]["base"] *= 1.1
            if what == "shared key":
                w[p + "mix.dkv"][m["kv_rank"]:] *= 1.05
        if what == "forget" and l["type"] == "mlstm":
            w[p + "mix.f.b"] += 0.25
        if what == "input" and l["type"] == "mlstm":
            w[p + "mix.i.b"] += 0.25
        if what == "gate":
            w[p + "mix.g"] *= 1.05
        if what == "keep" and l["mlp"]:
            g = l["mlp"]["router"]["groups"]
            g["keep"] = min(g["keep"] + 1, g["count"])
        if what == "top" and l["mlp"]:
            l["mlp"]["router"]["top"] -= 1
        if what == "alpha":
            w[p + "norm1.alpha"] *= 1.05
    if what == "mult":
        cfg["residual_mult"] *= 1.02
    if what == "embed":
        cfg["embedding"]["scale"] *= 1.02
    if what == "softcap":
        cfg["logit_softcap"] *= 1.5
    if what == "eps":
        cfg["norm"]["eps"] *= 100
    return cfg, w


@pytest.mark.parametrize("what", ["cap", "scale", "factor", "fast", "slow", "original", "base", "shared key", "forget", "input", "gate", "keep", "top", "alpha", "mult",
                                  "embed", "softcap", "eps"])
def test_mistakes_show_in_the_logits(models, what):
    """A mistake planted in the restatement moves the logits by far more than the tolerance, so the comparisons above would find the same
    mistake in the engine."""
    cfg, w, _ = models["mixed"]
    toks = tokens(cfg, 90, 7)
    assert error(O.forward(*_mutate(cfg, w, what), toks)[0], O.forward(cfg, w, toks)[0]) > (2 if what == "eps" else 50) * TOL


def test_a_lost_state_shows(models):
    cfg, w, _ = models["memories"]
    toks = tokens(cfg, 60, 8)
    assert error(O.forward(cfg, w, toks[20:])[0], O.forward(cfg, w, toks)[0][20:]) > 1000 * TOL


@pytest.mark.timeout(300)
def test_two_tensor_parallel_ranks(tmp_path):
    """Heads of both mixers, the output gates and the experts' columns are split over the ranks; the latents are on both."""
    cfg = M.config(64, 90, [M.mlstm(4, 16, 8, M.moe(6, 2, 48, 3, 2)), M.latent(6, 16, 8, 24, 40, 32, M.moe(4, 2, 32)), M.mlstm(2, 8, 24, None)])
    w = M.make_weights(cfg, 3, sharp=1.3)
    path = M.save(cfg, w, tmp_path)
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, tensor_parallel_size=2, distributed_executor_backend="mp")
    prompts = [tokens(cfg, n, n) for n in (5, 60)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True, detokenize=False))
    llm.shutdown()
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 12)


def test_combinations_that_are_not_served_are_refused(models):
    _, _, path = models["odd"]
    for kw in (dict(pipeline_parallel_size=2), dict(tensor_parallel_size=2), dict(speculative_config=dict(method="ngram", num_speculative_tokens=2)),
               dict(speculative_config=dict(method="mtp", num_speculative_tokens=1))):
        with pytest.raises(ValueError):
            LLM(model=path, dtype="float32", device="cpu", max_model_len=64, **kw)
