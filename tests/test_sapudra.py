"""The Sapudra decoder through the framework (loader, cache, runner, engine, shard runtime, trace replay) against the plain float64
statement in `sapudra_oracle.py`, on the CPU operators and, marked gpu, on the CUDA kernels in both number formats."""

import json
import os
import subprocess
import sys

import pytest
import torch

import sapudra_oracle as oracle
from lorax_b200.config import EngineConfig, ModelConfig
from lorax_b200.models.decoder import DecoderModel
from lorax_b200.models.mixers import RandomWeights, tensor_shapes
from lorax_b200.runtime.trace import TraceReplay
from lorax_b200.utils.weights import InMemoryWeights

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PLACES = [pytest.param("cpu", torch.float32, id="cpu"),
          pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="cuda-fp32"),
          pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="cuda-bf16")]


def dense(ff=44):
    return dict(kind="dense", ff=ff)


def moe(experts=10, top=3, ff=36, groups=(5, 3), scale=2.5, shared=52):
    m = dict(kind="moe", router=dict(experts=experts, top=top, scale=scale), expert=dict(ff=ff))
    if groups:
        m["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def layer(heads=6, kv_heads=2, dim=20, vdim=28, size=40, scale=0.3, mlp=None):
    return dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size)))


def config(layers, width=76, vocab=150, mult=0.4, eps=1e-5, cap=9.0, positions=900):
    c = dict(architecture="Sapudra", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, max_positions=positions, layers=layers)
    if cap:
        c["logit_softcap"] = cap
    return c


CONFIGS = {
    # sizes off every grid, keys and values of different widths, layers without a feed-forward, windows of one token and of a page
    "odd": config([layer(mlp=moe()), layer(heads=1, kv_heads=1, dim=7, vdim=90, size=1), layer(size=32, mlp=dense()),
                   layer(heads=5, kv_heads=5, dim=70, vdim=9, size=33, scale=0.1, mlp=moe(experts=7, top=1, groups=None, shared=0))]),
    # everything that can be 1, no cap, one group, a shared expert wider than several experts, a window past the sequence
    "plain": config([layer(heads=2, kv_heads=1, dim=16, vdim=16, size=1000, mlp=moe(experts=4, top=4, groups=(1, 1), scale=1.0, ff=20, shared=300)),
                     layer(heads=3, kv_heads=1, dim=24, vdim=24, size=64, mlp=moe(experts=6, top=2, groups=(6, 2), shared=40))],
                    width=100, mult=1.0, eps=3e-4, cap=None),
    # sizes of the tensor-core prompt kernel, many experts
    "aligned": config([layer(heads=4, kv_heads=2, dim=128, vdim=128, size=70, scale=0.09, mlp=moe(experts=40, top=6, ff=128, groups=(8, 3), shared=128)),
                       layer(heads=16, kv_heads=1, dim=128, vdim=120, size=31, scale=0.09, mlp=dense(256)),
                       layer(heads=34, kv_heads=2, dim=64, vdim=128, size=128, scale=0.12, mlp=moe(experts=16, top=2, groups=(4, 2)))],
                      width=256, vocab=320),
}


def weights_of(cfg, seed=0, sharp=2.0):
    """Random weights, rounded to bf16.  The norms' query weights are scaled so that single keys stand out, corrections so that many
    choice scores are negative."""
    rw = RandomWeights(ModelConfig.from_dict(cfg), "cpu", seed)
    out = {}
    for n in rw.shapes:
        t = rw.get_tensor(n)
        if n.endswith("mix.q.norm"):
            t = t * sharp
        if n.endswith("correction"):
            t = t * 3 - 0.7
        out[n] = t.to(torch.bfloat16)
    return out


def build(cfg, w, device, dtype):
    return DecoderModel.from_weights(ModelConfig.from_dict(cfg), InMemoryWeights(w), device, dtype)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def check(got, want, dtype, what=""):
    want = want.float()
    err = (got - want).pow(2).mean(-1).sqrt() / want.std()
    if dtype == torch.float32:
        assert err.max() < 3e-5, (what, float(err.max()))
    else:
        # rounding decides between experts whose choice scores are nearly equal: such tokens, and the few that look at them, may differ
        assert err.quantile(0.8) < 0.05, (what, float(err.quantile(0.8)))


def run_trace(replay, seqs, steps):
    """steps: list of [(name, tokens taken)]; every place is asked for.  -> name -> logits [tokens, vocab]"""
    at, out = {}, {}
    for step in steps:
        entries = []
        for name, n in step:
            a = at.get(name, 0)
            entries.append(dict(id=name, tokens=seqs[name][a: a + n], want=list(range(n))))
            at[name] = a + n
        logits, o = replay.step(entries), 0
        for name, n in step:
            out.setdefault(name, []).append(logits[o: o + n])
            o += n
            if at[name] == len(seqs[name]):
                replay.end(name)
    return {k: torch.cat(v) for k, v in out.items()}


# ---------------------------------------------------------------------------------------------- configuration, loading
def test_configuration_and_tensor_names():
    c = ModelConfig.from_dict(CONFIGS["odd"])
    assert c.model_type == "sapudra" and c.layer_style == "post" and c.residual_multiplier == 0.4 and c.final_logit_softcapping == 9.0
    assert c.max_position_embeddings == 900 and c.learned_positions and c.num_key_value_heads == 5
    m = c.layer_specs[0].moe
    assert (m.experts, m.top, m.ff, m.groups, m.keep, m.shared_ff, m.scale) == (10, 3, 36, 5, 3, 52, 2.5)
    assert c.layer_specs[1].moe is None and c.layer_specs[1].ff == 0 and c.layer_specs[3].moe.groups == 0
    shapes = tensor_shapes(c)
    assert shapes["l0.mix.q"] == (120, 76) and shapes["l0.mix.v"] == (56, 76) and shapes["l0.mix.o"] == (76, 168) and shapes["pos"] == (900, 76)
    assert shapes["l0.mlp.e9.down"] == (76, 36) and shapes["l0.mlp.shared.sg"] == (1, 76) and shapes["l0.norm2.b"] == (76,)
    assert "l1.norm2" not in shapes and "l1.mlp.up" not in shapes and "l3.mlp.shared.up" not in shapes and shapes["l2.mlp.up"] == (44, 76)
    assert ModelConfig.from_dict(CONFIGS["plain"]).final_logit_softcapping is None
    for bad in (moe(groups=(3, 1)), moe(top=11), moe(groups=(5, 1)), moe(groups=(5, 6))):
        with pytest.raises(ValueError):
            ModelConfig.from_dict(config([layer(mlp=bad)]))
    with pytest.raises(NotImplementedError):
        ModelConfig.from_dict(config([layer(mlp=dict(kind="other"))]))
    for bad in (dict(heads=5), dict(size=0)):
        with pytest.raises(ValueError):
            DecoderModel.random_init(ModelConfig.from_dict(config([layer(**bad)])), "cpu", torch.float32)
    with pytest.raises(NotImplementedError):
        DecoderModel.random_init(ModelConfig.from_dict(config([layer(dim=257)])), "cpu", torch.float32)


def test_what_the_design_does_not_offer_is_refused():
    from lorax_b200.server.runtime import ShardRuntime
    m = DecoderModel.random_init(ModelConfig.from_dict(CONFIGS["odd"]), "cpu", torch.float32)
    with pytest.raises(ValueError):
        m.quantize("fp8")
    with pytest.raises(ValueError, match="fp8"):
        ShardRuntime(m, None, EngineConfig(max_total_tokens=100, kv_cache_dtype="fp8"), num_blocks=16, max_batch=2)
    with pytest.raises(ValueError, match="positions"):             # more tokens than there are position vectors
        ShardRuntime(m, None, EngineConfig(max_total_tokens=901), num_blocks=64, max_batch=2)
    from lorax_b200.runtime.engine import Engine
    with pytest.raises(ValueError, match="positions"):
        Engine(m, EngineConfig(max_total_tokens=901), num_blocks=64, max_batch=2)


# ---------------------------------------------------------------------------------------------- mechanisms alone
def step_of(n, before=0):
    from test_mixers_gpu import make_step
    return make_step([], [(before, n)])


@pytest.mark.parametrize("H,G,d,dv,size", [(4, 2, 16, 8, 5), (3, 3, 8, 24, 1), (4, 1, 8, 8, 100), (2, 1, 8, 8, 64)])
def test_windowed_attention_and_head_norms(H, G, d, dv, size):
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(size)
    T = 70
    x = torch.randn(T, (H + G) * d + G * dv, generator=g)
    wq, wk = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) + 0.5
    f = x.double()
    q = oracle.rms_norm(f[:, : H * d].view(T, H, d), wq.double(), 1e-3)
    k = oracle.rms_norm(f[:, H * d: (H + G) * d].view(T, G, d), wk.double(), 1e-3)
    want = oracle.attend(q, k, f[:, (H + G) * d:].view(T, G, dv), 0.37, size)
    inp, nb, _ = step_of(T)
    cache, out = torch.zeros(nb, G, 32 * (d + dv)), torch.empty(T, H * dv)
    ref.qk_norm_kvwrite(x, H, G, d, dv, d, wq, wk, 1e-3, cache, inp.slots)
    ref.gqa_attn(x, cache, H, G, d, dv, 0.37, size, inp, out)
    assert torch.allclose(out.double().view(T, H, dv), want, atol=1e-5)


@pytest.mark.parametrize("E,top,groups", [(12, 3, (4, 2)), (12, 4, (12, 5)), (9, 2, None), (8, 8, (1, 1)), (6, 1, (2, 1))])
def test_routing(E, top, groups):
    """Negative choice scores, groups whose best expert is outranked by two good ones, weights without the correction."""
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(E)
    T = 50
    x, wr = torch.randn(T, 24, generator=g), torch.randn(E + 1, 24, generator=g) * 0.5
    corr = torch.randn(E, generator=g) - 1.2
    router = dict(top=top, scale=1.9)
    if groups:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    ids, w = oracle.route(x.double() @ wr[:E].double().t(), corr.double(), router)
    r = ref.moe_route(x, wr, top, 0, E, experts=E, score="sigmoid", correction=corr, groups=groups[0] if groups else 0,
                      keep=groups[1] if groups else 0, scale=1.9, shared=2)
    full = lambda i, v: torch.zeros(T, E).scatter_(1, i.long(), v.float())
    assert torch.allclose(full(r.topk_ids, r.topk_w[:, :top]), full(ids, w), atol=1e-5)
    assert torch.allclose(r.topk_w[:, top:].double(), oracle.sigmoid(x.double() @ wr[E:].double().t()).expand(T, 2), atol=1e-6)


@pytest.mark.parametrize("shared", [0, 20, 300])
def test_mixture_with_a_shared_expert(shared):
    from lorax_b200.models.mixers import MoeMlp
    cfg = config([layer(mlp=moe(shared=shared))], width=48)
    w = weights_of(cfg, seed=3)
    c = ModelConfig.from_dict(cfg)
    m = DecoderModel(c, "cpu", torch.float32)
    mlp = MoeMlp(c.layer_specs[0].moe, 48)
    mlp.load(lambda n: w["l0.mlp." + n].float(), lambda t: t, lambda t: t, m)
    x = torch.randn(9, 48, generator=torch.Generator().manual_seed(1))
    rows, (pos, wt) = mlp.run(m, x)
    got = (rows[pos.long()][:, :, :48] * wt[:, :, None]).sum(1)
    want = oracle.mixture(x.double(), {k: v.double() for k, v in w.items()}, "l0.mlp.", cfg["layers"][0]["mlp"])
    assert torch.allclose(got.double(), want, atol=1e-5)
    assert not rows[:, 48:].any()


def test_norms_embedding_and_activation():
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(1)
    x, res = torch.randn(5, 16, generator=g) + 3.0, torch.randn(5, 16, generator=g)
    w, b = torch.randn(16, generator=g), torch.randn(16, generator=g)
    x[:, 10:] = res[:, 10:] = w[10:] = b[10:] = 0
    want = oracle.layer_norm(x[:, :10].double(), w[:10].double(), b[:10].double(), 1e-3)
    r = res.clone()
    ref.norm_add(r, x, w, b, 0.3, 1e-3, 10, torch.float32)
    assert torch.allclose(r[:, :10].double(), res[:, :10].double() + 0.3 * want, atol=1e-5) and not r[:, 10:].any()
    got = ref.norm_stream(x, None, w, 1e-3, 0.0, 10, torch.float32, bias=b, layernorm=True, rows=torch.tensor([3, 0]))
    assert torch.allclose(got[:, :10].double(), want[[3, 0]], atol=1e-5) and not got[:, 10:].any()
    W = {"embed": torch.randn(20, 8, generator=g), "pos": torch.randn(30, 8, generator=g)}
    ids = torch.tensor([4, 19, 4])
    got = ref.embed_stream(ids, W["embed"], pos=W["pos"], positions=torch.tensor([7, 8, 9]))
    assert torch.allclose(got, oracle.embed(W, ids, 7))
    assert torch.allclose(ref.act_mul(x, 16, "relu2", gated=False), oracle.relu2(x))


# ---------------------------------------------------------------------------------------------- whole model
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompts_portions_and_single_tokens(name, device, dtype):
    """The same sequence whole, token by token, and in portions (down to two tokens, around page edges): the logits of every place."""
    cfg = CONFIGS[name]
    w = weights_of(cfg)
    m = build(cfg, w, device, dtype)
    T = 131
    ids = tokens(T, cfg["vocab"], 3)
    want = oracle.forward(cfg, w, ids)
    cuts = {"whole": [T], "single": [1] * T, "two": [2] * (T // 2) + [T % 2], "edges": [31, 2, 31, 1, 62, 2, 2],
            "prompt, then single": [97] + [1] * (T - 97)}
    replay = TraceReplay(m, 160)
    with torch.inference_mode():
        for what, cut in cuts.items():
            got = run_trace(replay, {what: ids}, [[(what, n)] for n in cut if n])[what]
            check(got, want, dtype, what)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("name", ["odd", "aligned"])
def test_mixed_batches_with_pages_used_again(name, device, dtype):
    """Prompts of unequal length beside decode rows, requests that sit out steps, pages handed on: every request against its own run
    alone.  The pool holds little more than what is live."""
    cfg = CONFIGS[name]
    w = weights_of(cfg, seed=1)
    m = build(cfg, w, device, dtype)
    lens = dict(a=70, b=9, c=150, d=33, e=1, f=64, g=40)
    seqs = {k: tokens(n, cfg["vocab"], 10 + i) for i, (k, n) in enumerate(lens.items())}
    steps = [[("a", 60), ("b", 3)], [("b", 1), ("c", 2), ("a", 1)], [("c", 61), ("a", 5), ("b", 1)], [("b", 4), ("a", 4), ("c", 1), ("d", 31)],
             [("e", 1), ("d", 1)], [("d", 1), ("f", 40), ("c", 50)], [("f", 2), ("c", 1)], [("c", 1), ("f", 1)], [("c", 30), ("f", 21), ("g", 39)],
             [("g", 1)], [("c", 4)]]
    with torch.inference_mode():
        got = run_trace(TraceReplay(m, 320), seqs, steps)
    for k, ids in seqs.items():
        check(got[k], oracle.forward(cfg, w, ids[: len(got[k])]), dtype, k)


def edge_model(size, dim, vdim, width=64):
    """One attention layer in which the query of token 1 singles out the key of token 2: queries read the first half of the stream, keys
    the second half with the same matrix, and token 1 has in its first half what token 2 has in its second."""
    cfg = config([layer(heads=2, kv_heads=1, dim=dim, vdim=vdim, size=size, scale=1.0)], width=width, vocab=40, mult=1.0, cap=None)
    w = {k: v.float() for k, v in weights_of(cfg, seed=size).items()}
    g = torch.Generator().manual_seed(size)
    half = width // 2
    u = 3.0 * torch.randn(half, generator=g)
    w["embed"] *= 0.3
    w["embed"][1, :half], w["embed"][2, half:] = u, u
    w["pos"] *= 0.1
    q, k = w["l0.mix.q"], torch.zeros(dim, width)
    k[:, half:] = q[:dim, :half]
    q[:, half:] = 0
    w["l0.mix.k"] = k
    w["l0.mix.q.norm"], w["l0.mix.k.norm"] = torch.full((dim,), 14.0 / dim), torch.ones(dim)
    return cfg, {k: t.to(torch.bfloat16) for k, t in w.items()}


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("size,dim,vdim", [(40, 24, 24), (64, 128, 128), (33, 20, 70), (300, 16, 16)])
def test_keys_just_inside_and_outside_the_window(size, dim, vdim, device, dtype):
    """A key that its query singles out, at the last place that the window holds, the next one, and at page borders; the query in a
    prompt, in a portion and decoded.  That the key decides is checked on the plain statement."""
    cfg, w = edge_model(size, dim, vdim)
    m = build(cfg, w, device, dtype)
    replay = TraceReplay(m, 1100)
    with torch.inference_mode():
        for at in (0, 31, 32, 45):
            for back in (size - 1, size, size // 2):
                ids = tokens(at + back + 1, 36, at + back)
                ids = [4 + i for i in ids]
                ids[at], ids[-1] = 2, 1
                without = list(ids)
                without[at] = 3
                want = oracle.forward(cfg, w, ids)
                change = (want[-1] - oracle.forward(cfg, w, without)[-1]).abs().max()
                assert change > 0.3 if back < size else change < 1e-12, (at, back, float(change))
                T = len(ids)
                for cut in ([T], [T - 2, 2] if T > 2 else [T], [T - 1, 1]):
                    got = run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"]
                    err = (got - want.float()).pow(2).mean(-1).sqrt() / want.std()
                    assert err.max() < (3e-5 if dtype == torch.float32 else 0.05), (at, back, cut, float(err.max()))


@pytest.mark.parametrize("device,dtype", PLACES)
def test_long_context_and_long_decoding(device, dtype):
    """Hundreds of tokens with windows far behind the sequence's end, most of them decoded one by one."""
    cfg = config([layer(heads=2, kv_heads=1, dim=16, vdim=16, size=90, mlp=dense(32)), layer(heads=2, kv_heads=2, dim=16, vdim=24, size=257)], width=64,
                 vocab=128)
    w = weights_of(cfg, seed=4, sharp=4.0)
    m = build(cfg, w, device, dtype)
    T = 600
    ids = tokens(T, 128, 5)
    want = oracle.forward(cfg, w, ids)
    replay = TraceReplay(m, T + 64)
    with torch.inference_mode():
        for cut in ([T], [320, 2, 278], [150] + [1] * (T - 150)):
            check(run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"], want, dtype, str(cut[:3]))


# ---------------------------------------------------------------------------------------------- engine, server, command line
@pytest.mark.parametrize("device,dtype", PLACES[:2])
@pytest.mark.parametrize("name", ["odd", "plain"])
def test_engine_generates_greedily(name, device, dtype):
    """More requests than rows, prompts joining a running batch: greedy tokens equal the plain statement's."""
    from lorax_b200.runtime.engine import Engine, GenRequest
    cfg = CONFIGS[name]
    w = weights_of(cfg, seed=2)
    m = build(cfg, w, device, dtype)
    eng = Engine(m, EngineConfig(max_total_tokens=160, max_batch_prefill_tokens=256), num_blocks=16, max_batch=3)
    prompts = [tokens(n, cfg["vocab"], 40 + n) for n in (5, 33, 1, 64, 2, 17)]
    news = [9, 4, 12, 6, 40, 1]
    with torch.inference_mode():
        for i, (p, n) in enumerate(zip(prompts, news)):
            eng.add_request(GenRequest(i + 1, list(p), n))
        eng.run()
    for i, (p, n) in enumerate(zip(prompts, news)):
        assert eng.finished[i + 1].output_ids == oracle.greedy(cfg, w, p, n), i
    assert eng.alloc.free_blocks == 15 and eng.kv.state_slots is None


def test_engine_samples():
    """Sampling parameters reach the design through the same sampler as every model: a seed repeats, top-1 is greedy."""
    from lorax_b200.runtime.engine import Engine
    from lorax_b200.sampling.chooser import NextTokenParams
    cfg = CONFIGS["odd"]
    w = weights_of(cfg, seed=2)
    m = build(cfg, w, "cpu", torch.float32)
    p = tokens(20, cfg["vocab"], 7)
    run = lambda params: Engine(m, EngineConfig(max_total_tokens=64), num_blocks=16, max_batch=2).generate([p, p], 6, params=params)
    seeded = [NextTokenParams(do_sample=True, temperature=2.0, seed=11), NextTokenParams(do_sample=True, top_k=1, seed=3)]
    with torch.inference_mode():
        a, b = run(seeded), run(seeded)
    assert a == b and a[1] == oracle.greedy(cfg, w, p, 6)


@pytest.mark.parametrize("spec", [0, 3])
def test_shard_serves_portions_prefixes_and_guesses(spec):
    """The shard runtime: a prompt in portions over several Prefill calls, a second request that joins the running batch in one pass and
    starts on cached pages, and (spec) guessed tokens that are checked in one pass."""
    from lorax_b200.server.runtime import ShardRuntime
    cfg = CONFIGS["odd"]
    w = weights_of(cfg, seed=5)
    m = build(cfg, w, "cpu", torch.float32)
    rt = ShardRuntime(m, None, EngineConfig(max_input_length=100, max_total_tokens=128, chunked_prefill=True, prefix_caching=not spec,
                                            speculative_tokens=spec), num_blocks=32, max_batch=4)
    pb = rt.pb
    rt.health()

    def req(rid, ids, new, blocks, cache_len=0, chunk=None):
        r = pb.Request(id=rid, inputs="", truncate=100, blocks=blocks, cache_len=cache_len)
        r.tokenized_inputs.ids.extend(ids)
        r.stopping_parameters.max_new_tokens = new
        if chunk is not None:
            r.chunk_len = chunk
        return r
    p1 = tokens(50, cfg["vocab"], 1)
    p1[20:40] = p1[:20]                                          # something to guess from
    p2 = p1[:32] + tokens(9, cfg["vocab"], 2)
    got = {1: [], 2: []}

    def take(resp):
        for gen in resp.generations:
            got[gen.request_id] += list(gen.next_tokens.ids)
        return resp
    with torch.inference_mode():
        for a, n in ((0, 20), (20, 3)):
            assert not rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=1, requests=[req(1, p1, 9, [1, 2], a, n)], size=1))).generations
        take(rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=1, requests=[req(1, p1, 9, [1, 2], 23)], size=1))))
        resp = take(rt.decode(pb.DecodeRequest(batches=[pb.CachedBatch(id=1)])))
        second = req(2, p2, 5, [3, 4]) if spec else req(2, p2, 5, [1, 4], 32)
        r2 = take(rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=2, requests=[second], size=1), decode_batches=[pb.CachedBatch(id=1)])))
        live = [b for b in (r2.batch,) if r2.HasField("batch")]
        for _ in range(20):
            if not live:
                break
            r = take(rt.decode(pb.DecodeRequest(batches=live)))
            live = [r.batch] if r.HasField("batch") else []
    assert got[1] == oracle.greedy(cfg, w, p1, 9) and got[2] == oracle.greedy(cfg, w, p2, 5)


def save_model(path, cfg, w):
    from safetensors.torch import save_file
    (path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(path / "model.safetensors"))


def test_trace_run_program(tmp_path):
    """bin/trace_run as a program: steps in, logits files and `done` lines out, exit code 0 at the end of its input."""
    import numpy as np
    cfg = CONFIGS["odd"]
    w = weights_of(cfg, seed=6)
    save_model(tmp_path, cfg, w)
    ids = tokens(12, cfg["vocab"], 1)
    steps = [dict(step=0, entries=[dict(id="x", tokens=ids[:9], want=[0, 8]), dict(id="y", tokens=ids[:2], want=[])], end=["y"]),
             dict(step=1, entries=[dict(id="x", tokens=ids[9:10], want=[])], end=[]),
             dict(step=2, entries=[dict(id="y", tokens=ids[:3], want=[2]), dict(id="x", tokens=ids[10:], want=[1])], end=["x", "y"])]
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([sys.executable, os.path.join(REPO, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                       timeout=300)
    assert p.returncode == 0 and [l for l in p.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1", "done 2"], p.stderr
    want = oracle.forward(cfg, w, ids)
    read = lambda n: torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(-1, cfg["vocab"])
    check(read(0), want[[0, 8]], torch.float32)
    check(read(2), torch.stack([oracle.forward(cfg, w, ids[:3])[2], want[11]]), torch.float32)
    assert not (out / "1.f32").exists()


def test_server_builds_the_runtime_from_a_checkpoint(tmp_path):
    from lorax_b200.server.runtime import ShardRuntime, build_runtime
    cfg = CONFIGS["plain"]
    w = weights_of(cfg, seed=7)
    save_model(tmp_path, cfg, w)
    rt = build_runtime(str(tmp_path), EngineConfig(max_input_length=40, max_total_tokens=64), device="cpu", source="local")
    assert type(rt) is ShardRuntime and not rt.model.recurrent and len(rt.model.layers) == 2
    rt.health()
    with pytest.raises(ValueError):
        rt.adapters.register("a", None, {})


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["odd", "aligned"])
def test_cuda_graphs_and_cache_sized_from_free_memory(name):
    """Decode steps as graphs and eagerly give the same tokens; a pool without a given size takes its share of the free memory."""
    from lorax_b200.runtime.engine import Engine, GenRequest
    cfg = CONFIGS[name]
    w = weights_of(cfg, seed=8)
    m = build(cfg, w, "cuda", torch.float32)
    outs = []
    with torch.inference_mode():
        for graphs in (True, False):
            kw = dict(num_blocks=32) if graphs else {}
            eng = Engine(m, EngineConfig(max_total_tokens=128, max_batch_prefill_tokens=256, max_input_length=100, memory_wiggle_room=0.04), max_batch=8,
                         use_graphs=graphs, **kw)
            assert eng.kv.num_blocks >= 16
            for i in range(5):
                eng.add_request(GenRequest(i + 1, tokens(3 + 7 * i, cfg["vocab"], i), 10 + 3 * i))
            eng.run()
            outs.append([eng.finished[i + 1].output_ids for i in range(5)])
    assert outs[0] == outs[1]
    assert outs[0][2] == oracle.greedy(cfg, w, tokens(17, cfg["vocab"], 2), 16)


@pytest.mark.gpu
def test_bf16_rows_do_not_depend_on_the_batch():
    """A request's logits alone, beside others and in portions: equal up to rounding, far below the distance to the exact values."""
    cfg = CONFIGS["aligned"]
    w = weights_of(cfg, seed=9)
    m = build(cfg, w, "cuda", torch.bfloat16)
    ids, other = tokens(90, cfg["vocab"], 1), tokens(77, cfg["vocab"], 2)
    with torch.inference_mode():
        alone = run_trace(TraceReplay(m, 128), {"x": ids}, [[("x", 90)]])["x"]
        beside = run_trace(TraceReplay(m, 320), {"x": ids, "y": other}, [[("y", 40), ("x", 33)], [("x", 57), ("y", 1)], [("y", 36)]])["x"]
    err = (alone - beside).pow(2).mean(-1).sqrt() / alone.std()
    assert err.quantile(0.8) < 0.02, float(err.quantile(0.8))
