"""The Vabunex decoder through the framework (loader, cache and state slots, runner, engine, shard runtime, trace replay) against the
plain float64 statement in `vabunex_oracle.py`, on the CPU operators and, marked gpu, on the CUDA kernels in both number formats."""

import json
import os
import subprocess
import sys

import pytest
import torch

import vabunex_oracle as oracle
from lorax_b200.config import EngineConfig, ModelConfig
from lorax_b200.models.decoder import DecoderModel
from lorax_b200.models.mixers import RandomWeights, tensor_shapes
from lorax_b200.runtime.trace import TraceReplay
from lorax_b200.utils.weights import InMemoryWeights

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PLACES = [pytest.param("cpu", torch.float32, id="cpu"),
          pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="cuda-fp32"),
          pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="cuda-bf16")]


def lightning(heads=3, dim=20, vdim=24, ff=40, decay=None):
    decay = decay or [0.5 + 0.4999 * h / max(heads - 1, 1) for h in range(heads)]
    return dict(type="lightning", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=decay), mlp=dict(kind="dense", ff=ff) if ff else None)


def wkv(heads=2, dim=24, ff=56):
    return dict(type="wkv", mixer=dict(heads=heads, dim=dim), mlp=dict(kind="dense", ff=ff) if ff else None)


def latent(heads=3, dim=24, rot=12, vdim=20, q_rank=28, kv_rank=36, ff=48, base=500.0, scale=0.3):
    return dict(type="latent_attention", mlp=dict(kind="dense", ff=ff) if ff else None,
                mixer=dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot)))


def config(layers, width=72, vocab=150, loop=None, eps=1e-5, scale=1.7):
    c = dict(architecture="Vabunex", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # sizes off every grid, a looped range, layers without a feed-forward
    "odd": config([latent(), lightning(ff=0), wkv(), latent(heads=1, dim=8, rot=2, vdim=9, q_rank=7, kv_rank=5, ff=0)], loop=(1, 3, 3)),
    # recurrent layers only; a decay of 1 and one of 0; one head
    "recurrent": config([wkv(heads=1, dim=40), lightning(heads=4, dim=16, vdim=48, decay=[1.0, 0.0, 0.97, 0.5]), lightning(heads=1, dim=70, vdim=10)],
                        width=100, vocab=97, eps=3e-4, scale=1.0),
    # attention only, a loop over everything
    "attention": config([latent(heads=5, dim=16, rot=16, vdim=32, kv_rank=64), latent(base=1e6, scale=-0.2)], width=64, loop=(0, 2, 2)),
    # sizes of the tensor-core kernels
    "aligned": config([lightning(heads=2, dim=64, vdim=64, ff=128), latent(heads=17, dim=64, rot=64, vdim=64, q_rank=96, kv_rank=128, ff=64, scale=0.09),
                       wkv(heads=2, dim=64, ff=64), latent(heads=2, dim=128, rot=64, vdim=128, q_rank=64, kv_rank=256, scale=0.07)], width=128, vocab=320,
                      loop=(2, 3, 2)),
}


def weights_of(cfg, seed=0, sharp=2.0):
    """Random weights, rounded to bf16.  Queries of the attention layers are scaled so that single keys stand out, decays reach from
    almost none to almost all."""
    rw = RandomWeights(ModelConfig.from_dict(cfg), "cpu", seed)
    out = {}
    for n in rw.shapes:
        t = rw.get_tensor(n)
        if n.endswith("mix.uq"):
            t = t * sharp
        out[n] = t.to(torch.bfloat16)
    return out


def build(cfg, w, device, dtype, max_positions=4096):
    return DecoderModel.from_weights(ModelConfig.from_dict(cfg), InMemoryWeights(w), device, dtype, max_positions=max_positions)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def check(got, want, dtype, what=""):
    want = want.float()
    err = ((got - want).pow(2).mean(-1).sqrt() / want.std()).max()
    assert err < (3e-5 if dtype == torch.float32 else 0.1), (what, float(err))


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
    assert c.model_type == "vabunex" and c.layer_schedule == [0, 1, 2, 1, 2, 1, 2, 3]
    assert c.layer_specs[1].ff == 0 and c.rms_norm_eps == 1e-5 and c.embedding_multiplier == 1.7
    shapes = tensor_shapes(c)
    assert shapes["l0.mix.uq"] == (3 * 36, 28) and shapes["l0.mix.dkv"] == (48, 72) and "l1.mlp.up" not in shapes
    assert shapes["l2.mix.mu.w"] == (72,) and shapes["head"] == (150, 72)
    with pytest.raises(NotImplementedError):
        ModelConfig.from_dict(config([dict(lightning(), mlp=dict(kind="other", ff=8))]))
    with pytest.raises(NotImplementedError):
        DecoderModel.random_init(ModelConfig.from_dict(config([dict(wkv(), type="unknown")])), "cpu", torch.float32)


def test_what_the_design_does_not_offer_is_refused():
    c = ModelConfig.from_dict(CONFIGS["recurrent"])
    m = DecoderModel.random_init(c, "cpu", torch.float32)
    with pytest.raises(ValueError):
        m.quantize("fp8")
    from lorax_b200.server.runtime import ShardRuntime
    for kw in (dict(prefix_caching=True), dict(speculative_tokens=2)):
        with pytest.raises(ValueError):
            ShardRuntime(m, None, EngineConfig(**kw), num_blocks=16, max_batch=2)


# ---------------------------------------------------------------------------------------------- mechanisms alone
def step_of(n, before=0, slot=1):
    from test_mixers_gpu import make_step
    inp, _, _ = make_step([], [(before, n)])
    inp.state_slots.fill_(slot)
    return inp


def test_recurrences_match_their_plain_statement():
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(0)
    T, H, d, dv = 37, 2, 16, 32
    q, k, v = (torch.randn(T, H * n, generator=g, dtype=torch.float64) for n in (d, d, dv))
    decay = torch.tensor([0.9, 0.999], dtype=torch.float64)
    want, S = oracle.linear_attention_scan(*(oracle.silu(x).view(T, H, -1) for x in (q, k, v)), decay)
    state = torch.full((3, H, d, dv), float("nan"))                  # a used slot: what it holds must not matter at position 0
    got = ref.linear_attn(q.float(), k.float(), v.float(), H, d, dv, decay.float(), state, step_of(T))
    assert torch.allclose(got.double().view(T, H, dv), want, atol=1e-4) and torch.allclose(state[1].double(), S, atol=1e-4)
    r, k, v, z = (torch.randn(T, H * d, generator=g, dtype=torch.float64) for _ in range(4))
    w0, u = torch.randn(H * d, generator=g, dtype=torch.float64), torch.randn(H * d, generator=g, dtype=torch.float64)
    w = torch.exp(-torch.exp(z + w0)).view(T, H, d)
    want, S = oracle.wkv_scan(r.view(T, H, d), k.view(T, H, d), v.view(T, H, d), w, u.view(H, d))
    state = torch.full((3, H, d, d), float("nan"))
    got = ref.wkv(r.float(), k.float(), v.float(), z.float(), w0.float(), u.float(), H, d, state, step_of(T))
    assert torch.allclose(got.double().view(T, H, d), want, atol=1e-4) and torch.allclose(state[1].double(), S, atol=1e-4)


def test_rotation_shift_and_norms_match_their_plain_statement():
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(1)
    pos = torch.tensor([0, 1, 77, 4095])
    x = torch.randn(4, 2 * 30, generator=g, dtype=torch.float64)
    y = x.float().clone()
    ref.rope_pairs(y, pos, ref.rope_table(10, 4096, 100.0), 2, 30, 20, 10)
    for i, p in enumerate(pos.tolist()):
        for h in range(2):
            s = slice(h * 30, h * 30 + 30)
            want = torch.cat([x[i, s][:20], oracle.rotate_pairs(x[i, s][20:], p, 100.0)])
            assert torch.allclose(y[i, s].double(), want, atol=2e-4)
    h, mu, shift = torch.randn(5, 8, generator=g), torch.rand(2, 8, generator=g), torch.randn(3, 8, generator=g)
    before = shift[1].clone()
    first = ref.token_shift(h, mu, shift.clone(), step_of(5))
    later = ref.token_shift(h, mu, shift, step_of(5, before=9))
    assert torch.allclose(first[1][0], h[0] - h[0] * mu[1]) and torch.allclose(later[1][0], h[0] + (before - h[0]) * mu[1])
    assert torch.allclose(later[0][3], h[3] + (h[2] - h[3]) * mu[0]) and torch.equal(shift[1], h[4])
    r, p, w = torch.randn(3, 16, generator=g), torch.randn(3, 16, generator=g), torch.randn(16, generator=g)
    r[:, 10:] = p[:, 10:] = 0
    want = oracle.rms((r + p)[:, :10].double(), 1e-3) * (1 + w[:10].double())
    assert torch.allclose(ref.norm_stream(r, p, w, 1e-3, 1.0, 10, torch.float32)[:, :10].double(), want, atol=1e-5)


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
def test_mixed_batches_with_pages_and_slots_used_again(name, device, dtype):
    """Prompts of unequal length beside decode rows, requests that sit out steps, pages and slots handed on: every request against its
    own run alone.  The pool holds little more than what is live."""
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
        if k in got and len(got[k]) == len(ids):
            check(got[k], oracle.forward(cfg, w, ids), dtype, k)
        else:
            check(got[k], oracle.forward(cfg, w, ids[: len(got[k])]), dtype, k)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_long_context_with_a_far_key(device, dtype):
    """One early token carries a key that a late query singles out among hundreds (the logits change when it is dropped), read from a
    prompt's portion and from decoded tokens."""
    cfg = config([latent(heads=2, dim=16, rot=16, vdim=16, q_rank=32, kv_rank=48, base=1e8, scale=0.25), wkv(heads=2, dim=16)], width=64, vocab=128)
    w = weights_of(cfg, seed=4, sharp=6.0)
    m = build(cfg, w, device, dtype)
    T = 700
    ids = tokens(T, 100, 5)
    ids[33] = 120
    want = oracle.forward(cfg, w, ids)
    other = list(ids)
    other[33] = 121
    assert (oracle.forward(cfg, w, other)[-1] - want[-1]).abs().max() > 1e-3
    replay = TraceReplay(m, T + 64)
    with torch.inference_mode():
        for cut in ([T], [320, 320] + [1] * 60, [650, 2, 48]):
            got = run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"]
            check(got, want, dtype, str(cut[:3]))


# ---------------------------------------------------------------------------------------------- engine, server, command line
@pytest.mark.parametrize("device,dtype", PLACES[:2])
@pytest.mark.parametrize("name", ["odd", "recurrent"])
def test_engine_generates_greedily(name, device, dtype):
    """More requests than rows and slots, prompts joining a running batch: greedy tokens equal the plain statement's."""
    from lorax_b200.runtime.engine import Engine
    cfg = CONFIGS[name]
    w = weights_of(cfg, seed=2)
    m = build(cfg, w, device, dtype)
    eng = Engine(m, EngineConfig(max_total_tokens=160, max_batch_prefill_tokens=256), num_blocks=16, max_batch=3)
    prompts = [tokens(n, cfg["vocab"], 40 + n) for n in (5, 33, 1, 64, 2, 17)]
    news = [9, 4, 12, 6, 40, 1]
    from lorax_b200.runtime.engine import GenRequest
    with torch.inference_mode():
        for i, (p, n) in enumerate(zip(prompts, news)):
            eng.add_request(GenRequest(i + 1, list(p), n))
        eng.run()
    for i, (p, n) in enumerate(zip(prompts, news)):
        assert eng.finished[i + 1].output_ids == oracle.greedy(cfg, w, p, n), i
    assert eng.alloc.free_blocks == 15
    assert len(eng.kv.state_slots.free) == eng.kv.state_slots.num_slots - 1 and not eng.kv.state_slots.of_request


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


def test_shard_serves_portions_of_prompts_and_fused_steps():
    """The shard runtime: a prompt in portions over several Prefill calls keeps its state slot, a second request joins a running batch
    in one pass, finished and cleared requests give their slots back."""
    from lorax_b200.server.runtime import ShardRuntime
    cfg = CONFIGS["odd"]
    w = weights_of(cfg, seed=5)
    m = build(cfg, w, "cpu", torch.float32)
    rt = ShardRuntime(m, None, EngineConfig(max_input_length=100, max_total_tokens=128, chunked_prefill=True), num_blocks=32, max_batch=4)
    pb = rt.pb
    rt.health()

    def req(rid, ids, new, blocks, cache_len=0, chunk=None):
        r = pb.Request(id=rid, inputs="", truncate=100, blocks=blocks, cache_len=cache_len)
        r.tokenized_inputs.ids.extend(ids)
        r.stopping_parameters.max_new_tokens = new
        if chunk is not None:
            r.chunk_len = chunk
        return r
    p1, p2 = tokens(50, cfg["vocab"], 1), tokens(13, cfg["vocab"], 2)
    with torch.inference_mode():
        got = {1: [], 2: []}

        def take(resp):
            for gen in resp.generations:
                got[gen.request_id] += list(gen.next_tokens.ids)
            return resp
        for a, n in ((0, 20), (20, 3)):
            assert not rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=1, requests=[req(1, p1, 7, [1, 2], a, n)], size=1))).generations
        with pytest.raises(RuntimeError):                     # a portion whose beginning this shard has not seen
            rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=9, requests=[req(9, p2, 2, [7], 5)], size=1)))
        take(rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=1, requests=[req(1, p1, 7, [1, 2], 23)], size=1))))
        take(rt.decode(pb.DecodeRequest(batches=[pb.CachedBatch(id=1)])))
        resp = take(rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=2, requests=[req(2, p2, 4, [3])], size=1), decode_batches=[pb.CachedBatch(id=1)])))
        assert rt.fused_stats["one_pass"] == 1
        while resp.HasField("batch"):
            resp = take(rt.decode(pb.DecodeRequest(batches=[resp.batch])))
    assert got[1] == oracle.greedy(cfg, w, p1, 7) and got[2] == oracle.greedy(cfg, w, p2, 4)
    assert not rt.kv.state_slots.of_request
    rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=3, requests=[req(3, p1, 7, [1, 2], 0, 20)], size=1)))
    assert len(rt.kv.state_slots.of_request) == 1
    rt.clear_cache(pb.ClearCacheRequest())
    assert not rt.kv.state_slots.of_request


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
    cfg = CONFIGS["recurrent"]
    w = weights_of(cfg, seed=7)
    save_model(tmp_path, cfg, w)
    rt = build_runtime(str(tmp_path), EngineConfig(max_input_length=40, max_total_tokens=64), device="cpu", source="local")
    assert type(rt) is ShardRuntime and rt.model.recurrent and not rt.model.layers[0].mixer.shapes() == {}
    rt.health()
    with pytest.raises(ValueError):
        rt.adapters.register("a", None, {})


@pytest.mark.gpu
def test_cuda_graphs_do_not_advance_the_state():
    """Capturing a decode graph runs the step once outside the capture: the live requests' state must not notice."""
    from lorax_b200.runtime.engine import Engine, GenRequest
    cfg = CONFIGS["recurrent"]
    w = weights_of(cfg, seed=8)
    m = build(cfg, w, "cuda", torch.float32)
    outs = []
    with torch.inference_mode():
        for graphs in (True, False):
            eng = Engine(m, EngineConfig(max_total_tokens=128), num_blocks=32, max_batch=8, use_graphs=graphs)
            for i in range(5):
                eng.add_request(GenRequest(i + 1, tokens(3 + 7 * i, cfg["vocab"], i), 10 + 3 * i))
            eng.run()
            outs.append([eng.finished[i + 1].output_ids for i in range(5)])
    assert outs[0] == outs[1]
    assert outs[0][2] == oracle.greedy(cfg, w, tokens(17, cfg["vocab"], 2), 16)


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["aligned", "recurrent"])
def test_cache_is_sized_from_free_memory(name):
    """No block count given: a maximum prefill is measured and the pool takes its share of what is left beside the states."""
    from lorax_b200.runtime.engine import Engine
    cfg = CONFIGS[name]
    w = weights_of(cfg, seed=9)
    m = build(cfg, w, "cuda", torch.float32)
    with torch.inference_mode():
        eng = Engine(m, EngineConfig(max_total_tokens=128, max_batch_prefill_tokens=256, max_input_length=100, memory_wiggle_room=0.04), max_batch=4)
        p = tokens(21, cfg["vocab"], 3)
        assert eng.kv.num_blocks >= 16
        assert eng.generate([p, p[:5]], 6) == [oracle.greedy(cfg, w, p, 6), oracle.greedy(cfg, w, p[:5], 6)]


@pytest.mark.gpu
def test_prompts_that_fill_the_gpu_take_one_segment_each():
    """Many heads and several prompts: the recurrences run without the pass over segment states; same results as alone."""
    cfg = config([wkv(heads=64, dim=64, ff=0), lightning(heads=60, dim=64, vdim=128, ff=0)], width=64, vocab=100)
    w = weights_of(cfg, seed=10)
    m = build(cfg, w, "cuda", torch.bfloat16)
    from lorax_b200.runtime.runner import PrefillItem
    seqs = [tokens(n, 100, n) for n in (150, 149, 131, 90)]
    with torch.inference_mode():
        r = TraceReplay(m, 640)
        for i in range(4):
            r.alloc.extend(r.held.setdefault(str(i), []), len(seqs[i]))
        items = [PrefillItem(s, 0, r.held[str(i)], state_slot=i + 1, logit_rows=[0, 63, 64, len(s) - 1]) for i, s in enumerate(seqs)]
        assert r.runner._prefill_inputs(items)[0].seg_len == 192
        _, _, logits = r.runner.prefill(items)
        for i, s in enumerate(seqs):
            check(logits[4 * i: 4 * i + 4].float().cpu(), oracle.forward(cfg, w, s)[[0, 63, 64, len(s) - 1]], torch.bfloat16)
