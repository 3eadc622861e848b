"""The Fegolorn decoder through the framework (loader, paged cache, runner, engine, shard runtime, trace replay) against the plain float64
statement in `fegolorn_oracle.py`, on the CPU operators and, marked gpu, on the CUDA kernels in both number formats."""

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import fegolorn_oracle as oracle
from lorax_b200.config import EngineConfig, ModelConfig
from lorax_b200.models.decoder import DecoderModel
from lorax_b200.models.mixers import RandomWeights, tensor_shapes
from lorax_b200.runtime.trace import TraceReplay
from lorax_b200.utils.weights import InMemoryWeights

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PLACES = [pytest.param("cpu", torch.float32, id="cpu"),
          pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="cuda-fp32"),
          pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="cuda-bf16")]
BANDS = dict(factor=3.0, low=1.0, high=5.0, original=90)


@pytest.fixture(autouse=True)
def _one_thread():
    """The tensors are small: threads would cost more than they bring."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def dense(ff=44, limit=0.7):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts=10, top=3, ff=36, shared=50):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def attention(mlp=None, weights_of=None, heads=6, kv_heads=2, dim=20, vdim=28, scale=0.3, dims=12, base=300.0, scaling=BANDS):
    rot = dict(base=base, dims=dims)
    if scaling:
        rot["scaling"] = scaling
    layer = dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=rot))
    return layer if weights_of is None else dict(layer, weights_of=weights_of)


def latent(mlp=None, weights_of=None, heads=3, dim=24, rot_dim=10, vdim=36, kv_rank=40, size=40, scale=0.25, base=200.0):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dim))
    if size:
        m["mask"] = dict(size=size)
    layer = dict(type="latent_attention", mlp=mlp, mixer=m)
    return layer if weights_of is None else dict(layer, weights_of=weights_of)


def config(layers, width=76, vocab=150, eps=1e-5, bigram=(61, 31, 5), scale=1.3, cap=9.0):
    e = dict(scale=scale)
    if bigram:
        e["bigram"] = dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2])
    c = dict(architecture="Fegolorn", vocab=vocab, width=width, norm=dict(eps=eps), embedding=e, layers=layers)
    if cap:
        c["logit_softcap"] = cap
    return c


CONFIGS = {
    # sizes off every grid, layers without a feed-forward, layers that use the weights of an earlier one, of one that does so itself, and
    # of a later one
    "odd": config([latent(moe()), attention(dense()), latent(moe(), weights_of=0), attention(dense(), weights_of=1), latent(moe(), weights_of=2),
                   attention(None, weights_of=7, heads=3, kv_heads=3, dim=70, vdim=10, dims=70, scaling=None, scale=0.1),
                   latent(None, heads=5, dim=9, rot_dim=2, vdim=7, kv_rank=23, size=33, scale=0.4),
                   attention(None, heads=3, kv_heads=3, dim=70, vdim=10, dims=70, scaling=None, scale=0.1)]),
    # everything that can be 1, windows of one token and past the sequence, a rotation of one pair, bands of factor 1, negative scale,
    # neither token pairs nor a cap
    "plain": config([attention(moe(experts=1, top=1, ff=20, shared=None), heads=1, kv_heads=1, dim=16, vdim=2, dims=2, scaling=dict(BANDS, factor=1.0)),
                     latent(dense(1, 50.0), heads=1, dim=1, rot_dim=16, vdim=1, kv_rank=1, size=1),
                     latent(moe(experts=4, top=4, shared=5), size=1000, scale=-0.3), latent(None, size=None),
                     attention(moe(experts=6, top=2, shared=None), heads=4, kv_heads=1, dim=24, vdim=24, scale=-0.4)], width=100, eps=3e-4, bigram=None, cap=None),
    # sizes of the tensor-core kernels
    "aligned": config([latent(moe(experts=40, top=6, ff=128, shared=320), heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=256, size=70, scale=0.07),
                       attention(dense(256, 1.5), heads=4, kv_heads=2, dim=128, vdim=120, dims=64, scale=0.09),
                       latent(dense(256, 1.5), heads=18, dim=64, rot_dim=32, vdim=128, kv_rank=128, size=33, scale=0.1),
                       attention(moe(experts=16, top=2, ff=64, shared=64), heads=16, kv_heads=1, dim=128, vdim=128, dims=128, scale=0.09),
                       latent(None, heads=6, dim=64, rot_dim=48, vdim=64, kv_rank=512, size=150, scale=0.1),
                       latent(dense(256, 1.5), weights_of=2, heads=18, dim=64, rot_dim=32, vdim=128, kv_rank=128, size=33, scale=0.1)],
                      width=256, vocab=320, bigram=(127, 61, 3)),
}


def weights_of(cfg, seed=0, sharp=2.0):
    """Random weights, rounded to bf16.  Queries are scaled so that single keys stand out."""
    rw = RandomWeights(ModelConfig.from_dict(cfg), "cpu", seed)
    out = {}
    for n in rw.shapes:
        t = rw.get_tensor(n)
        if n.endswith(("mix.q", "q.norm")):
            t = t * sharp
        if n.endswith("router"):
            t = t * 2
        if n.endswith("router.b"):
            t = t * 8
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
        assert err.max() < 3e-5, (what, float(err.max()), int(err.argmax()))
    else:
        # rounding decides between experts whose scores are nearly equal: such tokens, and the few that look at them, may differ
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
    assert c.model_type == "fegolorn" and c.layer_style == "sandwich" and c.hidden_act == "silu" and c.norm_type == "rms"
    assert c.residual_gate and c.layer_scale and c.norm_scalar and c.bigram == (61, 31, 5) and c.final_logit_softcapping == 9.0
    m = c.layer_specs[0].moe
    assert (m.experts, m.top, m.ff, m.score, m.renorm, m.gated, m.bias, m.shared_ff, m.shared_gate) == (10, 3, 36, "softmax", True, True, True, 50, False)
    assert [s.weights_of for s in c.layer_specs] == [None, None, 0, 1, 0, 7, None, None]
    assert (c.layer_specs[1].act, c.layer_specs[1].limit) == ("clamped_swiglu", 0.7)
    shapes = tensor_shapes(c)
    assert shapes["l0.mix.q"] == (3 * 34, 76) and shapes["l0.mix.dkv"] == (50, 76) and shapes["l0.mix.uv"] == (108, 40) and shapes["l0.mix.g"] == (108, 76)
    assert shapes["l1.mix.q"] == (120, 76) and shapes["l1.mix.k.norm"] == (20,) and shapes["l1.mix.v"] == (56, 76) and shapes["l1.mix.o"] == (76, 168)
    assert shapes["l0.norm1"] == shapes["l0.norm2b"] == shapes["final.norm"] == () and shapes["l0.ls2"] == (76,) and shapes["l1.rg1"] == (76, 76)
    assert shapes["l1.rg2.b"] == (76,) and shapes["l0.mlp.router.b"] == (10,) and shapes["l0.mlp.shared.up"] == (50, 76) and shapes["bigram"] == (62, 76)
    for absent in ("l0.mix.dq", "l1.mix.g", "l0.mlp.shared.sg", "l0.mlp.correction", "l2.mix.q", "l5.norm1", "l6.norm2", "l6.ls2", "l7.rg2", "pos", "l0.norm1.b"):
        assert absent not in shapes, absent
    assert sorted({n.split(".")[0] for n in shapes if n[0] == "l"}) == ["l0", "l1", "l6", "l7"]
    for bad in ([attention(moe(top=11))], [attention(weights_of=1)], [attention(weights_of=0)], [attention(), attention(weights_of=0, dim=24)],
                [attention(), attention(dense(), weights_of=0)], [attention(), latent(weights_of=0)],
                [attention(weights_of=1), attention(weights_of=0)]):
        with pytest.raises(ValueError):
            ModelConfig.from_dict(config(bad))
    build_ = lambda layers: DecoderModel.random_init(ModelConfig.from_dict(config(layers)), "cpu", torch.float32)
    for bad in ([attention(heads=5)], [attention(dims=22)], [attention(dims=3)], [attention(vdim=7)], [latent(rot_dim=5)], [latent(size=-2)]):
        with pytest.raises(ValueError):
            build_(bad)
    for bad in ([attention(dim=257)], [dict(attention(), type="other")], [attention(dict(kind="other"))]):
        with pytest.raises(NotImplementedError):
            build_(bad)


def test_layers_share_weights_and_not_their_cache():
    from lorax_b200.runtime.kv_cache import cache_bytes, make_cache
    m = DecoderModel.random_init(ModelConfig.from_dict(CONFIGS["odd"]), "cpu", torch.float32)
    assert m.layers[2] is m.layers[0] and m.layers[4] is m.layers[0] and m.layers[5] is m.layers[7] and m.layers[3] is m.layers[1]
    kv = make_cache(m, EngineConfig(), 4, 2)
    assert len(kv.layers) == 9 and len({t.data_ptr() for t in kv.layers}) == 9 and kv.state_slots is None
    assert kv.layers[0].shape == (4, 32, 48 + 16) and kv.layers[1].shape == (4, 2, 32 * (64 + 64)) and kv.layers[8].shape == (4, 32)
    assert kv.layers[8].dtype == torch.int32
    per_block, fixed = cache_bytes(m, EngineConfig(), 2)
    assert fixed == 0 and sum(t.numel() * t.element_size() for t in kv.layers) == per_block * 4
    assert m.context_windows == [33, 40]


def test_what_the_design_does_not_offer_is_refused():
    from lorax_b200.server.runtime import ShardRuntime
    m = DecoderModel.random_init(ModelConfig.from_dict(CONFIGS["odd"]), "cpu", torch.float32, max_positions=500)
    assert not m.recurrent
    with pytest.raises(ValueError):
        m.quantize("fp8")
    for kw in (dict(kv_cache_dtype="fp8"), dict(max_total_tokens=501)):
        with pytest.raises(ValueError):
            ShardRuntime(m, None, EngineConfig(**dict(dict(max_total_tokens=100), **kw)), num_blocks=32, max_batch=2)


# ---------------------------------------------------------------------------------------------- mechanisms alone
def step_of(n, before=0):
    from test_mixers_gpu import make_step
    return make_step([], [(before, n)])


@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(61, 31, 5), (1, 3, 2), (997, 1 << 33, 12345678901), (40, 0, 1)])
def test_token_pairs_across_portions(buckets, mul_prev, mul_cur):
    """The token before is carried by the pages, over portions of any size, single tokens and other requests' ids in a page."""
    from lorax_b200.ops import reference as ref
    from test_mixers_gpu import make_step
    g = torch.Generator().manual_seed(buckets)
    T, V, width = 70, 50, 8
    W = dict(embed=torch.randn(V, width, generator=g).double(), bigram=torch.randn(buckets + 1, width, generator=g).double())
    ids = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    want = oracle.embed(ids.tolist(), W, dict(scale=0.6, bigram=dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)))
    for cut in ([T], [1] * T, [31, 2, 30, 1, 6]):
        pages, out, at = torch.randint(0, V, (12, 32), generator=g, dtype=torch.int32), [], 0
        for n in cut:
            dec = n == 1 and at > 0
            inp, _, _ = make_step([at + 1] if dec else [], [] if dec else [(at, n)], pages_per_seq=4)
            out.append(ref.embed_stream(ids[at: at + n], W["embed"].float(), 0.6, bigram=(W["bigram"].float(), (buckets, mul_prev, mul_cur), pages, inp)))
            at += n
        assert torch.allclose(torch.cat(out).double(), want, atol=1e-5)


@pytest.mark.parametrize("scaling", [None, BANDS, dict(factor=8.0, low=1.0, high=4.0, original=8192), dict(factor=2.0, low=0.5, high=0.5001, original=64),
                                     dict(factor=1.0, low=1.0, high=2.0, original=5), dict(factor=4.0, low=1.0, high=4.0, original=1)])
@pytest.mark.parametrize("n,base", [(2, 100.0), (12, 300.0), (64, 500000.0)])
def test_frequency_bands(n, base, scaling):
    from lorax_b200.ops import reference as ref
    f = oracle.frequencies(n, base, scaling)
    a = torch.arange(0, 3000, 37, dtype=torch.float64)[:, None] * f
    table = ref.rope_table(n, 3000, base, scaling=scaling)[::37].double()
    assert torch.allclose(table, torch.cat([a.cos(), a.sin()], -1), atol=1e-6)


@pytest.mark.parametrize("H,G,d,dv,dims,first", [(4, 2, 16, 12, 16, 0), (3, 3, 20, 2, 6, 700), (6, 1, 10, 34, 2, 33), (1, 1, 64, 64, 64, 2000)])
def test_normed_heads_rotated_values_and_outputs_turned_back(H, G, d, dv, dims, first):
    """Attention of the last rows of a sequence over all of its keys, heads padded as the layers pad them.  One query and key stand out."""
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(d)
    T, n, dk, dw = first + 40, 40, 64, 64
    q, k, v = (torch.randn(T, h, w, generator=g) for h, w in ((H, d), (G, d), (G, dv)))
    q[-1], k[first // 2] = k[first // 2].repeat_interleave(H // G, 0) * 3, k[first // 2] * 2
    wq, wk = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) + 0.5
    f, fv = oracle.frequencies(dims, 300.0, BANDS), oracle.frequencies(dv, 300.0)
    norm = lambda x, w: oracle.turn(oracle.rms_norm(x.double(), w.double(), 1e-3), dims, f)
    want = oracle.turn(oracle.attend(norm(q, wq), norm(k, wk), oracle.turn(v.double(), dv, fv), 0.4, oracle.visible(T)), dv, fv, back=True)
    pad = torch.nn.functional.pad
    rows = torch.cat([pad(x, (0, w - x.shape[2])).reshape(T, -1) for x, w in ((q, dk), (k, dk), (v, dw))], 1)
    inp, nb, _ = step_of(n, first)
    cs, vcs = ref.rope_table(dims, T, 300.0, scaling=BANDS), ref.rope_table(dv, T, 300.0)
    cache, out = torch.zeros(nb, G, 32 * (dk + dw)), torch.empty(n, H * dw)
    args = lambda a, b: (rows[a:b], H, G, dk, dw, d, pad(wq, (0, dk - d)), pad(wk, (0, dk - d)), 1e-3, cache)
    if first:
        old, _, _ = step_of(first)
        table = inp.block_tables[0]
        ref.qk_norm_kvwrite(*args(0, first), torch.tensor([int(table[t // 32]) * 32 + t % 32 for t in range(first)]), positions=old.positions, cos_sin=cs,
                            v_cos_sin=vcs)
    ref.qk_norm_kvwrite(*args(first, T), inp.slots, positions=inp.positions, cos_sin=cs, v_cos_sin=vcs)
    ref.gqa_attn(rows[first:], cache, H, G, dk, dw, 0.4, 0, inp, out, turn_back=vcs)
    assert torch.allclose(out.view(n, H, dw)[:, :, :dv].double(), want[first:], atol=2e-4) and not out.view(n, H, dw)[:, :, dv:].any()


@pytest.mark.parametrize("kw", [dict(), dict(size=1), dict(size=None), dict(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1), dict(size=16, rot_dim=16, scale=-0.6)])
def test_latent_attention_mixer(kw):
    """The mixer itself in portions, against the statement."""
    from lorax_b200.models.mixers import LatentAttentionMixer
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(7)
    T, width, p = 50, 24, latent(**kw)["mixer"]
    mx = LatentAttentionMixer(dict(p, gate="element", rot_layout="halves"), width)
    W = {n: torch.randn(*s, generator=g) for n, s in mx.shapes().items()}
    h = torch.randn(T, width, generator=g)
    want = oracle.latent_attention(h.double(), {k: v.double() for k, v in W.items()}, "", p, 1e-3)

    class Model:
        ops, eps, dtype = ref, 1e-3, torch.float32
        rope_table = staticmethod(lambda rot, base, scaling=None: ref.rope_table(rot, 64, base, scaling=scaling))
    mx.load(lambda n: W[n], lambda t: t, lambda t: t.contiguous(), Model)
    proj = {n: torch.nn.functional.pad(h, (0, mx.W - width)) @ t.t() for n, t in mx.in_parts(lambda n: W[n])}
    cache, y, at = torch.randn(4, 32, mx.kvp + mx.rp), torch.empty(T, mx.out_dim), 0
    for n in (1, 30, 2, 17):
        inp, _, _ = step_of(n, at)
        inp.block_tables = torch.tensor([[3, 1]], dtype=torch.int32)
        inp.slots = torch.tensor([(3, 1)[t // 32] * 32 + t % 32 for t in range(at, at + n)])
        mx.run(Model, None, {k: v[at: at + n] for k, v in proj.items()}, y[at: at + n], inp, cache)
        at += n
    assert torch.allclose(y.view(T, mx.H, mx.dvp)[:, :, : mx.dv].reshape(T, -1).double(), want, atol=1e-4)


@pytest.mark.parametrize("E,top", [(12, 3), (9, 1), (8, 8), (1, 1)])
def test_routing_with_a_bias(E, top):
    """The bias takes part in the choice and in the weights; shared experts count once."""
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(E)
    T = 50
    x, wr, b = torch.randn(T, 24, generator=g), torch.randn(E, 24, generator=g) * 0.5, torch.randn(E, generator=g) * 2
    ids, w = oracle.route(x.double() @ wr.double().t() + b.double(), top)
    r = ref.moe_route(x, wr, top, 0, E, experts=E, score="softmax", renorm=True, bias=b, shared=2, shared_gate=False)
    full = lambda i, v: torch.zeros(T, E).scatter_(1, i.long(), v.float())
    assert torch.allclose(full(r.topk_ids, r.topk_w[:, :top]), full(ids, w), atol=1e-6) and (r.topk_w[:, top:] == 1).all()
    if 1 < top < E:
        assert (ids.sort(-1).values != oracle.route(x.double() @ wr.double().t(), top)[0].sort(-1).values).any()


def test_feed_forwards():
    from lorax_b200.models.mixers import make_mlp
    for mlp in (moe(), moe(ff=70, shared=None), moe(experts=2, top=2, shared=200), dense(20), dense(20, 0.05), dense(33, 100.0)):
        cfg = config([attention(mlp)], width=48)
        w = {k: v * (4 if k.endswith((".gate", ".up")) else 1) for k, v in weights_of(cfg, seed=3).items()}
        c = ModelConfig.from_dict(cfg)
        m = DecoderModel(c, "cpu", torch.float32)
        mod = make_mlp(c.layer_specs[0], 48)
        g = torch.Generator().manual_seed(1)
        beside = torch.randn(48, 48, generator=g), torch.randn(48, generator=g)
        mod.load(lambda n: w["l0.mlp." + n].float(), lambda t: t, lambda t: t, m, beside=beside)
        x = torch.randn(9, 48, generator=g)
        rows, pairs, z = mod.run_beside(m, x)
        got = rows if pairs is None else (rows[pairs[0].long()][:, :, :48] * pairs[1][:, :, None]).sum(1)
        want = oracle.feed_forward(x.double(), {k: v.double() for k, v in w.items()}, "l0.mlp.", mlp)
        assert torch.allclose(got.double(), want, atol=1e-4) and torch.allclose(z, x @ beside[0].t() + beside[1], atol=1e-4)


def test_a_sublayer_is_gated_normed_scaled_added_and_normed_for_the_next():
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(2)
    T, n, W = 9, 44, 48
    x, y, z, w, nxt = (torch.randn(*s, generator=g) for s in ((T, W), (T, W), (T, W), (W,), (W,)))
    for t in (x, y, w, nxt):
        t[..., n:] = 0
    res = x.clone()
    rows = torch.tensor([7, 0, 3], dtype=torch.int32)
    h = ref.norm_add(res, y, w, None, 1.0, 0.3, n, torch.float32, layernorm=False, gate=z, next_weight=nxt)
    picked = ref.norm_add(x.clone(), y, w, None, 1.0, 0.3, n, torch.float32, layernorm=False, gate=z, next_weight=nxt, rows=rows)
    d = lambda t: t[..., :n].double()
    want = d(x) + oracle.rms_norm(d(y) * oracle.sigmoid(d(z)), d(w), 0.3)
    assert torch.allclose(d(res), want, atol=1e-5) and torch.allclose(d(h), oracle.rms_norm(want, d(nxt), 0.3), atol=1e-5)
    assert torch.equal(picked, h[rows.long()])


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


def edge_model(kind, size, dim, vdim, width=64):
    """One layer in which the query of token 1 singles out the key of token 2: queries read the first half of the stream, keys (or the
    latent) the second half with the same matrix, and token 1 has in its first half what token 2 has in its second.  The rotated
    dimensions are left out, and the token pairs."""
    cfg = config([attention(heads=2, kv_heads=1, dim=dim, vdim=vdim, scale=24.0 / dim, dims=4, scaling=None) if kind == "attention" else
                  latent(heads=2, dim=dim, rot_dim=16, vdim=vdim, kv_rank=128, size=size, scale=1.5 * dim ** -0.5)], width=width, vocab=40, scale=1.0)
    w = {k: v.float() for k, v in weights_of(cfg, seed=dim + vdim, sharp=1.0).items()}
    g = torch.Generator().manual_seed(dim)
    half, p = width // 2, "l0.mix."
    u = 3.0 * torch.randn(half, generator=g)
    w["embed"] *= 0.3
    w["embed"][1, :half], w["embed"][2, half:] = u, u
    w["bigram"] *= 0
    if kind == "attention":
        q, k = torch.randn(2, dim, width, generator=g) * width ** -0.5, torch.zeros(dim, width)
        q[1] = q[0]
        q[:, :4], q[:, :, half:] = 0, 0
        k[:, half:] = q[0, :, :half]
        w[p + "q"], w[p + "k"], w[p + "q.norm"], w[p + "k.norm"] = q.reshape(2 * dim, width), k, torch.ones(dim), torch.ones(dim)
    else:
        rank = 128
        down, up = torch.zeros(rank + 16, width), torch.randn(dim, rank, generator=g) * rank ** -0.5
        down[:rank, half:] = torch.randn(rank, half, generator=g) * half ** -0.5
        q = torch.zeros(2, dim + 16, width)
        q[:, :dim, :half] = up @ down[:rank, half:]
        w[p + "q"], w[p + "dkv"], w[p + "uk"], w[p + "dkv.norm"] = q.reshape(-1, width), down, torch.cat([up, up]), torch.ones(rank)
    return cfg, {k: t.to(torch.bfloat16) for k, t in w.items()}


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("size,dim,vdim", [(40, 24, 24), (64, 128, 128), (33, 64, 70), (300, 64, 64)])
def test_keys_just_inside_and_outside_the_window(size, dim, vdim, device, dtype):
    """A key that its query singles out, at the last place that the window holds, the next one, and at page borders; the query in a
    prompt, in a portion and decoded.  That the key decides is checked on the plain statement."""
    cfg, w = edge_model("latent_attention", size, dim, vdim)
    m = build(cfg, w, device, dtype)
    replay = TraceReplay(m, 1100)
    with torch.inference_mode():
        for at in (0, 31, 32, 45):
            for back in (size - 1, size, size // 2):
                ids = [4 + i for i in tokens(at + back + 1, 36, at + back)]
                ids[at], ids[-1] = 2, 1
                without = list(ids)
                without[at] = 3
                want = oracle.forward(cfg, w, ids)
                change = (want[-1] - oracle.forward(cfg, w, without)[-1]).abs().max()
                assert change > 0.2 if back < size else change < 1e-12, (at, back, float(change))
                T = len(ids)
                for cut in ([T], [T - 2, 2], [T - 1, 1], [max(T - 30, 1), min(T - 1, 30)]):
                    got = run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"]
                    err = (got - want.float()).pow(2).mean(-1).sqrt() / want.std()
                    assert err.max() < (3e-5 if dtype == torch.float32 else 0.05), (at, back, cut, float(err.max()))


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("dim,vdim", [(24, 30), (128, 128)])
def test_a_key_far_away(dim, vdim, device, dtype):
    """One key among hundreds, its value turned by its own position and back by the query's."""
    cfg, w = edge_model("attention", None, dim, vdim)
    m = build(cfg, w, device, dtype)
    replay = TraceReplay(m, 700)
    with torch.inference_mode():
        for at, T in ((0, 600), (63, 501), (64, 66)):
            ids = [4 + i for i in tokens(T, 36, at)]
            ids[at], ids[-1] = 2, 1
            without = list(ids)
            without[at] = 3
            want = oracle.forward(cfg, w, ids)
            assert (want[-1] - oracle.forward(cfg, w, without)[-1]).abs().max() > 0.2
            for cut in ([T], [T - 2, 2], [T - 1, 1]):
                got = run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"]
                err = (got - want.float()).pow(2).mean(-1).sqrt() / want.std()
                assert err.max() < (3e-5 if dtype == torch.float32 else 0.05), (at, cut, float(err.max()))


@pytest.mark.parametrize("device,dtype", PLACES)
def test_first_tokens_and_token_pairs(device, dtype):
    """The first tokens of a sequence, and a stream that depends on the token before through nothing but the pair's vector."""
    cfg = config([attention(dense(20), heads=2, kv_heads=1, dim=16, vdim=20), latent(None, heads=2, size=1)], width=64)
    w = weights_of(cfg, seed=3)
    w["bigram"] = w["bigram"] * 3
    m = build(cfg, w, device, dtype)
    ids = tokens(40, cfg["vocab"], 4)
    want = oracle.forward(cfg, w, ids)
    blind = copy.deepcopy(cfg)
    blind["embedding"]["bigram"]["mul_prev"] = 0
    assert ((want - oracle.forward(blind, w, ids)).pow(2).mean(-1).sqrt()[1:] > 0.2 * want.std()).double().mean() > 0.8
    replay = TraceReplay(m, 64)
    with torch.inference_mode():
        for cut in ([40], [1] * 8 + [32], [2, 3, 1, 34], [32, 1, 7]):
            got = run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"]
            check(got, want, dtype, str(cut[:3]))
            check(got[:9], want[:9], dtype, str(cut[:3]))


@pytest.mark.parametrize("device,dtype", PLACES)
def test_long_context_and_long_decoding(device, dtype):
    """Hundreds of tokens, windows far behind the sequence's end, most tokens decoded one by one."""
    cfg = config([latent(dense(32), heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=128, size=90), attention(None, heads=2, kv_heads=2, dim=16, vdim=24),
                  latent(dense(32), weights_of=0, heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=128, size=90)], width=64, vocab=128)
    w = weights_of(cfg, seed=4, sharp=3.0)
    m = build(cfg, w, device, dtype)
    T = 600
    ids = tokens(T, 128, 5)
    want = oracle.forward(cfg, w, ids)
    other = oracle.forward(cfg, w, [(ids[0] + 1) % 128] + ids[1:])
    assert (want[-1] - other[-1]).abs().max() > 1e-4             # (a lost key would show)
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
        out = eng.finished[i + 1].output_ids
        assert len(out) == n and oracle.is_greedy(cfg, w, p, out), i
    assert eng.alloc.free_blocks == 15


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
    assert a == b and oracle.is_greedy(cfg, w, p, a[1])


@pytest.mark.parametrize("spec", [0, 3])
def test_shard_serves_portions_prefixes_and_guesses(spec):
    """The shard runtime: a prompt in portions over several Prefill calls, a second request that joins the running batch in one pass and
    starts on cached pages (whose last token it needs), and (spec) guessed tokens that are checked in one pass."""
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
        take(rt.decode(pb.DecodeRequest(batches=[pb.CachedBatch(id=1)])))
        second = req(2, p2, 5, [3, 4]) if spec else req(2, p2, 5, [1, 4], 32)
        r2 = take(rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=2, requests=[second], size=1), decode_batches=[pb.CachedBatch(id=1)])))
        live = [b for b in (r2.batch,) if r2.HasField("batch")]
        for _ in range(20):
            if not live:
                break
            r = take(rt.decode(pb.DecodeRequest(batches=live)))
            live = [r.batch] if r.HasField("batch") else []
    assert len(got[1]) == 9 and oracle.is_greedy(cfg, w, p1, got[1]) and len(got[2]) == 5 and oracle.is_greedy(cfg, w, p2, got[2])


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
    cfg = CONFIGS["odd"]
    w = weights_of(cfg, seed=7)
    save_model(tmp_path, cfg, w)
    rt = build_runtime(str(tmp_path), EngineConfig(max_input_length=40, max_total_tokens=64), device="cpu", source="local")
    assert type(rt) is ShardRuntime and not rt.model.recurrent and len(rt.model.layers) == 8
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
    assert oracle.is_greedy(cfg, w, tokens(17, cfg["vocab"], 2), outs[0][2])


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
