"""The Saredra decoder through the framework (loader, cache and state slots, runner, engine, shard runtime, trace replay) against the
plain float64 statement in `saredra_oracle.py`, on the CPU operators and, marked gpu, on the CUDA kernels in both number formats."""

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import saredra_oracle as oracle
from lorax_b200.config import EngineConfig, ModelConfig
from lorax_b200.models.decoder import DecoderModel
from lorax_b200.models.mixers import RandomWeights, tensor_shapes
from lorax_b200.runtime.trace import TraceReplay
from lorax_b200.utils.weights import InMemoryWeights

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PLACES = [pytest.param("cpu", torch.float32, id="cpu"),
          pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="cuda-fp32"),
          pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="cuda-bf16")]
YARN = dict(factor=4.0, original=60, fast=8.0, slow=0.5)


@pytest.fixture(autouse=True)
def _one_thread():
    """The tensors are small: threads would cost more than they bring."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def dense(ff=44):
    return dict(kind="dense", ff=ff)


def moe(experts=10, top=3, ff=36, groups=(5, 3)):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
    if groups:
        m["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    return m


def heads(heads=6, kv_heads=2, dim=20, vdim=28, size=40, scale=0.3, dims=12, base=300.0, scaling=None, softcap=7.0):
    rot = dict(base=base, dims=dims)
    if scaling:
        rot["scaling"] = scaling
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=softcap, mask=dict(size=size), rot=rot)


def attention(mlp=None, kv_from=None, **kw):
    m = heads(**kw)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mlp=mlp, mixer=m)


def parallel(mlp=None, left=None, conv=3, right=None, scales=(0.7, 1.3)):
    l = dict(heads(**dict(dict(scaling=YARN), **(left or {}))), conv=conv)
    r = dict(heads=6, vdim=12, state=20, groups=3, norm_groups=4, conv=2, **{})
    r.update(right or {})
    return dict(type="parallel", mlp=mlp, mixer=dict(left=l, right=r, left_scale=scales[0], right_scale=scales[1]))


def config(layers, width=76, vocab=150, eps=1e-5):
    return dict(architecture="Saredra", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


CONFIGS = {
    # sizes off every grid, parts of the norm that cut through heads, keys taken from layers in front with other windows, layers without a
    # feed-forward
    "odd": config([attention(), parallel(moe()), attention(dense(), kv_from=0, size=9, scale=0.5, softcap=3.0),
                   parallel(None, left=dict(heads=3, kv_heads=3, dim=70, vdim=9, dims=70, size=33, scale=0.1), conv=6, right=dict(conv=5, norm_groups=1)),
                   attention(moe(experts=7, top=1, groups=None), kv_from=0, size=70)]),
    # everything that can be 1, a window past the sequence, a rotation of one pair, a factor of 1, negative scale
    "plain": config([parallel(moe(experts=4, top=4, groups=(1, 1), ff=20), left=dict(heads=1, kv_heads=1, dim=16, vdim=16, dims=2, size=1000, scaling=dict(YARN, factor=1.0)),
                              conv=1, right=dict(heads=1, vdim=1, state=1, groups=1, norm_groups=1, conv=1), scales=(1.0, 1.0)),
                     parallel(moe(experts=6, top=2, groups=(6, 2)), left=dict(heads=2, kv_heads=1, dim=8, vdim=24, dims=8, size=1, scaling=None, scale=-0.4),
                              conv=2, right=dict(heads=5, vdim=3, state=7, groups=5, norm_groups=5, conv=3), scales=(-0.5, 0.25)),
                     attention(dense(30), heads=2, kv_heads=2, dim=24, vdim=24, size=32, dims=6)], width=100, eps=3e-4),
    # sizes of the tensor-core kernels, many experts
    "aligned": config([parallel(moe(experts=40, top=6, ff=128, groups=(8, 3)), left=dict(heads=4, kv_heads=2, dim=128, vdim=128, dims=64, size=70, scale=0.09),
                                conv=4, right=dict(heads=4, vdim=64, state=128, groups=2, norm_groups=2, conv=4)),
                       attention(dense(256), heads=16, kv_heads=1, dim=128, vdim=120, size=31, scale=0.09, dims=128),
                       attention(moe(experts=16, top=2, groups=(4, 2), ff=64), kv_from=1, heads=4, kv_heads=1, dim=128, vdim=120, size=150, dims=128),
                       parallel(None, left=dict(heads=34, kv_heads=2, dim=64, vdim=128, size=128, scale=0.12, dims=32),
                                right=dict(heads=2, vdim=128, state=64, groups=1, norm_groups=8, conv=4))], width=256, vocab=320),
}


def weights_of(cfg, seed=0, sharp=2.5, slow=2.0):
    """Random weights, rounded to bf16.  Queries are scaled so that single keys stand out, decays slowed so that states reach far."""
    rw = RandomWeights(ModelConfig.from_dict(cfg), "cpu", seed)
    out = {}
    for n in rw.shapes:
        t = rw.get_tensor(n)
        if n.endswith("mix.q") or n.endswith("left.q"):
            t = t * sharp
        if n.endswith("A_log"):
            t = t - slow
        if n.endswith("router"):
            t = t * 2
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
    assert c.model_type == "saredra" and c.layer_style == "pre" and c.hidden_act == "silu" and c.norm_type == "rms"
    m = c.layer_specs[1].moe
    assert (m.experts, m.top, m.ff, m.groups, m.keep, m.score, m.renorm, m.group_top, m.gated, m.shared_ff) == (10, 3, 36, 5, 3, "softmax", False, 1, True, 0)
    assert c.num_attention_heads == 6 and c.num_key_value_heads == 3 and c.head_dim == 70
    shapes = tensor_shapes(c)
    assert shapes["l0.mix.q"] == (120, 76) and shapes["l0.mix.v"] == (56, 76) and shapes["l0.mix.o"] == (76, 168) and shapes["l0.mix.g"] == (168, 76)
    assert shapes["l1.mix.left.k.b"] == (40,) and shapes["l1.mix.left.v.conv"] == (56, 3) and shapes["l1.mix.left.sink"] == (6,)
    assert shapes["l1.mix.right.in"] == (72 + 72 + 120 + 6, 76) and shapes["l1.mix.right.conv"] == (192, 2) and shapes["l1.mix.right.conv.b"] == (192,)
    assert shapes["l1.mix.right.norm"] == (72,) and shapes["l1.mix.right.o"] == (76, 72) and shapes["l1.mlp.e9.gate"] == (36, 76)
    for absent in ("l0.norm2", "l0.mix.q.b", "l0.mix.sink", "l1.mix.left.g", "l2.mix.k", "l4.mix.v", "l1.mlp.correction", "l3.mlp.up", "pos", "final.norm.b"):
        assert absent not in shapes, absent
    for bad in (moe(groups=(3, 1)), moe(top=11), moe(groups=(5, 1)), moe(groups=(5, 6))):
        with pytest.raises(ValueError):
            ModelConfig.from_dict(config([attention(bad)]))
    build_ = lambda layers: DecoderModel.random_init(ModelConfig.from_dict(config(layers)), "cpu", torch.float32)
    for bad in ([attention(heads=5)], [attention(size=0)], [attention(dims=22)], [attention(dims=3)], [attention(kv_from=0)], [attention(kv_from=1), attention()],
                [attention(), attention(kv_from=0), attention(kv_from=1)], [attention(), attention(kv_from=0, kv_heads=3)],
                [parallel(right=dict(groups=4))], [parallel(right=dict(norm_groups=5))]):
        with pytest.raises(ValueError):
            build_(bad)
    for bad in ([attention(dim=257)], [parallel(conv=10)], [parallel(right=dict(state=300))], [dict(attention(), type="other")], [attention(dict(kind="other"))]):
        with pytest.raises(NotImplementedError):
            build_(bad)


def test_keys_of_another_layer_take_no_memory():
    from lorax_b200.runtime.kv_cache import cache_bytes, make_cache
    m = DecoderModel.random_init(ModelConfig.from_dict(CONFIGS["odd"]), "cpu", torch.float32)
    kv = make_cache(m, EngineConfig(), 4, 2)
    assert kv.layers[2] is kv.layers[0] and kv.layers[4] is kv.layers[0] and kv.layers[1]["left"]["kv"] is not kv.layers[0]
    slots = kv.state_slots.num_slots
    assert kv.layers[1]["left"]["conv"].shape == (slots, 2, (6 + 2) * 64 + 2 * 64) and kv.layers[1]["right"]["conv"].shape == (slots, 1, 6 * 16 + 2 * 3 * 32)
    per_block, fixed = cache_bytes(m, EngineConfig(), 2)
    every = []

    def walk(x):
        for t in (x.values() if isinstance(x, dict) else [x]):
            walk(t) if isinstance(t, dict) else every.append(t)
    for entry in kv.layers:
        walk(entry)
    unique = {t.data_ptr(): t for t in every if t.numel()}.values()
    assert sum(t.numel() * t.element_size() for t in unique) == per_block * 4 + fixed


def test_what_the_design_does_not_offer_is_refused():
    from lorax_b200.server.runtime import ShardRuntime
    m = DecoderModel.random_init(ModelConfig.from_dict(CONFIGS["odd"]), "cpu", torch.float32, max_positions=500)
    assert m.recurrent
    with pytest.raises(ValueError):
        m.quantize("fp8")
    for kw in (dict(kv_cache_dtype="fp8"), dict(prefix_caching=True), dict(speculative_tokens=2), dict(max_total_tokens=501)):
        with pytest.raises(ValueError):
            ShardRuntime(m, None, EngineConfig(**dict(dict(max_total_tokens=100), **kw)), num_blocks=32, max_batch=2)
    only = DecoderModel.random_init(ModelConfig.from_dict(config([attention(), attention(kv_from=0)])), "cpu", torch.float32)
    assert not only.recurrent
    ShardRuntime(only, None, EngineConfig(max_total_tokens=100, prefix_caching=True), num_blocks=16, max_batch=2)


# ---------------------------------------------------------------------------------------------- mechanisms alone
def step_of(n, before=0):
    from test_mixers_gpu import make_step
    return make_step([], [(before, n)])


@pytest.mark.parametrize("H,G,d,dv,size,cap,sharp", [(4, 2, 16, 8, 5, 3.0, 1), (3, 3, 8, 24, 1, 50.0, 30), (4, 1, 8, 8, 100, 2.0, 5), (2, 1, 8, 8, 64, 0.0, 1)])
def test_attention_with_caps_sinks_and_gates(H, G, d, dv, size, cap, sharp):
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(size)
    T = 70
    x = torch.randn(T, (H + G) * d + G * dv, generator=g) * sharp
    gate, sink = torch.randn(T, H * dv, generator=g) * 3, torch.randn(H, generator=g) * 4
    f = x.double()
    want = oracle.attend(f[:, : H * d].view(T, H, d), f[:, H * d: (H + G) * d].view(T, G, d), f[:, (H + G) * d:].view(T, G, dv), 0.37, size, cap, sink.double())
    want = (want * 1.7).reshape(T, -1) * oracle.sigmoid(gate.double())
    inp, nb, _ = step_of(T)
    cache, out = torch.zeros(nb, G, 32 * (d + dv)), torch.empty(T, H * dv)
    q = ref.conv_rope_kvwrite(x, H, G, d, dv, None, 0, inp.positions, cache, inp)
    ref.gqa_attn(q, cache, H, G, d, dv, 0.37, size, inp, out, softcap=cap, sink=sink, gate=gate, out_scale=1.7)
    assert torch.allclose(out.double(), want, atol=1e-4 * sharp)


@pytest.mark.parametrize("rot", [dict(base=700.0, dims=10), dict(base=50.0, dims=16, scaling=YARN), dict(base=5e4, dims=2, scaling=dict(YARN, factor=32.0)),
                                 dict(base=9.0, dims=12, scaling=dict(factor=3.0, original=4000, fast=32.0, slow=1.0)),
                                 dict(base=1e4, dims=8, scaling=dict(factor=2.0, original=100, fast=1.0, slow=1.0))])
def test_rotation(rot):
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(1)
    H, G, d, T, first = 3, 1, 16, 40, 900
    x = torch.randn(T, (H + G) * d + G * d, generator=g)
    inp, nb, _ = step_of(T, first)
    want = oracle.rotate(x[:, : (H + G) * d].double().view(T, H + G, d), rot, first)
    table = ref.rope_table(rot["dims"], 1000, rot["base"], scaling=rot.get("scaling"))
    cache = torch.zeros(nb, G, 32 * 2 * d)
    q = ref.conv_rope_kvwrite(x, H, G, d, d, table, rot["dims"], inp.positions, cache, inp)
    k, _ = ref._kv_planes(cache, inp.block_tables[0, : (first + T + 31) // 32], d, d, first + T)
    assert torch.allclose(q.double().view(T, H, d), want[:, :H], atol=1e-4) and torch.allclose(k[first:].double(), want[:, H:], atol=1e-4)


@pytest.mark.parametrize("taps", [1, 2, 4, 9])
def test_short_convolutions_carry_their_rows(taps):
    """In portions shorter and longer than the taps, over a state that holds another request's rows."""
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(taps)
    T, C = 23, 8
    u, w, b = torch.randn(T, C, generator=g), torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    want = oracle.silu(oracle.causal_conv(u.double(), w.double(), b.double()))
    for cut in ([T], [1] * T, [2, 1, 7, 13]):
        state, out, at = torch.randn(3, taps - 1, C, generator=g), [], 0
        for n in cut:
            inp, _, _ = step_of(n, at)
            inp.state_slots[:] = 2
            out.append(ref.causal_conv(u[at: at + n], w.t(), b, "silu", state, inp))
            at += n
        assert torch.allclose(torch.cat(out).double(), want, atol=1e-5)


@pytest.mark.parametrize("H,P,N,G,parts", [(6, 12, 20, 3, 4), (1, 1, 1, 1, 1), (4, 8, 5, 1, 2), (3, 7, 16, 3, 7)])
def test_state_space_recurrence_and_gated_norm(H, P, N, G, parts):
    """Large and tiny step sizes, through the mixer itself."""
    from lorax_b200.models.mixers import Mamba2Mixer
    g = torch.Generator().manual_seed(H)
    p = dict(heads=H, vdim=P, state=N, groups=G, norm_groups=parts, conv=3)
    mx, T, width = Mamba2Mixer(dict(p, out_scale=0.6), 24), 50, 24
    W = {n: torch.randn(*s, generator=g) for n, s in mx.shapes().items()}
    W["dt_bias"] = torch.linspace(-12.0, 6.0, H)
    W["in"][-H:] *= 4
    h = torch.randn(T, width, generator=g)
    want = 0.6 * oracle.mamba2(h.double(), {k: v.double() for k, v in W.items()}, "", p, 1e-3)

    class Model:
        from lorax_b200.ops import reference as ops
        eps, dtype = 1e-3, torch.float32
    mx.load(lambda n: W[n], lambda t: t, lambda t: t.contiguous(), Model)
    proj = {n: torch.nn.functional.pad(h, (0, mx.W - width)) @ t.t() for n, t in mx.in_parts(lambda n: W[n])}
    cache = {n: torch.randn(3, *dims) for n, (dims, _) in mx.cache_shape(Model)["state"].items()}
    y = torch.empty(T, mx.out_dim)
    at = 0
    for n in (1, 30, 2, 17):
        inp, _, _ = step_of(n, at)
        inp.state_slots[:] = 1
        mx.run(Model, None, {k: v[at: at + n] for k, v in proj.items()}, y[at: at + n], inp, cache)
        at += n
    assert torch.allclose(y[:, : H * P].double(), want, atol=2e-4) and not y[:, H * P:].any()


@pytest.mark.parametrize("E,top,groups", [(12, 3, (4, 2)), (12, 4, (12, 5)), (9, 2, None), (8, 8, (1, 1)), (6, 1, (2, 1))])
def test_routing(E, top, groups):
    """Groups by their largest score, weights that do not sum to one."""
    from lorax_b200.ops import reference as ref
    g = torch.Generator().manual_seed(E)
    T = 50
    x, wr = torch.randn(T, 24, generator=g), torch.randn(E, 24, generator=g) * 0.5
    router = dict(top=top, experts=E)
    if groups:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    ids, w = oracle.route(x.double() @ wr.double().t(), router)
    r = ref.moe_route(x, wr, top, 0, E, experts=E, score="softmax", groups=groups[0] if groups else 0, keep=groups[1] if groups else 0, group_top=1,
                      renorm=False)
    full = lambda i, v: torch.zeros(T, E).scatter_(1, i.long(), v.float())
    assert torch.allclose(full(r.topk_ids, r.topk_w), full(ids, w), atol=1e-6) and (top == E or float(w.sum(-1).min()) < 0.9)


def test_feed_forwards():
    from lorax_b200.models.mixers import DenseMlp, MoeMlp
    for mlp in (moe(), moe(ff=70, groups=None), dense(20)):
        cfg = config([attention(mlp)], width=48)
        w = weights_of(cfg, seed=3)
        c = ModelConfig.from_dict(cfg)
        m = DecoderModel(c, "cpu", torch.float32)
        spec = c.layer_specs[0]
        mod = MoeMlp(spec.moe, 48) if spec.moe else DenseMlp(spec.ff, 48, spec.gated)
        mod.load(lambda n: w["l0.mlp." + n].float(), lambda t: t, lambda t: t, m)
        x = torch.randn(9, 48, generator=torch.Generator().manual_seed(1))
        rows, pairs = mod.run(m, x)
        W = {k: v.double() for k, v in w.items()}
        if pairs is None:
            got, want = rows, oracle.feed_forward(x.double(), W, "l0.mlp.")
        else:
            got, want = (rows[pairs[0].long()][:, :, :48] * pairs[1][:, :, None]).sum(1), oracle.mixture(x.double(), W, "l0.mlp.", mlp)
            assert not rows[:, 48:].any()
        assert torch.allclose(got.double(), want, atol=1e-5)


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
    """Prompts of unequal length beside decode rows, requests that sit out steps, pages and slots handed on: every request against its own
    run alone.  The pool holds little more than what is live."""
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
    """One layer in which the query of token 1 singles out the key of token 2: queries read the first half of the stream, keys the second
    half with the same matrix, and token 1 has in its first half what token 2 has in its second.  The rotated dimensions are left out, the
    convolutions pass their input on, a mixer beside the attention is silent."""
    kw = dict(heads=2, kv_heads=1, dim=dim, vdim=vdim, size=size, scale=1.0, dims=4, softcap=20.0)
    cfg = config([attention(**kw) if kind == "attention" else parallel(left=kw)], width=width, vocab=40)
    w = {k: v.float() for k, v in weights_of(cfg, seed=size, sharp=1.0).items()}
    g = torch.Generator().manual_seed(size)
    half, p = width // 2, "l0.mix." if kind == "attention" else "l0.mix.left."
    u = 3.0 * torch.randn(half, generator=g)
    w["embed"] *= 0.3
    w["embed"][1, :half], w["embed"][2, half:] = u, u
    q, k = torch.randn(2, dim, width, generator=g) * (16.0 / dim) ** 0.5 * width ** -0.5, torch.zeros(dim, width)
    q[1] = q[0]
    q[:, :4], q[:, :, half:] = 0, 0
    k[:, half:] = q[0, :, :half]
    w[p + "q"], w[p + "k"] = q.reshape(2 * dim, width), k
    for n in [n for n in w if n.startswith(p) and n.endswith(".b")]:
        w[n] *= 0
    for n in [n for n in w if n.startswith(p) and n.endswith(".conv")]:
        w[n] = torch.zeros_like(w[n])
        w[n][:, -1] = 1
    if kind != "attention":
        w["l0.mix.right.o"] *= 0
    return cfg, {k: t.to(torch.bfloat16) for k, t in w.items()}


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("kind,size,dim,vdim", [("attention", 40, 24, 24), ("parallel", 64, 128, 128), ("attention", 33, 20, 70), ("parallel", 300, 16, 16)])
def test_keys_just_inside_and_outside_the_window(kind, size, dim, vdim, device, dtype):
    """A key that its query singles out, at the last place that the window holds, the next one, and at page borders; the query in a
    prompt, in a portion and decoded.  That the key decides is checked on the plain statement."""
    cfg, w = edge_model(kind, size, dim, vdim)
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
                for cut in ([T], [T - 2, 2] if T > 2 else [T], [T - 1, 1]):
                    got = run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"]
                    err = (got - want.float()).pow(2).mean(-1).sqrt() / want.std()
                    assert err.max() < (3e-5 if dtype == torch.float32 else 0.05), (at, back, cut, float(err.max()))


@pytest.mark.parametrize("device,dtype", PLACES)
def test_sinks_capped_scores_and_first_tokens(device, dtype):
    """Sinks far above and below the scores, scores far beyond their cap, the first tokens of a sequence."""
    cfg = config([parallel(dense(20), left=dict(heads=4, kv_heads=2, dim=16, vdim=16, size=50, softcap=2.0)),
                  attention(None, heads=2, kv_heads=1, dim=16, vdim=20, softcap=45.0)], width=64)
    w = weights_of(cfg, seed=3, sharp=30.0)
    w["l0.mix.left.sink"] = torch.tensor([12.0, -40.0, 0.0, 3.0], dtype=torch.bfloat16)
    quiet = dict(w)
    quiet["l0.mix.left.sink"] = torch.full((4,), -1e4, dtype=torch.bfloat16)
    m = build(cfg, w, device, dtype)
    ids = tokens(90, cfg["vocab"], 4)
    want = oracle.forward(cfg, w, ids)
    assert ((want - oracle.forward(cfg, quiet, ids)).pow(2).mean(-1).sqrt() > 0.02 * want.std()).all()
    uncapped = copy.deepcopy(cfg)
    uncapped["layers"][0]["mixer"]["left"]["softcap"] = 0
    assert ((want - oracle.forward(uncapped, w, ids)).pow(2).mean(-1).sqrt()[1:] > 0.05 * want.std()).double().mean() > 0.8
    replay = TraceReplay(m, 128)
    with torch.inference_mode():
        for cut in ([90], [1] * 8 + [82], [2, 3, 1, 84]):
            check(run_trace(replay, {"x": ids}, [[("x", n)] for n in cut])["x"], want, dtype, str(cut[:3]))


@pytest.mark.parametrize("device,dtype", PLACES)
def test_long_context_and_long_decoding(device, dtype):
    """Hundreds of tokens with windows far behind the sequence's end and states that remember its beginning, most tokens decoded one by one."""
    cfg = config([parallel(dense(32), left=dict(heads=2, kv_heads=1, dim=16, vdim=16, size=90), right=dict(heads=2, vdim=64, state=64, groups=1, norm_groups=2)),
                  attention(None, heads=2, kv_heads=2, dim=16, vdim=24, size=257), attention(None, kv_from=1, heads=4, kv_heads=2, dim=16, vdim=24, size=31)],
                 width=64, vocab=128)
    w = weights_of(cfg, seed=4, sharp=4.0, slow=5.0)
    m = build(cfg, w, device, dtype)
    T = 600
    ids = tokens(T, 128, 5)
    want = oracle.forward(cfg, w, ids)
    other = oracle.forward(cfg, w, [(ids[0] + 1) % 128] + ids[1:])
    assert (want[-1] - other[-1]).abs().max() > 1e-3             # (a lost state would show)
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
    assert eng.alloc.free_blocks == 15 and len(eng.kv.state_slots.free) == eng.kv.state_slots.num_slots - 1


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


def test_shard_serves_portions_of_prompts_and_fused_steps():
    """The shard runtime: a prompt in portions over several Prefill calls, and a second request that joins the running batch in one pass."""
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
    p1, p2 = tokens(50, cfg["vocab"], 1), tokens(41, cfg["vocab"], 2)
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
        r2 = take(rt.prefill(pb.PrefillRequest(batch=pb.Batch(id=2, requests=[req(2, p2, 5, [3, 4])], size=1), decode_batches=[pb.CachedBatch(id=1)])))
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
    cfg = CONFIGS["plain"]
    w = weights_of(cfg, seed=7)
    save_model(tmp_path, cfg, w)
    rt = build_runtime(str(tmp_path), EngineConfig(max_input_length=40, max_total_tokens=64), device="cpu", source="local")
    assert type(rt) is ShardRuntime and rt.model.recurrent and len(rt.model.layers) == 3
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
