"""Kernels of the layer-by-layer designs against the PyTorch statement of the same operator (`ops.reference`), in bf16 and in fp32."""

import pytest
import torch

pytestmark = pytest.mark.gpu
PAGE = 32
DTYPES = (torch.bfloat16, torch.float32)


def make_step(dec, pre, slots=None, seg_len=64, seed=0, pages_per_seq=None, windows=(0,)):
    """StepInputs (on the CPU) of decode rows with contexts `dec` and prompt portions `pre` = [(tokens before, tokens)], over shuffled
    pages and state slots.  -> (inp, number of blocks, number of state slots)"""
    from lorax_b200.models.decoder import StepInputs
    from lorax_b200.ops import reference
    g = torch.Generator().manual_seed(seed)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    spans = [(max(c - 1, 0), 1) for c in dec] + list(pre)
    width = pages_per_seq or max((b + n + PAGE - 1) // PAGE for b, n in spans) + 1
    blocks = (1 + torch.randperm(width * len(spans), generator=g)).view(len(spans), width).to(torch.int32)
    sl = (1 + torch.randperm(len(spans), generator=g)).to(torch.int32)
    nd = len(dec)
    pos, slot = [], []
    for i, (b, n) in enumerate(spans):
        for t in range(b, b + n):
            pos.append(t)
            dead = i < nd and dec[i] <= 0
            slot.append(-1 if dead else int(blocks[i, t // PAGE]) * PAGE + t % PAGE)
    T = len(pos)
    kw = dict(input_ids=torch.zeros(T, dtype=torch.int32), positions=i32(pos), slots=i32(slot))
    if not pre:
        inp = StepInputs(is_prefill=False, block_tables=blocks, ctx_lens=i32(dec), state_slots=sl, **kw)
    else:
        q = [n for _, n in pre]
        cu = [0]
        for _, n in pre:
            cu.append(cu[-1] + n)
        contexts = {w: reference.context_offsets([b for b, _ in pre], q, w) for w in windows}
        ss, s0 = reference.prefill_tiles(q, seg_len)
        ts, t0 = reference.prefill_tiles(q, 128)
        t64s, t64q = reference.prefill_tiles(q)
        inp = StepInputs(is_prefill=True, block_tables=blocks[nd:].contiguous(), cu_q=i32(cu), cache_lens=i32([b for b, _ in pre]),
                         state_slots=sl[nd:].contiguous(), n_decode=nd, dec_block_tables=blocks[:nd].contiguous(), ctx_lens=i32(dec),
                         dec_state_slots=sl[:nd].contiguous(), seg_seq=i32(ss), seg_q0=i32(s0), seg_len=seg_len, q128_seq=i32(ts),
                         q128_q0=i32(t0), tile_seq=i32(t64s), tile_q0=i32(t64q), contexts={w: (i32(o), o[-1]) for w, o in contexts.items()}, **kw)
    return inp, width * len(spans) + 1, len(spans) + 1


def to_dev(x):
    import dataclasses
    if isinstance(x, torch.Tensor):
        return x.cuda()
    moved = {f.name: getattr(x, f.name).cuda() for f in dataclasses.fields(x) if isinstance(getattr(x, f.name), torch.Tensor)}
    if x.contexts is not None:
        moved["contexts"] = {w: (t.cuda(), n) for w, (t, n) in x.contexts.items()}
    return dataclasses.replace(x, **moved)


def close(got, want, dtype, rows=None, tol16=2e-2, tol32=2e-5):
    got, want = got.float().cpu(), want.float()
    if rows is not None:
        got, want = got[rows], want[rows]
    assert torch.isfinite(got).all()
    err = (got - want).norm() / want.norm().clamp_min(1e-6)
    worst = (got - want).abs().max() / want.abs().max().clamp_min(1e-6)
    tol = tol32 if dtype == torch.float32 else tol16
    assert err < tol and worst < 4 * tol, (float(err), float(worst))


STEPS = {
    "decode": ([1, 2, 33, 0, 700], []),
    "prompts": ([], [(0, 1), (0, 64), (0, 65), (0, 300), (31, 2), (64, 130)]),
    "mixed": ([5, 0, 64, 1], [(0, 129), (70, 3), (200, 64), (1, 2)]),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS))
@pytest.mark.parametrize("H,d,dv", [(3, 16, 48), (2, 64, 32), (4, 128, 128), (3, 64, 64), (2, 128, 192), (1, 256, 80), (2, 48, 144)])
def test_linear_attention_recurrence(dtype, step, H, d, dv):
    from lorax_b200.ops import native, reference
    inp, _, ns = make_step(*STEPS[step])
    T = inp.positions.shape[0]
    g = torch.Generator().manual_seed(1)
    x = torch.randn(T, H * (2 * d + dv), generator=g).to(dtype)
    decay = torch.linspace(0.3, 0.9995, H)
    if H > 2:
        decay[0], decay[1] = 0.0, 1.0
    state = torch.randn(ns, H, d, dv, generator=g)
    q, k, v = x[:, : H * d], x[:, H * d: 2 * H * d], x[:, 2 * H * d:]
    st = state.clone()
    want = reference.linear_attn(q.float(), k.float(), v.float(), H, d, dv, decay, st, inp)
    xd, sd = x.cuda(), state.cuda()
    got = native.linear_attn(xd[:, : H * d], xd[:, H * d: 2 * H * d], xd[:, 2 * H * d:], H, d, dv, decay.cuda(), sd, to_dev(inp))
    live = [i for i in range(T) if i >= len(STEPS[step][0]) or STEPS[step][0][i] > 0]
    close(got, want, dtype, live, tol16=6e-3)
    close(sd, st, dtype, tol16=6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS))
@pytest.mark.parametrize("H,d,strong", [(3, 16, False), (2, 64, False), (2, 64, True), (1, 128, False), (2, 80, True), (1, 256, False)])
def test_wkv_recurrence(dtype, step, H, d, strong):
    """`strong`: decays so strong (and so weak) that products over a few tokens under- and overflow unless they are formed safely."""
    from lorax_b200.ops import native, reference
    inp, _, ns = make_step(*STEPS[step], seed=3)
    T, C = inp.positions.shape[0], H * d
    g = torch.Generator().manual_seed(2)
    r, k, v, z = (torch.randn(T, C, generator=g).to(dtype) for _ in range(4))
    w0 = torch.randn(C, generator=g) * (3.0 if strong else 1.0) + (1.0 if strong else -2.0)
    u = torch.randn(C, generator=g)
    state = torch.randn(ns, H, d, d, generator=g)
    st = state.clone()
    want = reference.wkv(r.float(), k.float(), v.float(), z.float(), w0, u, H, d, st, inp)
    sd = state.cuda()
    got = native.wkv(r.cuda(), k.cuda(), v.cuda(), z.cuda(), w0.cuda(), u.cuda(), H, d, sd, to_dev(inp))
    live = [i for i in range(T) if i >= len(STEPS[step][0]) or STEPS[step][0][i] > 0]
    close(got, want, dtype, live, tol16=2e-4)
    close(sd, st, dtype, tol16=2e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS))
def test_token_shift(dtype, step):
    from lorax_b200.ops import native, reference
    inp, _, ns = make_step(*STEPS[step], seed=4)
    T, W = inp.positions.shape[0], 112
    g = torch.Generator().manual_seed(2)
    h, mu, shift = torch.randn(T, W, generator=g).to(dtype), torch.rand(5, W, generator=g), torch.randn(ns, W, generator=g).to(dtype)
    sh = shift.clone()
    want = reference.token_shift(h, mu, sh, inp)
    sd = shift.cuda()
    got = native.token_shift(h.cuda(), mu.cuda(), sd, to_dev(inp))
    live = [i for i in range(T) if i >= len(STEPS[step][0]) or STEPS[step][0][i] > 0]
    assert torch.equal(sd.cpu(), sh)
    assert torch.allclose(got.cpu().float()[:, live], want.float()[:, live], atol=2e-2 if dtype == torch.bfloat16 else 1e-6)


def latent_case(H, dk, rot, dv, kv, inp, nb, dtype, peak, seed=5):
    """Random queries, cache and expansion weights.  `peak`: every query matches one far key of its own context far better than all
    others, so a key that is lost or misplaced shows."""
    g = torch.Generator().manual_seed(seed)
    T = inp.positions.shape[0]
    q = torch.randn(T, H * (dk + rot), generator=g).to(dtype)
    cache = torch.randn(nb, PAGE, kv + rot, generator=g).to(dtype)
    uk, uv = torch.randn(H, dk, kv, generator=g) * kv ** -0.5, torch.randn(H, dv, kv, generator=g) * kv ** -0.5
    if peak:
        nd, dbt, _, ctx = inp.decode_view(T)
        for t in range(T):
            if t < nd:
                bt, keys = dbt[t], int(ctx[t])
            else:
                b = int(torch.searchsorted(inp.cu_q[1:], torch.tensor(t - nd), right=True))
                bt, keys = inp.block_tables[b], int(inp.cache_lens[b]) + (t - nd - int(inp.cu_q[b])) + 1
            if keys <= 0:
                continue
            j = (0, keys - 1, keys // 3, keys // 32 * 32, max(keys // 32 * 32 - 1, 0))[t % 5]
            j = min(j, keys - 1)
            kr = cache[int(bt[j // PAGE]), j % PAGE, kv:].float()
            q.view(T, H, dk + rot)[t, :, dk:] = (kr * 2.0).to(dtype)
    return q, cache, uk.to(dtype), uv.to(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("peak", [False, True])
@pytest.mark.parametrize("step", list(STEPS) + ["long"])
@pytest.mark.parametrize("H,dk,rot,dv,kv", [(3, 32, 16, 48, 80), (2, 128, 64, 128, 512), (5, 64, 64, 64, 256), (17, 64, 64, 128, 128)])
def test_latent_attention(dtype, peak, step, H, dk, rot, dv, kv):
    """Absorbed and expanded form, decode rows, portions and whole prompts: gated outputs against the fp32 statement."""
    from lorax_b200.ops import native, reference
    dec, pre = STEPS[step] if step in STEPS else ([1000, 1500], [(1000, 300), (0, 500), (129, 40)])
    inp, nb, _ = make_step(dec, pre, seed=6)
    T = inp.positions.shape[0]
    q, cache, uk, uv = latent_case(H, dk, rot, dv, kv, inp, nb, dtype, peak)
    gate = torch.randn(T, 32, generator=torch.Generator().manual_seed(9)).to(dtype)
    scale = (dk + rot) ** -0.5
    head = dk + rot
    ql = torch.empty(T, H * kv)
    reference.gemm_heads(q.float(), uk.float().transpose(1, 2).contiguous(), ql, head)
    o = reference.latent_attn(ql, q.float(), cache.float(), H, kv, head, dk, rot, scale, inp)
    want = torch.zeros(T, H * dv)
    reference.gemm_heads(o, uv.float(), want, kv, gate=gate.float())
    live = [i for i in range(T) if i >= len(dec) or dec[i] > 0]

    d = to_dev(inp)
    qd, cd, gd = q.cuda(), cache.cuda(), gate.cuda()
    qld = torch.empty(T, H * kv, dtype=dtype, device="cuda")
    native.gemm_heads(qd, uk.transpose(1, 2).contiguous().cuda(), qld, head)
    od = native.latent_attn(qld, qd, cd, H, kv, head, dk, rot, scale, d)
    got = torch.zeros(T, H * dv, dtype=dtype, device="cuda")
    native.gemm_heads(od, uv.cuda(), got, kv, gate=gd)
    close(got, want, dtype, live)
    if pre:
        ukv = torch.cat([uk, uv], 1).reshape(H * (dk + dv), kv).contiguous().cuda()
        out = torch.zeros(T, H * dv, dtype=dtype, device="cuda")
        if native.latent_prefill(qd, cd, ukv, gd, out, H, dk, rot, dv, scale, d, len(dec)):
            native.workspace(out.device).check_status()
            close(out, want, dtype, list(range(len(dec), T)))


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_preparation_and_rotation(dtype):
    from lorax_b200.ops import native, reference
    inp, nb, _ = make_step([7, 0, 40], [(0, 50), (33, 5)], seed=8)
    T = inp.positions.shape[0]
    g = torch.Generator().manual_seed(3)
    qr, kr, rot, rp, H, dk = 96, 80, 10, 16, 3, 32
    x = torch.randn(T, qr + kr + rp, generator=g).to(dtype)
    qn, kn = torch.rand(qr, generator=g) + 0.5, torch.rand(kr, generator=g) + 0.5
    cs = reference.rope_table(rot, 128, 10000.0)
    cache = torch.zeros(nb, PAGE, kr + rp)
    want = reference.latent_prep(x[:, :qr].float(), x[:, qr:].float(), qn, kn, 90, 75, rot, 1e-5, cs, inp.positions, inp.slots, cache)
    xd, cd = x.cuda(), torch.zeros(nb, PAGE, kr + rp, dtype=dtype, device="cuda")
    got = native.latent_prep(xd[:, :qr], xd[:, qr:], qn.cuda(), kn.cuda(), 90, 75, rot, 1e-5, cs.cuda(), inp.positions.cuda(), inp.slots.cuda(), cd)
    close(got, want, dtype, tol16=5e-3)
    close(cd, cache, dtype, tol16=5e-3)
    q = torch.randn(T, H * (dk + rp), generator=g).to(dtype)
    qf, qd = q.float(), q.cuda()
    reference.rope_pairs(qf, inp.positions, cs, H, dk + rp, dk, rot)
    native.rope_pairs(qd, inp.positions.cuda(), cs.cuda(), H, dk + rp, dk, rot)
    close(qd, qf, dtype, tol16=5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,n", [(1, 16, 9), (5, 208, 200), (67, 4096, 4096), (3, 5120, 5100)])
def test_stream_norms_and_products(dtype, T, W, n):
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T)
    res, pend, w = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g).to(dtype), torch.randn(W, generator=g) * 0.2
    rd, rf = res.cuda(), res.clone()
    for p in (None, pend):
        want = reference.norm_stream(rf, None if p is None else p.float(), w, 1e-5, 1.0, n, torch.float32)
        got = native.norm_stream(rd, None if p is None else p.cuda(), w.cuda(), 1e-5, 1.0, n, dtype)
        close(got, want, dtype, tol16=4e-3)
        assert torch.allclose(rd.cpu(), rf, atol=1e-6)              # the stream itself stays fp32
    table = torch.randn(50, W, generator=g).to(dtype)
    ids = torch.randint(0, 50, (T,), generator=g, dtype=torch.int32)
    assert torch.equal(native.embed_stream(ids.cuda(), table.cuda(), 0.75).cpu(), reference.embed_stream(ids, table, 0.75))
    for group, act in ((16, "silu"), (W, "sigmoid")):
        x, gate = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g).to(dtype)
        out = torch.zeros(T, W + 16, dtype=dtype, device="cuda")
        want = reference.norm_gate(x, group, group - 3, w, gate.float(), act, 1e-5, torch.zeros(T, W))
        native.norm_gate(x.cuda(), group, group - 3, w.cuda(), gate.cuda(), act, 1e-5, out[:, :W])
        close(out[:, :W], want, dtype, tol16=4e-3)
        assert not out[:, W:].any()


@pytest.mark.parametrize("T,N,K", [(1, 640, 192), (7, 48, 16), (130, 200, 96)])
def test_32_bit_products_and_head(T, N, K):
    """The fp32 operators: no reduced-precision multiply anywhere."""
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T)
    x, w = torch.randn(T, K, generator=g), torch.randn(N, K, generator=g)
    want = (x.double() @ w.double().t()).float()
    close(native.gemm(x.cuda(), w.cuda()), want, torch.float32, tol32=2e-6)
    inter = N // 2 // 4 * 4
    close(native.act_mul(want.cuda(), inter, "gelu_tanh"), reference.act_mul(want, inter, "gelu_tanh"), torch.float32, tol32=2e-6)
    ids, lps = native.argmax_logprob(want.cuda())
    ri, rl = reference.argmax_logprob(want)
    assert torch.equal(ids.cpu(), ri) and torch.allclose(lps.cpu(), rl, atol=1e-4)
    t = torch.randn(8, 16, generator=g)
    assert torch.allclose(native.tanh_(t.cuda()).cpu(), torch.tanh(t), atol=1e-6)


# ---------------------------------------------------------------------------------------------- grouped-query attention
def gqa_case(H, G, dk, dv, window, inp, nb, dtype, peak, seed=11):
    """Random queries over a random cache.  `peak`: every query matches one key of its own context far better than all others: the
    oldest that the window holds, the newest that it does not, the first token, itself, one at a page's edge, in turn."""
    g = torch.Generator().manual_seed(seed)
    T = inp.positions.shape[0]
    q = torch.randn(T, H * dk, generator=g).to(dtype)
    cache = torch.randn(nb, G, PAGE * (dk + dv), generator=g).to(dtype)
    if peak:
        nd, dbt, _, ctx = inp.decode_view(T)
        keys = cache[:, :, : PAGE * dk].view(nb, G, PAGE, dk).float()
        for t in range(T):
            if t < nd:
                bt, n = dbt[t], int(ctx[t])
            else:
                b = int(torch.searchsorted(inp.cu_q[1:], torch.tensor(t - nd), right=True))
                bt, n = inp.block_tables[b], int(inp.cache_lens[b]) + (t - nd - int(inp.cu_q[b])) + 1
            if n <= 0:
                continue
            w = window or n
            j = (n - w, n - w - 1, 0, n - 1, n // PAGE * PAGE, n // PAGE * PAGE - 1)[t % 6]
            j = min(max(j, 0), n - 1)
            for h in range(H):
                kr = keys[int(bt[j // PAGE]), h // (H // G), j % PAGE]
                q.view(T, H, dk)[t, h] = (kr * 3.0).to(dtype)
    return q, cache


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("peak", [False, True])
@pytest.mark.parametrize("step", list(STEPS) + ["long"])
@pytest.mark.parametrize("H,G,dk,dv,window", [(4, 2, 64, 64, 33), (6, 2, 128, 64, 1), (8, 2, 128, 128, 200), (3, 3, 128, 128, 64), (40, 2, 64, 128, 31),
                                              (2, 1, 256, 256, 100), (4, 1, 64, 256, 257), (2, 2, 256, 64, 0), (4, 1, 128, 256, 32),
                                              (4, 4, 256, 128, 5000), (16, 4, 128, 128, 128)])
def test_grouped_query_attention(dtype, peak, step, H, G, dk, dv, window):
    from lorax_b200.ops import native, reference
    dec, pre = STEPS[step] if step in STEPS else ([1000, 1500], [(1000, 300), (0, 500), (129, 40)])
    inp, nb, _ = make_step(dec, pre, seed=12)
    T = inp.positions.shape[0]
    q, cache = gqa_case(H, G, dk, dv, window, inp, nb, dtype, peak)
    want = torch.empty(T, H * dv)
    reference.gqa_attn(q.float(), cache.float(), H, G, dk, dv, dk ** -0.5, window, inp, want)
    out = torch.full((T, H * dv + 8), 3.0, dtype=dtype, device="cuda")
    native.gqa_attn(q.cuda(), cache.cuda(), H, G, dk, dv, dk ** -0.5, window, to_dev(inp), out)
    native.workspace(out.device).check_status()
    live = [i for i in range(T) if i >= len(dec) or dec[i] > 0]
    close(out[:, : H * dv], want, dtype, live, tol16=5e-3)
    assert (out[:, H * dv:] == 3.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,n", [(4, 2, 64, 64, 64), (6, 2, 128, 64, 80), (1, 1, 64, 256, 3), (5, 5, 256, 128, 200)])
def test_query_and_key_norms_with_cache_write(dtype, H, G, dk, dv, n):
    from lorax_b200.ops import native, reference
    inp, nb, _ = make_step([7, 0, 40], [(0, 50), (33, 5)], seed=8)
    T = inp.positions.shape[0]
    g = torch.Generator().manual_seed(3)
    x = torch.randn(T, (H + G) * dk + G * dv, generator=g)
    heads = x[:, : (H + G) * dk].view(T, H + G, dk)
    heads[:, :, n:] = 0
    x = x.to(dtype)
    wq, wk = torch.rand(dk, generator=g) + 0.5, torch.rand(dk, generator=g) + 0.5
    cache = torch.zeros(nb, G, PAGE * (dk + dv))
    xf, xd, cd = x.float(), x.cuda(), torch.zeros(nb, G, PAGE * (dk + dv), dtype=dtype, device="cuda")
    reference.qk_norm_kvwrite(xf, H, G, dk, dv, n, wq, wk, 1e-3, cache, inp.slots)
    native.qk_norm_kvwrite(xd, H, G, dk, dv, n, wq.cuda(), wk.cuda(), 1e-3, cd, inp.slots.cuda())
    close(xd[:, : H * dk], xf[:, : H * dk], dtype, tol16=5e-3)
    close(cd, cache, dtype, tol16=5e-3)


# ---------------------------------------------------------------------------------------------- norms of sublayer outputs, experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layernorm", [True, False])
@pytest.mark.parametrize("T,W,n,k", [(1, 16, 9, 0), (5, 208, 200, 3), (67, 4096, 4096, 0), (3, 5120, 5100, 9), (9, 2048, 2048, 2)])
def test_norm_added_to_the_stream(dtype, layernorm, T, W, n, k):
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T)
    pad = lambda t: torch.cat([t[..., :n], torch.zeros(*t.shape[:-1], W - n)], -1)
    res, w, b = pad(torch.randn(T, W, generator=g)), pad(1 + 0.2 * torch.randn(W, generator=g)), pad(torch.randn(W, generator=g))
    rows = max(T * k, T)
    y = torch.zeros(rows, W + 128)
    y[:, :W] = pad(torch.randn(rows, W, generator=g) + 0.7)
    y = y.to(dtype)
    pairs = None
    if k:
        pos = torch.randperm(T * k, generator=g).view(T, k).to(torch.int32)
        pos[0, 0] = -1
        pairs = (pos, torch.randn(T, k, generator=g))
    rf, rd = res.clone(), res.cuda()
    reference.norm_add(rf, y.float(), w, b, 0.3, 1e-5, n, torch.float32, layernorm, pairs)
    got = native.norm_add(rd, y.cuda(), w.cuda(), b.cuda(), 0.3, 1e-5, n, dtype, layernorm, tuple(p.cuda() for p in pairs) if k else None)
    close(rd, rf, torch.float32, tol32=1e-5)
    close(got, rf, dtype, tol16=4e-3)
    rows = torch.randint(0, T, (4,), generator=g, dtype=torch.int32)
    want = reference.norm_stream(rf, None, w, 1e-5, 0.0, n, torch.float32, bias=b, layernorm=layernorm, rows=rows) if layernorm else None
    if layernorm:
        close(native.norm_stream(rd, None, w.cuda(), 1e-5, 0.0, n, dtype, bias=b.cuda(), layernorm=True, rows=rows.cuda()), want, dtype, tol16=4e-3)
    table, pt = torch.randn(50, W, generator=g).to(dtype), torch.randn(20, W, generator=g).to(dtype)
    ids, at = torch.randint(0, 50, (T,), generator=g, dtype=torch.int32), torch.randint(0, 20, (T,), generator=g, dtype=torch.int32)
    c, cd = torch.empty(T, W, dtype=dtype), torch.empty(T, W, dtype=dtype, device="cuda")
    assert torch.equal(native.embed_stream(ids.cuda(), table.cuda(), 1.0, pos=pt.cuda(), positions=at.cuda(), copy=cd).cpu(),
                       reference.embed_stream(ids, table, 1.0, pos=pt, positions=at, copy=c))
    assert torch.equal(cd.cpu(), c)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,groups,keep,shared,W,ff", [(1, 8, 2, 0, 0, 0, 64, 128), (7, 12, 3, 4, 2, 1, 208, 128), (300, 40, 6, 8, 3, 2, 64, 256),
                                                           (65, 256, 8, 8, 4, 1, 128, 128), (2000, 64, 4, 64, 9, 3, 96, 128), (33, 6, 6, 2, 2, 1, 64, 128),
                                                           (40, 5, 1, 1, 1, 0, 48, 128), (700, 33, 32, 0, 0, 1, 64, 128)])
def test_experts_chosen_by_corrected_sigmoids_in_groups(dtype, T, E, k, groups, keep, shared, W, ff):
    """Choice, weights, sorted rows and the two grouped products; corrections so large that choice scores are negative and that score
    and choice order differ."""
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, W, generator=g).to(dtype)
    rows = (E + 1 + 15) // 16 * 16
    wr = torch.zeros(rows, W)
    wr[: E + 1] = torch.randn(E + 1, W, generator=g) * W ** -0.5 * 2
    wr = wr.to(dtype)
    corr = torch.randn(E, generator=g) * 0.7 - 0.6
    up = (torch.randn(E + shared, ff, W, generator=g) * W ** -0.5).to(dtype)
    down = (torch.randn(E + shared, 128, ff, generator=g) * ff ** -0.5).to(dtype)
    kw = dict(experts=E, score="sigmoid", groups=groups, keep=keep, scale=1.7, shared=shared)
    want = reference.moe_route(x.float(), wr.float(), k, 0, E, correction=corr, **kw)
    r = native.moe_route(x.cuda(), wr.cuda(), k, 0, E, correction=corr.cuda(), **kw)
    ids = r.topk_ids.cpu().long()
    # rows whose choice hangs on a difference below rounding are left out of the comparison of the choice
    clear = (ids.sort(-1).values == want.topk_ids.long().sort(-1).values).all(-1)
    assert clear.float().mean() > 0.99
    dense = lambda r: torch.zeros(T, E).scatter_(1, r.topk_ids.cpu().long(), r.topk_w.cpu()[:, :k])
    assert torch.allclose(dense(r)[clear], dense(want)[clear], atol=1e-5)
    if shared:
        assert torch.allclose(r.topk_w.cpu()[:, k:], want.topk_w[:, k:], atol=1e-5)
    seg, pos = r.seg.tolist(), r.pos.cpu().long()
    assert seg[0] == 0 and seg[E] == T * k and [seg[E + 1 + i] for i in range(shared)] == [T * k + (i + 1) * T for i in range(shared)]
    for j in range(k):
        assert all(seg[e] <= p < seg[e + 1] for e, p in zip(ids[:, j].tolist(), pos[:, j].tolist()))
    assert sorted(pos.flatten().tolist()) == list(range(T * (k + shared)))
    assert torch.equal(r.xg.cpu()[pos[:, :k]], x[:, None].expand(T, k, W))
    for i in range(shared):
        assert torch.equal(pos[:, k + i], T * k + i * T + torch.arange(T))
    avg = max(1, T * k // E)
    a = native.moe_grouped_gemm(r.xg, up.cuda(), r.seg, avg, shared=shared, tokens=T, act="relu2")
    y = native.moe_grouped_gemm(a, down.cuda(), r.seg, avg)
    native.workspace(y.device).check_status()
    # the reference products on the kernel's own order of rows
    af = reference.moe_grouped_gemm(r.xg.cpu().float(), up.float(), r.seg.cpu(), avg, shared=shared, tokens=T, act="relu2")
    close(a, af, dtype, tol16=5e-3)
    close(y, reference.moe_grouped_gemm(a.cpu().float(), down.float(), r.seg.cpu(), avg), dtype, tol16=5e-3)


# ---------------------------------------------------------------------------------------------- convolutions, state space recurrence, gated experts
SHORT = {"portions": ([3, 0, 1, 40], [(0, 1), (5, 1), (0, 2), (9, 2), (33, 7), (0, 9), (64, 8), (2, 70), (0, 200)])}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS) + ["portions"])
@pytest.mark.parametrize("taps,C", [(1, 16), (2, 272), (3, 48), (4, 528), (5, 40), (9, 256)])
def test_causal_convolution(dtype, step, taps, C):
    from lorax_b200.ops import native, reference
    dec, pre = {**STEPS, **SHORT}[step]
    inp, _, ns = make_step(dec, pre)
    T = inp.positions.shape[0]
    g = torch.Generator().manual_seed(taps)
    x = torch.randn(T, C + 24, generator=g).to(dtype)
    w, b, state = torch.randn(taps, C, generator=g), torch.randn(C, generator=g), torch.randn(ns, taps - 1, C, generator=g).to(dtype)
    live = [i for i in range(T) if i >= len(dec) or dec[i] > 0]
    for bias, act in ((b, "silu"), (None, "")):
        st, sd = state.float().clone(), state.cuda()
        want = reference.causal_conv(x[:, 8: 8 + C].float(), w, bias, act, st, inp)
        got = native.causal_conv(x.cuda()[:, 8: 8 + C], w.cuda(), bias.cuda() if bias is not None else None, act, sd, to_dev(inp))
        close(got, want, dtype, live, tol16=4e-3, tol32=2e-6)
        assert torch.equal(sd.float().cpu(), st)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS) + ["portions"])
@pytest.mark.parametrize("H,G,dk,dv,rot,taps", [(4, 2, 64, 64, 12, 0), (6, 2, 128, 64, 128, 3), (3, 0, 64, 128, 30, 0), (1, 1, 256, 128, 2, 4), (5, 5, 64, 256, 0, 7),
                                                (2, 2, 128, 128, 64, 1)])
def test_convolution_rotation_and_cache_write(dtype, step, H, G, dk, dv, rot, taps):
    from lorax_b200.ops import native, reference
    dec, pre = {**STEPS, **SHORT}[step]
    inp, nb, ns = make_step(dec, pre)
    T, C = inp.positions.shape[0], (H + G) * dk + G * dv
    g = torch.Generator().manual_seed(taps)
    x = torch.randn(T, C + 16, generator=g).to(dtype)
    table = reference.rope_table(rot, 1024, 500.0) if rot else None
    cache = torch.randn(nb, max(G, 1), PAGE * (dk + dv), generator=g).to(dtype)
    w = torch.randn(taps, C, generator=g) if taps else None
    state = torch.randn(ns, max(taps - 1, 0), C, generator=g).to(dtype)
    xf, cf, st = x[:, :C].float().clone(), cache.float().clone(), state.float().clone()
    want = reference.conv_rope_kvwrite(xf, H, G, dk, dv, table, rot, inp.positions, cf, inp, w, st)
    xd, cd, sd = x.cuda(), cache.cuda(), state.cuda()
    di = to_dev(inp)
    got = native.conv_rope_kvwrite(xd, H, G, dk, dv, table.cuda() if rot else None, rot, di.positions, cd, di, w.cuda() if taps else None, sd)
    live = [i for i in range(T) if i >= len(dec) or dec[i] > 0]
    close(got[:, : H * dk], want[:, : H * dk], dtype, live, tol16=4e-3, tol32=3e-6)
    close(cd, cf, dtype, tol16=4e-3, tol32=3e-6)
    assert torch.equal(sd.float().cpu(), st)
    if not taps:
        assert got.data_ptr() == xd.data_ptr() and torch.equal(xd[:, H * dk:].cpu(), x[:, H * dk:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS) + ["portions", "long"])
@pytest.mark.parametrize("H,G,n,p,strong", [(6, 3, 16, 48, False), (4, 1, 128, 64, False), (4, 2, 64, 128, True), (3, 3, 128, 64, True), (2, 1, 48, 16, False),
                                            (2, 2, 256, 64, True), (1, 1, 16, 16, False), (6, 2, 64, 32, False)])
def test_state_space_recurrence(dtype, step, H, G, n, p, strong):
    """Decays from almost none to almost everything within one token."""
    from lorax_b200.ops import native, reference
    dec, pre = {**STEPS, **SHORT, "long": ([700], [(100, 333), (0, 640)])}[step]
    inp, _, ns = make_step(dec, pre, seg_len=128 if step == "long" else 64)
    T = inp.positions.shape[0]
    g = torch.Generator().manual_seed(H)
    xbc = torch.randn(T, H * p + 2 * G * n, generator=g).to(dtype)
    dt = torch.randn(T, 16, generator=g).to(dtype)
    bias = torch.linspace(-9.0, 3.0 if strong else -1.0, H)
    A, D = -torch.exp(torch.linspace(-1.0, 3.0 if strong else 0.5, H)), torch.randn(H, generator=g)
    state = torch.randn(ns, H, n, p, generator=g)
    st, sd = state.clone(), state.cuda()
    want = reference.ssd(xbc.float(), dt.float(), H, G, n, p, bias, A, D, st, inp)
    got = native.ssd(xbc.cuda(), dt.cuda(), H, G, n, p, bias.cuda(), A.cuda(), D.cuda(), sd, to_dev(inp))
    live = [i for i in range(T) if i >= len(dec) or dec[i] > 0]
    close(got, want, dtype, live, tol16=1e-3)
    close(sd, st, dtype, tol16=1e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,vd,parts", [(1, 6, 12, 4), (5, 1, 1, 1), (70, 4, 64, 2), (3, 64, 64, 1), (9, 128, 80, 1), (4, 3, 7, 7), (6, 8, 128, 8)])
def test_gated_group_norm(dtype, T, H, vd, parts):
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T)
    pp, out_dim = (vd + 15) // 16 * 16, (H * vd + 15) // 16 * 16
    y, z, w = torch.randn(T, H * pp, generator=g) * 3, torch.randn(T, H * pp + 32, generator=g).to(dtype), torch.randn(H * vd, generator=g)
    want = reference.gate_norm(y, z[:, 16:].float(), H, vd, parts, w, 1e-4, torch.empty(T, out_dim))
    out = torch.full((T, out_dim + 48), 5.0, dtype=dtype, device="cuda")
    native.gate_norm(y.cuda(), z.cuda()[:, 16:], H, vd, parts, w.cuda(), 1e-4, out[:, 32: 32 + out_dim])
    close(out[:, 32: 32 + out_dim], want, dtype, tol16=4e-3)
    assert (out[:, :32] == 5.0).all() and (out[:, 32 + out_dim:] == 5.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sinks", ["none", "zero", "high", "low"])
@pytest.mark.parametrize("step", list(STEPS) + ["long"])
@pytest.mark.parametrize("H,G,dk,dv,window,cap", [(4, 2, 64, 64, 33, 5.0), (8, 2, 128, 128, 200, 30.0), (3, 3, 128, 128, 64, 0.0), (34, 2, 64, 128, 0, 2.0),
                                                  (2, 1, 256, 256, 100, 50.0), (4, 1, 128, 256, 1, 1.0), (16, 4, 128, 128, 128, 15.0)])
def test_attention_with_caps_sinks_and_gates(dtype, sinks, step, H, G, dk, dv, window, cap):
    from lorax_b200.ops import native, reference
    dec, pre = STEPS[step] if step in STEPS else ([1000, 1500], [(1000, 300), (0, 500), (129, 40)])
    inp, nb, _ = make_step(dec, pre, seed=12)
    T = inp.positions.shape[0]
    q, cache = gqa_case(H, G, dk, dv, window, inp, nb, dtype, True)
    g = torch.Generator().manual_seed(1)
    sink = {"none": None, "zero": torch.zeros(H), "high": torch.randn(H, generator=g) + 25.0, "low": torch.randn(H, generator=g) - 90.0}[sinks]
    gate = torch.randn(T, H * dv + 16, generator=g).to(dtype) * 2 if sinks != "low" else None
    scale = 0.02 if sinks == "zero" else dk ** -0.5
    want = torch.empty(T, H * dv)
    reference.gqa_attn(q.float(), cache.float(), H, G, dk, dv, scale, window, inp, want, softcap=cap, sink=sink,
                       gate=gate[:, 8: 8 + H * dv].float() if gate is not None else None, out_scale=0.7)
    out = torch.full((T, H * dv + 8), 3.0, dtype=dtype, device="cuda")
    native.gqa_attn(q.cuda(), cache.cuda(), H, G, dk, dv, scale, window, to_dev(inp), out, softcap=cap, sink=sink.cuda() if sink is not None else None,
                    gate=gate.cuda()[:, 8: 8 + H * dv] if gate is not None else None, out_scale=0.7)
    native.workspace(out.device).check_status()
    live = [i for i in range(T) if i >= len(dec) or dec[i] > 0]
    close(out[:, : H * dv], want, dtype, live, tol16=5e-3, tol32=4e-5)
    assert (out[:, H * dv:] == 3.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,groups,keep,W,ff", [(1, 8, 2, 0, 0, 64, 64), (7, 12, 3, 4, 2, 208, 128), (300, 40, 6, 8, 3, 64, 192), (65, 256, 8, 8, 4, 128, 64),
                                                    (33, 6, 6, 2, 2, 64, 64), (40, 5, 1, 1, 1, 48, 64), (700, 33, 32, 0, 0, 64, 64)])
def test_gated_experts_chosen_by_softmax_in_groups(dtype, T, E, k, groups, keep, W, ff):
    """Groups by their largest score, weights over all experts that are not renormalised, silu(gate) * up in the product's epilogue."""
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, W, generator=g).to(dtype)
    wr = torch.zeros((E + 15) // 16 * 16, W)
    wr[:E] = torch.randn(E, W, generator=g) * W ** -0.5 * 2
    wr = wr.to(dtype)
    up, down = (torch.randn(E, 2 * ff, W, generator=g) * W ** -0.5).to(dtype), (torch.randn(E, 128, ff, generator=g) * ff ** -0.5).to(dtype)
    kw = dict(experts=E, score="softmax", groups=groups, keep=keep, group_top=1, renorm=False)
    want = reference.moe_route(x.float(), wr.float(), k, 0, E, **kw)
    r = native.moe_route(x.cuda(), wr.cuda(), k, 0, E, **kw)
    ids = r.topk_ids.cpu().long()
    clear = (ids.sort(-1).values == want.topk_ids.long().sort(-1).values).all(-1)
    assert clear.float().mean() > 0.99
    dense = lambda r: torch.zeros(T, E).scatter_(1, r.topk_ids.cpu().long(), r.topk_w.cpu())
    assert torch.allclose(dense(r)[clear], dense(want)[clear], atol=1e-5)
    avg = max(1, T * k // E)
    a = native.moe_grouped_gemm(r.xg, up.cuda(), r.seg, avg, act="swiglu")
    y = native.moe_grouped_gemm(a, down.cuda(), r.seg, avg)
    native.workspace(y.device).check_status()
    assert a.shape == (T * k, ff)
    close(a, reference.moe_grouped_gemm(r.xg.cpu().float(), up.float(), r.seg.cpu(), avg, act="swiglu"), dtype, tol16=5e-3)
    close(y, reference.moe_grouped_gemm(a.cpu().float(), down.float(), r.seg.cpu(), avg), dtype, tol16=5e-3)
    # the norm that reads the stream next forms the weighted sums
    res, w = torch.randn(T, 128, generator=g), torch.randn(128, generator=g)
    rows = torch.randint(0, T, (3,), generator=g, dtype=torch.int32)
    pairs = (r.pos.cpu(), r.topk_w.cpu())
    for at in (None, rows):
        rf, rd = res.clone(), res.cuda()
        wn = reference.norm_stream(rf, y.cpu().float(), w, 1e-5, 0.0, 120, torch.float32, pairs=pairs, rows=at)
        gn = native.norm_stream(rd, y, w.cuda(), 1e-5, 0.0, 120, dtype, pairs=(r.pos, r.topk_w), rows=at.cuda() if at is not None else None)
        close(gn, wn, dtype, tol16=4e-3)
        if at is None:
            close(rd, rf, torch.float32, tol32=1e-5)
        plain = reference.norm_stream(res.clone(), y[:T].cpu().float(), w, 1e-5, 0.0, 120, torch.float32, rows=at)
        close(native.norm_stream(res.cuda(), y[:T], w.cuda(), 1e-5, 0.0, 120, dtype, rows=at.cuda() if at is not None else None), plain, dtype, tol16=4e-3)


@pytest.mark.parametrize("T,N,K", [(1, 48, 16), (70, 200, 96)])
def test_32_bit_product_with_bias(T, N, K):
    from lorax_b200.ops import native
    g = torch.Generator().manual_seed(T)
    x, w, b = torch.randn(T, K, generator=g), torch.randn(N, K, generator=g), torch.randn(N, generator=g)
    close(native.gemm(x.cuda(), w.cuda(), bias=b.cuda()), (x.double() @ w.double().t() + b).float(), torch.float32, tol32=2e-6)


# ---------------------------------------------------------------------------------------------- sandwich norms, turned values, windowed latents
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS) + ["long"])
@pytest.mark.parametrize("window", [1, 33, 64, 200])
@pytest.mark.parametrize("H,dk,rot,dv,kv", [(3, 32, 16, 48, 80), (2, 128, 64, 128, 512), (5, 64, 48, 64, 256), (17, 64, 16, 128, 128), (4, 128, 32, 128, 128)])
def test_latent_attention_with_windows_and_element_gates(dtype, window, step, H, dk, rot, dv, kv):
    """Both forms over queries that each match one key far better than all others: inside the window, at its edges, or just outside."""
    from lorax_b200.ops import native, native_mixers, reference
    dec, pre = STEPS[step] if step in STEPS else ([1000, 1500], [(1000, 300), (0, 500), (129, 40)])
    inp, nb, _ = make_step(dec, pre, seed=6, windows=(window,))
    T, head = inp.positions.shape[0], dk + rot
    q, cache, uk, uv = latent_case(H, dk, rot, dv, kv, inp, nb, dtype, False)
    nd, dbt, _, ctx = inp.decode_view(T)
    for t in range(T):
        b = int(torch.searchsorted(inp.cu_q[1:], torch.tensor(t - nd), right=True)) if t >= nd else 0
        bt, keys = (dbt[t], int(ctx[t])) if t < nd else (inp.block_tables[b], int(inp.cache_lens[b]) + (t - nd - int(inp.cu_q[b])) + 1)
        j = keys - 1 - (0, window - 1, window, window // 2, 1)[t % 5]
        if 0 <= j < keys:
            q.view(T, H, head)[t, :, dk:] = (cache[int(bt[j // PAGE]), j % PAGE, kv:].float() * 2.0).to(dtype)
    wide = torch.randn(T, H * dv + 32, generator=torch.Generator().manual_seed(9)).to(dtype)
    gate, scale = wide[:, 16: 16 + H * dv], head ** -0.5
    ql, want = torch.empty(T, H * kv), torch.zeros(T, H * dv)
    reference.gemm_heads(q.float(), uk.float().transpose(1, 2).contiguous(), ql, head)
    o = reference.latent_attn(ql, q.float(), cache.float(), H, kv, head, dk, rot, scale, inp, window=window)
    reference.gemm_heads(o, uv.float(), want, kv, gate=gate.float(), wide_gate=True)
    live = [i for i in range(T) if i >= len(dec) or dec[i] > 0]

    d, gd = to_dev(inp), wide.cuda()[:, 16: 16 + H * dv]
    rows = torch.zeros(T, H * head + 64, dtype=dtype, device="cuda")              # (queries within wider rows)
    qd, cd = rows[:, : H * head].copy_(q.cuda()), cache.cuda()
    qld, got = torch.empty(T, H * kv, dtype=dtype, device="cuda"), torch.zeros(T, H * dv, dtype=dtype, device="cuda")
    native.gemm_heads(qd, uk.transpose(1, 2).contiguous().cuda(), qld, head)
    od = native.latent_attn(qld, qd, cd, H, kv, head, dk, rot, scale, d, window=window)
    native.gemm_heads(od, uv.cuda(), got, kv, gate=gd, wide_gate=True)
    close(got, want, dtype, live)
    if pre:
        ukv = torch.cat([uk, uv], 1).reshape(H * (dk + dv), kv).contiguous().cuda()
        out = torch.zeros(T, H * dv, dtype=dtype, device="cuda")
        done = native.latent_prefill(qd, cd, ukv, gd, out, H, dk, rot, dv, scale, d, len(dec), window=window, wide_gate=True)
        assert done == (dtype == torch.bfloat16 and dk != 32 and T - len(dec) >= native_mixers.LATENT_EXPAND_MIN_ROWS * len(pre))
        if done:
            native.workspace(out.device).check_status()
            close(out, want, dtype, list(range(len(dec), T)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rot,rp,H,dk", [(10, 16, 3, 32), (64, 64, 5, 128), (16, 16, 9, 48)])
def test_latent_preparation_without_a_query_latent(dtype, rot, rp, H, dk):
    from lorax_b200.ops import native, reference
    inp, nb, _ = make_step([7, 0, 40], [(0, 50), (33, 5)], seed=8)
    T, kr, head = inp.positions.shape[0], 80, dk + rp
    g = torch.Generator().manual_seed(rot)
    x = torch.randn(T, H * head + kr + rp, generator=g).to(dtype)
    kn, cs = torch.rand(kr, generator=g) + 0.5, reference.rope_table(rot, 128, 10000.0)
    cache, xf = torch.zeros(nb, PAGE, kr + rp), x.float().clone()
    assert reference.latent_prep(None, xf[:, H * head:], None, kn, 0, 75, rot, 1e-5, cs, inp.positions, inp.slots, cache, q=xf, heads=H, head=head, off=dk) is None
    xd, cd = x.cuda(), torch.zeros(nb, PAGE, kr + rp, dtype=dtype, device="cuda")
    native.latent_prep(None, xd[:, H * head:], None, kn.cuda(), 0, 75, rot, 1e-5, cs.cuda(), inp.positions.cuda(), inp.slots.cuda(), cd, q=xd, heads=H,
                       head=head, off=dk)
    close(xd, xf, dtype, tol16=5e-3)
    close(cd, cache, dtype, tol16=5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,n,k,gated", [(7, 80, 76, 0, True), (1, 2048, 2048, 0, True), (33, 4096, 4090, 5, True), (3, 7168, 7168, 0, False), (5, 16384, 16384, 2, True)])
def test_gated_norm_added_and_the_stream_normed(dtype, T, W, n, k, gated):
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T)
    pad = lambda t: torch.cat([t[..., :n], torch.zeros(*t.shape[:-1], W - n)], -1)
    res, w, nxt = pad(torch.randn(T, W, generator=g)), pad(1 + 0.2 * torch.randn(W, generator=g)), pad(torch.randn(W, generator=g))
    y = torch.zeros(max(T * k, T), W + 128)
    y[:, :W] = pad(torch.randn(y.shape[0], W, generator=g))
    y, z = y.to(dtype), torch.randn(T, W + 16, generator=g).to(dtype)[:, 8: 8 + W] if gated else None
    pairs = None
    if k:
        pos = torch.randperm(T * k, generator=g).view(T, k).to(torch.int32)
        pos[0, 0] = -1
        pairs = (pos, torch.randn(T, k, generator=g))
    on = lambda t: t.cuda() if t is not None else None
    for rows in (None, torch.randint(0, T, (4,), generator=g, dtype=torch.int32)):
        rf, rd = res.clone(), res.cuda()
        want = reference.norm_add(rf, y.float(), w, None, 0.7, 1e-5, n, torch.float32, False, pairs, gate=z.float() if gated else None, next_weight=nxt, rows=rows)
        got = native.norm_add(rd, y.cuda(), w.cuda(), None, 0.7, 1e-5, n, dtype, False, tuple(p.cuda() for p in pairs) if k else None, gate=on(z),
                              next_weight=nxt.cuda(), rows=on(rows))
        close(got, want, dtype, tol16=5e-3)
        if rows is None:
            close(rd, rf, torch.float32, tol32=3e-5)
    none = native.norm_add(res.cuda(), y.cuda(), w.cuda(), None, 0.7, 1e-5, n, dtype, False, next_weight=nxt.cuda(), rows=torch.empty(0, dtype=torch.int32).cuda()) \
        if not k else torch.empty(0, W)
    assert none.shape == (0, W)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("limit", [0.3, 1.5, 100.0])
def test_clamped_gated_activation(dtype, limit):
    from lorax_b200.ops import native, reference
    x = (torch.randn(37, 2 * 96 + 40, generator=torch.Generator().manual_seed(1)) * 3).to(dtype)
    want = reference.act_mul(x.float(), 96, "clamped_swiglu", True, limit=limit)
    close(native.act_mul(x.cuda(), 96, "clamped_swiglu", True, limit=limit), want, dtype, tol16=4e-3, tol32=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS))
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(61, 31, 5), (1, 3, 2), (997, 1 << 33, 12345678901)])
def test_token_pairs(dtype, step, buckets, mul_prev, mul_cur):
    from lorax_b200.ops import native, reference
    inp, nb, _ = make_step(*STEPS[step], seed=2)
    T, V, W = inp.positions.shape[0], 50, 80
    g = torch.Generator().manual_seed(buckets)
    table, vectors = torch.randn(V, W, generator=g).to(dtype), torch.randn(buckets + 1, W, generator=g).to(dtype)
    ids, pages = (torch.randint(0, V, s, generator=g, dtype=torch.int32) for s in ((T,), (nb, PAGE)))
    pd = pages.cuda()
    got = native.embed_stream(ids.cuda(), table.cuda(), 0.6, bigram=(vectors.cuda(), (buckets, mul_prev, mul_cur), pd, to_dev(inp)))
    want = reference.embed_stream(ids, table, 0.6, bigram=(vectors, (buckets, mul_prev, mul_cur), pages, inp))
    live = [i for i in range(T) if i >= len(STEPS[step][0]) or STEPS[step][0][i] > 0]
    assert torch.allclose(got.cpu()[live], want[live], atol=1e-6) and torch.equal(pd.cpu(), pages)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,shared", [(1, 8, 2, 1), (70, 16, 4, 3), (300, 40, 6, 0), (33, 200, 9, 1), (9, 1, 1, 2)])
def test_routing_with_a_bias_and_shared_experts_of_weight_one(dtype, T, E, k, shared):
    from lorax_b200.ops import native, reference
    g = torch.Generator().manual_seed(T + E)
    W = 96
    x, wr, b = torch.randn(T, W, generator=g).to(dtype), torch.zeros((E + 8) // 8 * 8, W), torch.randn(E, generator=g)
    wr[:E] = torch.randn(E, W, generator=g) * W ** -0.5
    wr = wr.to(dtype)
    kw = dict(experts=E, score="softmax", renorm=True, shared=shared, shared_gate=False)
    want = reference.moe_route(x.float(), wr.float(), k, 0, E, bias=b, **kw)
    r = native.moe_route(x.cuda(), wr.cuda(), k, 0, E, bias=b.cuda(), **kw)
    clear = (r.topk_ids.cpu().long().sort(-1).values == want.topk_ids.long().sort(-1).values).all(-1)
    assert clear.float().mean() > 0.98
    dense = lambda r: torch.zeros(T, E).scatter_(1, r.topk_ids.cpu().long(), r.topk_w.cpu()[:, :k])
    assert torch.allclose(dense(r)[clear], dense(want)[clear], atol=1e-5) and (r.topk_w[:, k:] == 1).all() and r.topk_w.shape[1] == k + shared


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,n,rot,vd", [(6, 2, 64, 64, 20, 12, 28), (16, 2, 128, 128, 128, 64, 128), (3, 3, 128, 64, 70, 70, 10), (5, 1, 256, 256, 256, 2, 250)])
def test_normed_heads_and_values_rotated_into_the_cache(dtype, H, G, dk, dv, n, rot, vd):
    from lorax_b200.ops import native, reference
    inp, nb, _ = make_step([7, 0, 40], [(0, 50), (33, 5)], seed=8)
    T = inp.positions.shape[0]
    g = torch.Generator().manual_seed(n)
    x = torch.randn(T, (H + G) * dk + G * dv, generator=g)
    x[:, : (H + G) * dk].view(T, H + G, dk)[:, :, n:] = 0
    x[:, (H + G) * dk:].view(T, G, dv)[:, :, vd:] = 0
    x = x.to(dtype)
    wq, wk = torch.rand(dk, generator=g) + 0.5, torch.rand(dk, generator=g) + 0.5
    cs, vcs = reference.rope_table(rot, 128, 300.0), reference.rope_table(vd, 128, 300.0)
    for tables in ((cs, vcs), (cs, None), (None, vcs)):
        on = [t.cuda() if t is not None else None for t in tables]
        cache, cd = torch.zeros(nb, G, PAGE * (dk + dv)), torch.zeros(nb, G, PAGE * (dk + dv), dtype=dtype, device="cuda")
        xf, xd = x.float().clone(), x.cuda()
        reference.qk_norm_kvwrite(xf, H, G, dk, dv, n, wq, wk, 1e-3, cache, inp.slots, positions=inp.positions, cos_sin=tables[0], v_cos_sin=tables[1])
        native.qk_norm_kvwrite(xd, H, G, dk, dv, n, wq.cuda(), wk.cuda(), 1e-3, cd, inp.slots.cuda(), positions=inp.positions.cuda(), cos_sin=on[0], v_cos_sin=on[1])
        close(xd[:, : H * dk], xf[:, : H * dk], dtype, tol16=5e-3)
        close(cd, cache, dtype, tol16=5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", list(STEPS) + ["long"])
@pytest.mark.parametrize("H,G,dk,dv,vd,gated", [(6, 2, 64, 64, 28, False), (8, 2, 128, 128, 128, True), (3, 1, 128, 64, 64, False), (17, 1, 64, 256, 250, True), (4, 2, 128, 128, 90, False)])
def test_attention_outputs_turned_back(dtype, step, H, G, dk, dv, vd, gated):
    from lorax_b200.ops import native, reference
    dec, pre = STEPS[step] if step in STEPS else ([1000, 1500], [(1000, 300), (0, 500), (129, 40)])
    inp, nb, _ = make_step(dec, pre, seed=12)
    T = inp.positions.shape[0]
    q, cache = gqa_case(H, G, dk, dv, 0, inp, nb, dtype, True)
    turn = reference.rope_table(vd, 1600, 300.0)
    gate = torch.randn(T, H * dv, generator=torch.Generator().manual_seed(1)).to(dtype) if gated else None
    want = torch.empty(T, H * dv)
    reference.gqa_attn(q.float(), cache.float(), H, G, dk, dv, dk ** -0.5, 0, inp, want, gate=gate.float() if gated else None, turn_back=turn)
    out = torch.empty(T, H * dv, dtype=dtype, device="cuda")
    native.gqa_attn(q.cuda(), cache.cuda(), H, G, dk, dv, dk ** -0.5, 0, to_dev(inp), out, gate=gate.cuda() if gated else None, turn_back=turn.cuda())
    native.workspace(out.device).check_status()
    close(out, want, dtype, [i for i in range(T) if i >= len(dec) or dec[i] > 0], tol16=5e-3, tol32=4e-5)
