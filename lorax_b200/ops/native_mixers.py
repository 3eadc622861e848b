"""Bindings of the kernels of the layer-by-layer designs (`models/mixers.py`): `csrc/kernels/stream.cu`, `recurrent.cu`,
`conv_rope.cu`, `latent_attn.cu` and `gqa.cu`.  Every operator exists for bf16 and for fp32 activations.  Imported into :mod:`lorax_b200.ops.native`."""

from __future__ import annotations

import ctypes
from ctypes import POINTER, Structure, c_float, c_int, c_longlong, c_void_p
from typing import Optional

import torch

from . import native as nv

P, I, L, F = c_void_p, c_int, c_longlong, c_float


class StepRows(Structure):
    _fields_ = [("nd", I), ("dec_slots", P), ("ctx_lens", P), ("dec_bt", P), ("B", I), ("cu_q", P), ("cache_lens", P), ("slots", P),
                ("bt", P), ("max_blocks", I), ("dec_max_blocks", I)]


class EmbedPairs(Structure):
    _fields_ = [("vectors", P), ("pages", P), ("slots", P), ("mul_prev", L), ("mul_cur", L), ("buckets", I), ("page", I), ("rows", StepRows)]


class RecParams(Structure):
    _fields_ = [("q", P), ("k", P), ("v", P), ("z", P), ("ldq", L), ("ldk", L), ("ldv", L), ("ldz", L), ("decay", P), ("w0", P), ("u", P), ("skip", P),
                ("state", P), ("out", P), ("H", I), ("d", I), ("dv", I), ("hpg", I), ("rows", StepRows), ("seg_seq", P), ("seg_q0", P), ("nseg", I),
                ("seg_len", I), ("seg_state", P), ("seg_decay", P)]


class LinTcParams(Structure):
    _fields_ = [("q", P), ("k", P), ("v", P), ("ldq", L), ("ldk", L), ("ldv", L), ("decay", P), ("state", P), ("seg_state", P), ("out", P),
                ("H", I), ("dv", I), ("rows", StepRows), ("seg_seq", P), ("seg_q0", P), ("seg_len", I), ("hpg", I), ("z", P), ("ldz", L), ("w0", P),
                ("A", P), ("skip", P), ("seg_decay", P)]


class WkvTcParams(Structure):
    _fields_ = [("r", P), ("k", P), ("v", P), ("z", P), ("ldr", L), ("ldk", L), ("ldv", L), ("ldz", L), ("w0", P), ("u", P), ("state", P),
                ("seg_state", P), ("seg_decay", P), ("out", P), ("H", I), ("rows", StepRows), ("seg_seq", P), ("seg_q0", P), ("seg_len", I)]


class LatentPrepParams(Structure):
    _fields_ = [("dq", P), ("dkv", P), ("ld_dq", L), ("ld_dkv", L), ("dq_norm", P), ("dkv_norm", P), ("cq", P), ("cache", P),
                ("positions", P), ("slots", P), ("cos_sin", P), ("QR", I), ("KR", I), ("R", I), ("q_rank", I), ("kv_rank", I), ("rot", I),
                ("eps", F), ("q", P), ("ldq", L), ("H", I), ("head", I), ("off", I)]


class LatentAttnParams(Structure):
    _fields_ = [("q_lat", P), ("ld_ql", L), ("q", P), ("ldq", L), ("head", I), ("rot_off", I), ("cache", P), ("out", P), ("ldo", L),
                ("rows", StepRows), ("H", I), ("KR", I), ("R", I), ("page", I), ("scale", F), ("window", I)]


class LatentDecodeParams(Structure):
    _fields_ = [("q_lat", P), ("ld_ql", L), ("q", P), ("ldq", L), ("head", I), ("rot_off", I), ("cache", P), ("out", P), ("ldo", L),
                ("rows", StepRows), ("H", I), ("R", I), ("page", I), ("nsplit", I), ("scale", F), ("part_o", P), ("part_ml", P), ("window", I)]


class NormAddParams(Structure):
    _fields_ = [("residual", P), ("y", P), ("ldy", L), ("w", P), ("b", P), ("copy", P), ("pos", P), ("weights", P), ("k", I), ("W", I), ("n", I),
                ("layernorm", I), ("inv_n", F), ("eps", F), ("mult", F), ("gate", P), ("ldg", L), ("next_w", P), ("rows", P)]


class QkNormParams(Structure):
    _fields_ = [("qkv", P), ("ld", L), ("cache", P), ("slots", P), ("q_norm", P), ("k_norm", P), ("T", I), ("H", I), ("G", I), ("DK", I),
                ("DV", I), ("page", I), ("inv_n", F), ("eps", F), ("positions", P), ("cos_sin", P), ("v_cos_sin", P), ("rot", I), ("v_rot", I), ("P", I)]


class GqaF32Params(Structure):
    _fields_ = [("q", P), ("ldq", L), ("cache", P), ("out", P), ("ldo", L), ("rows", StepRows), ("T", I), ("H", I), ("G", I), ("DK", I),
                ("DV", I), ("page", I), ("window", I), ("scale", F), ("softcap", F), ("out_scale", F), ("sink", P), ("gate", P), ("ldg", L), ("turn", P),
                ("turn_dims", I), ("turn_rows", I)]


class NormStreamParams(Structure):
    _fields_ = [("residual", P), ("pending", P), ("ldp", L), ("w", P), ("out", P), ("pos", P), ("weights", P), ("rows", P), ("k", I), ("W", I),
                ("inv_n", F), ("eps", F), ("w_offset", F)]


class GateNormParams(Structure):
    _fields_ = [("y", P), ("z", P), ("w", P), ("out", P), ("ldz", L), ("ldo", L), ("H", I), ("vd", I), ("PP", I), ("part", I), ("ncols", I), ("eps", F)]


class ConvParams(Structure):
    _fields_ = [("x", P), ("ldx", L), ("out", P), ("ldo", L), ("w", P), ("b", P), ("state", P), ("rows", StepRows), ("tile_seq", P), ("tile_q0", P),
                ("C", I), ("taps", I), ("silu", I), ("dec_ctas", I), ("cache", P), ("slots", P), ("positions", P), ("cos_sin", P), ("P", I),
                ("rot", I), ("H", I), ("G", I), ("DK", I), ("DV", I), ("page", I)]


SIGNATURES = {
    "lx_embed_pairs_bytes": ([], I),
    "lx_embed_stream": ([P, P, P, I, I, I, F, P, P, I, P, P, I, P], I),
    "lx_norm_add_bytes": ([], I),
    "lx_norm_add": ([P, I, I, P], I),
    "lx_norm_rows": ([P, P, P, P, P, I, I, I, F, F, I, I, P], I),
    "lx_gqa_page_size": ([], I),
    "lx_qk_norm_bytes": ([], I),
    "lx_qk_norm_kvwrite": ([P, I, P], I),
    "lx_gqa_f32_bytes": ([], I),
    "lx_gqa_attn_f32": ([P, P], I),
    "lx_gqa_decode": ([P, L, P, P, I, P, P, L, P, P, I, I, I, I, I, I, F, I, F, P, P, L, F, P, I, I, P], I),
    "lx_gqa_prefill": ([P, L, P, P, I, P, P, P, P, I, P, L, I, I, I, I, I, F, F, P, P, L, F, P, I, I, P], I),
    "lx_gqa_prefill_tc": ([P, L, I, P, I, P, I, P, P, P, P, I, P, L, I, I, I, I, F, F, P, P, L, F, P, I, I, P, P], I),
    "lx_norm_stream_bytes": ([], I),
    "lx_norm_stream": ([P, I, I, P], I),
    "lx_gate_norm_bytes": ([], I),
    "lx_gate_norm": ([P, I, I, P], I),
    "lx_conv_bytes": ([], I),
    "lx_conv": ([P, I, I, I, P], I),
    "lx_norm_gate": ([P, P, P, L, P, L, I, I, I, I, F, I, I, P], I),
    "lx_tanh": ([P, L, I, P], I),
    "lx_act_mul_f32": ([P, P, I, I, L, L, I, I, P], I),
    "lx_clamped_swiglu": ([P, P, I, I, L, L, F, F, I, P], I),
    "lx_argmax_f32": ([P, L, I, I, P, P, F, P], I),
    "lx_gemm_batched": ([P, L, L, P, L, L, P, L, L, P, L, I, I, I, I, F, P, I, I, P], I),
    "lx_step_rows_bytes": ([], I),
    "lx_rec_params_bytes": ([], I),
    "lx_recurrence": ([P, I, I, I, P], I),
    "lx_linear_attn_tc_bytes": ([], I),
    "lx_linear_attn_tc_supported": ([I, I], I),
    "lx_linear_attn_tc": ([P, I, I, I, I, P], I),
    "lx_wkv_tc_bytes": ([], I),
    "lx_wkv_tc_supported": ([I], I),
    "lx_wkv_tc": ([P, I, I, P], I),
    "lx_silu_cols": ([P, L, I, I, P], I),
    "lx_token_shift": ([P, P, P, P, I, I, I, P, I, P], I),
    "lx_latent_prep_bytes": ([], I),
    "lx_latent_attn_bytes": ([], I),
    "lx_latent_prep": ([P, I, I, P], I),
    "lx_rope_pairs": ([P, L, P, P, I, I, I, I, I, I, P], I),
    "lx_latent_attn": ([P, I, I, P], I),
    "lx_latent_decode_bytes": ([], I),
    "lx_latent_decode_supported": ([I, I], I),
    "lx_latent_decode": ([P, I, I, P], I),
    "lx_latent_gather": ([P, P, I, P, P, I, I, I, I, I, I, P, P, P], I),
    "lx_latent_prefill_supported": ([I, I, I], I),
    "lx_latent_prefill": ([P, L, I, P, P, I, P, P, P, P, P, I, P, L, P, L, I, I, I, I, F, I, I, P, P], I),
}


def check_layouts(lib):
    for name, st in (("lx_step_rows_bytes", StepRows), ("lx_embed_pairs_bytes", EmbedPairs), ("lx_rec_params_bytes", RecParams), ("lx_latent_prep_bytes", LatentPrepParams),
                     ("lx_latent_attn_bytes", LatentAttnParams), ("lx_latent_decode_bytes", LatentDecodeParams),
                     ("lx_linear_attn_tc_bytes", LinTcParams), ("lx_wkv_tc_bytes", WkvTcParams),
                     ("lx_norm_add_bytes", NormAddParams), ("lx_qk_norm_bytes", QkNormParams), ("lx_gqa_f32_bytes", GqaF32Params),
                     ("lx_norm_stream_bytes", NormStreamParams), ("lx_gate_norm_bytes", GateNormParams), ("lx_conv_bytes", ConvParams)):
        if getattr(lib, name)() != ctypes.sizeof(st):
            raise nv.NativeError(f"{name}: C++ says {getattr(lib, name)()} bytes, ctypes says {ctypes.sizeof(st)}")


def _f32(t: torch.Tensor) -> int:
    return int(t.dtype == torch.float32)


def _p(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def step_rows(inp, T: int) -> StepRows:
    nd, dbt, slots, ctx = inp.decode_view(T)
    r = StepRows()
    r.nd = nd
    if nd:
        r.dec_slots, r.ctx_lens, r.dec_bt, r.dec_max_blocks = _p(slots), _p(ctx), _p(dbt), dbt.shape[1]
    if inp.is_prefill:
        r.B, r.cu_q, r.cache_lens, r.slots = inp.cache_lens.shape[0], _p(inp.cu_q), _p(inp.cache_lens), _p(inp.state_slots)
        r.bt, r.max_blocks = _p(inp.block_tables), inp.block_tables.shape[1]
    return r


def embed_stream(ids, table, mult: float = 1.0, pos=None, positions=None, copy=None, bigram=None):
    T, W = ids.shape[0], table.shape[1]
    out = torch.empty(T, W, dtype=torch.float32, device=table.device)
    pairs = None
    if bigram is not None:
        vectors, (buckets, mul_prev, mul_cur), pages, inp = bigram
        pairs = ctypes.byref(EmbedPairs(_p(vectors), _p(pages), _p(inp.slots), mul_prev, mul_cur, buckets, pages.shape[1], step_rows(inp, T)))
    nv._check(nv.load().lx_embed_stream(_p(ids), _p(table), _p(out), T, W, table.shape[0], mult, _p(pos), _p(positions) if pos is not None else None,
                                        pos.shape[0] if pos is not None else 0, _p(copy), pairs, _f32(table), nv._stream()), "lx_embed_stream")
    return out


def norm_stream(residual, pending, weight, eps: float, weight_offset: float, n: int, dtype, bias=None, layernorm: bool = False, rows=None,
                pairs=None):
    """(with `rows`, pending is added to the rows it takes on the way and `residual` stays as it is)"""
    T, W = residual.shape
    if rows is not None:
        T = rows.shape[0]
    out = torch.empty(T, W, dtype=dtype, device=residual.device)
    if T == 0:
        return out
    if layernorm or (rows is not None and pending is None):
        assert pending is None
        nv._check(nv.load().lx_norm_rows(_p(residual), _p(rows), _p(weight), _p(bias), _p(out), T, W, n, eps, weight_offset, int(layernorm),
                                         _f32(out), nv._stream()), "lx_norm_rows")
        return out
    pos, w = pairs if pairs is not None else (None, None)
    p = NormStreamParams(_p(residual), _p(pending), pending.stride(0) if pending is not None else 0, _p(weight), _p(out), _p(pos), _p(w), _p(rows),
                         pos.shape[1] if pos is not None else 0, W, 1.0 / n, eps, weight_offset)
    nv._check(nv.load().lx_norm_stream(ctypes.byref(p), T, _f32(out), nv._stream()), "lx_norm_stream")
    return out


def norm_add(residual, y, weight, bias, mult: float, eps: float, n: int, dtype, layernorm: bool = True, pairs=None, gate=None,
             next_weight=None, rows=None):
    T, W = residual.shape
    if rows is not None:
        T = rows.shape[0]
    copy = torch.empty(T, W, dtype=dtype, device=residual.device) if dtype != torch.float32 or next_weight is not None else None
    pos, w = pairs if pairs is not None else (None, None)
    p = NormAddParams(_p(residual), _p(y), y.stride(0), _p(weight), _p(bias), _p(copy), _p(pos), _p(w), pos.shape[1] if pos is not None else 0, W,
                      n, int(layernorm), 1.0 / n, eps, mult, _p(gate), gate.stride(0) if gate is not None else 0, _p(next_weight), _p(rows))
    nv._check(nv.load().lx_norm_add(ctypes.byref(p), T, _f32(y), nv._stream()), "lx_norm_add")
    return residual if copy is None else copy


def norm_gate(x, group: int, n: int, weight, gate, act: str, eps: float, out):
    T, C = x.shape
    nv._check(nv.load().lx_norm_gate(_p(x), _p(weight), _p(gate), gate.stride(0), _p(out), out.stride(0), T, C // group, group, n, eps,
                                     int(act == "silu"), _f32(out), nv._stream()), "lx_norm_gate")
    return out


def tanh_(x):
    assert x.is_contiguous()
    nv._check(nv.load().lx_tanh(_p(x), x.numel(), _f32(x), nv._stream()), "lx_tanh")
    return x


def gate_norm(y, z, H: int, p: int, parts: int, weight, eps: float, out):
    T, C = y.shape
    a = GateNormParams(_p(y), _p(z), _p(weight), _p(out), z.stride(0), out.stride(0), H, p, C // H, H * p // parts, out.shape[1], eps)
    nv._check(nv.load().lx_gate_norm(ctypes.byref(a), T, _f32(out), nv._stream()), "lx_gate_norm")
    return out


def gemm_f32(x, w, out=None, out_scale: float = 1.0, bias=None):
    T, K = x.shape
    N = w.shape[0]
    if out is None:
        out = torch.empty(T, N, dtype=torch.float32, device=x.device)
    nv._check(nv.load().lx_gemm_batched(_p(x), x.stride(0), 0, _p(w), w.stride(0), 0, _p(out), out.stride(0), 0, None, 0, T, N, K, 1, out_scale,
                                        _p(bias), 0, 1, nv._stream()), "lx_gemm_batched")
    return out


STACK_GROUPED_MAX_ROWS = 256
_segments = {}


def _stack_segments(n: int, T: int, device) -> torch.Tensor:
    key = (n, T, device)
    if key not in _segments:
        _segments[key] = torch.arange(0, (n + 1) * T, T, dtype=torch.int32, device=device)
    return _segments[key]


def gemm_stack(x, w):
    """x [n, T, K], w [n, N, K] -> [n, T, N]: one product per stacked pair."""
    n, T, K = x.shape
    N = w.shape[1]
    out = torch.empty(n, T, N, dtype=x.dtype, device=x.device)
    if x.dtype == torch.bfloat16 and T <= STACK_GROUPED_MAX_ROWS and N % 128 == 0 and x.is_contiguous():
        # few rows: all products stream their weights in one launch (the grouped GEMM of the expert layers, one group per pair)
        nv.moe_grouped_gemm(x.view(n * T, K), w, _stack_segments(n, T, x.device), T, out.view(n * T, N))
        return out
    for i in range(n):
        nv.gemm(x[i], w[i], out=out[i])
    return out


def gemm_heads(x, w, out, x_head: int, gate=None, wide_gate: bool = False):
    """out[:, h * N : (h + 1) * N] = x[:, h * x_head : h * x_head + K] @ w[h]^T (* sigmoid(gate[:, h]), or of the output's own gate column)."""
    H, N, K = w.shape
    T = x.shape[0]
    nv._check(nv.load().lx_gemm_batched(_p(x), x.stride(0), x_head, _p(w), K, N * K, _p(out), out.stride(0), N, _p(gate),
                                        gate.stride(0) if gate is not None else 0, T, N, K, H, 1.0, None, int(wide_gate), _f32(x), nv._stream()),
              "lx_gemm_batched")
    return out


def _recurrence(mode: int, q, k, v, z, decay, w0, u, H: int, d: int, dv: int, state, inp, skip=None, hpg: int = 1):
    T = q.shape[0]
    out = torch.empty(T, H * dv, dtype=torch.float32, device=q.device)
    p = RecParams()
    p.q, p.k, p.v, p.z = _p(q), _p(k), _p(v), _p(z)
    p.ldq, p.ldk, p.ldv, p.ldz = q.stride(0), k.stride(0), v.stride(0), z.stride(0) if z is not None else 0
    p.decay, p.w0, p.u, p.skip, p.state, p.out = _p(decay), _p(w0), _p(u), _p(skip), _p(state), _p(out)
    p.H, p.d, p.dv, p.hpg, p.rows = H, d, dv, hpg, step_rows(inp, T)
    multi = 0
    hold = None
    if inp.is_prefill:
        p.seg_seq, p.seg_q0, p.nseg, p.seg_len = _p(inp.seg_seq), _p(inp.seg_q0), inp.seg_seq.shape[0], inp.seg_len
        multi = int(p.nseg > p.rows.B)
        if multi:
            hold = torch.empty(p.nseg * H * d * (dv + 1), dtype=torch.float32, device=q.device)
            p.seg_state, p.seg_decay = _p(hold), hold.data_ptr() + 4 * p.nseg * H * d * dv
    lib = nv.load()
    step, prompts = (1 if p.rows.nd else 0), p.rows.B > 0

    def passes(what):
        if what:
            nv._check(lib.lx_recurrence(ctypes.byref(p), mode, what, _f32(q), nv._stream()), "lx_recurrence")
            nv.launch_count += bin(what).count("1") - 1

    if mode in (0, 2) and prompts and q.dtype == torch.bfloat16 and lib.lx_linear_attn_tc_supported(d, dv):
        t = LinTcParams(p.q, p.k, p.v, p.ldq, p.ldk, p.ldv, p.decay, p.state, p.seg_state, p.out, H, dv, p.rows, p.seg_seq, p.seg_q0, p.seg_len,
                        hpg, p.z, p.ldz, p.w0, p.u, p.skip, p.seg_decay)

        def chunks(states):
            nv._check(lib.lx_linear_attn_tc(ctypes.byref(t), d, p.nseg, states, int(mode == 2), nv._stream()), "lx_linear_attn_tc")
        passes(step)
        nd = p.rows.nd
        for x, cols in () if mode == 2 else (((q, 2 * H * d + H * dv),) if k.data_ptr() == q.data_ptr() + 2 * H * d and v.data_ptr() == k.data_ptr() + 2 * H * d
                        else ((q, H * d), (k, H * d), (v, H * dv))):
            nv._check(lib.lx_silu_cols(_p(x[nd:]), x.stride(0), T - nd, cols, nv._stream()), "lx_silu_cols")
        if multi:
            chunks(1)
            passes(4)
        chunks(0)
        return out
    if mode == 1 and prompts and q.dtype == torch.bfloat16 and lib.lx_wkv_tc_supported(d):
        t = WkvTcParams(p.q, p.k, p.v, p.z, p.ldq, p.ldk, p.ldv, p.ldz, p.w0, p.u, p.state, p.seg_state, p.seg_decay, p.out, H, p.rows,
                        p.seg_seq, p.seg_q0, p.seg_len)

        def blocks(states):
            nv._check(lib.lx_wkv_tc(ctypes.byref(t), p.nseg, states, nv._stream()), "lx_wkv_tc")
        passes(step)
        if multi:
            blocks(1)
            passes(4)
        blocks(0)
        return out
    passes(step | (6 if multi else 0) | (8 if prompts else 0))
    return out


def linear_attn(q, k, v, H: int, d: int, dv: int, decay, state, inp):
    """(q, k and v are consumed: prompt rows may be overwritten by their silu)"""
    return _recurrence(0, q, k, v, None, decay, None, None, H, d, dv, state, inp)


def wkv(r, k, v, z, w0, u, H: int, d: int, state, inp):
    return _recurrence(1, r, k, v, z, None, w0, u, H, d, d, state, inp)


def ssd(xbc, dt, H: int, G: int, n: int, p: int, dt_bias, A, D, state, inp):
    x, B, C = xbc[:, : H * p], xbc[:, H * p: H * p + G * n], xbc[:, H * p + G * n:]
    return _recurrence(2, C, B, x, dt, None, dt_bias, A, H, n, p, state, inp, skip=D, hpg=H // G)


def _conv(x, C: int, taps: int, w, b, state, inp, out, attn: bool, **more):
    T = x.shape[0]
    p = ConvParams()
    p.x, p.ldx, p.out, p.ldo, p.w, p.b, p.state = _p(x), x.stride(0), _p(out), out.stride(0), _p(w), _p(b), _p(state)
    p.rows, p.C, p.taps = step_rows(inp, T), C, taps
    tiles = 0
    if inp.is_prefill:
        p.tile_seq, p.tile_q0, tiles = _p(inp.tile_seq), _p(inp.tile_q0), inp.tile_seq.shape[0]
    for k, v in more.items():
        setattr(p, k, v)
    nv._check(nv.load().lx_conv(ctypes.byref(p), tiles, int(attn), _f32(x), nv._stream()), "lx_conv")
    return out


def causal_conv(x, w, b, act: str, state, inp):
    taps, C = w.shape
    return _conv(x, C, taps, w, b, state, inp, torch.empty(x.shape[0], C, dtype=x.dtype, device=x.device), False, silu={"": 0, "silu": 1}[act])


def conv_rope_kvwrite(qkv, H: int, G: int, dk: int, dv: int, cos_sin, rot: int, positions, cache, inp, conv_w=None, conv_state=None):
    out = qkv if conv_w is None else torch.empty(qkv.shape[0], H * dk, dtype=qkv.dtype, device=qkv.device)
    more = dict(rot=rot, H=H, G=G, DK=dk, DV=dv, page=cache.shape[2] // (dk + dv), cache=_p(cache), slots=_p(inp.slots), positions=_p(positions))
    if rot:
        more.update(cos_sin=_p(cos_sin), P=cos_sin.shape[0])
    return _conv(qkv, (H + G) * dk + G * dv, 0 if conv_w is None else conv_w.shape[0], conv_w, None, conv_state, inp, out, True, **more)


def token_shift(h, mu, shift, inp):
    T, W = h.shape
    out = torch.empty(mu.shape[0], T, W, dtype=h.dtype, device=h.device)
    rows = step_rows(inp, T)
    nv._check(nv.load().lx_token_shift(_p(h), _p(mu), _p(shift), _p(out), mu.shape[0], W, T, ctypes.byref(rows), _f32(h), nv._stream()),
              "lx_token_shift")
    nv.launch_count += int(rows.B > 0)
    return out


def latent_prep(dq, dkv, dq_norm, dkv_norm, q_rank: int, kv_rank: int, rot: int, eps: float, cos_sin, positions, slots, cache, q=None,
                heads: int = 0, head: int = 0, off: int = 0):
    T, QR, KR = dkv.shape[0], dq_norm.shape[0] if dq is not None else 0, dkv_norm.shape[0]
    cq = torch.empty(T, QR, dtype=dq.dtype, device=dq.device) if dq is not None else None
    p = LatentPrepParams(_p(dq), _p(dkv), dq.stride(0) if dq is not None else 0, dkv.stride(0), _p(dq_norm), _p(dkv_norm), _p(cq), _p(cache), _p(positions), _p(slots),
                         _p(cos_sin), QR, KR, cache.shape[2], q_rank, kv_rank, rot, eps, _p(q), q.stride(0) if q is not None else 0, heads, head, off)
    nv._check(nv.load().lx_latent_prep(ctypes.byref(p), T, _f32(dkv), nv._stream()), "lx_latent_prep")
    return cq


def rope_pairs(x, positions, cos_sin, H: int, head: int, off: int, rot: int):
    nv._check(nv.load().lx_rope_pairs(_p(x), x.stride(0), _p(positions), _p(cos_sin), x.shape[0], H, head, off, rot, _f32(x), nv._stream()),
              "lx_rope_pairs")


def latent_attn(q_lat, q, cache, H: int, kv_rank: int, head: int, rot_off: int, rot: int, scale: float, inp, window: int = 0):
    T = q.shape[0]
    out = torch.empty(T, H * kv_rank, dtype=q.dtype, device=q.device)
    lib = nv.load()
    if q.dtype == torch.bfloat16 and lib.lx_latent_decode_supported(kv_rank, kv_rank + rot):
        d = LatentDecodeParams()
        d.q_lat, d.ld_ql, d.q, d.ldq, d.head, d.rot_off = _p(q_lat), q_lat.stride(0), _p(q), q.stride(0), head, rot_off
        d.cache, d.out, d.ldo, d.rows = _p(cache), _p(out), out.stride(0), step_rows(inp, T)
        d.H, d.R, d.page, d.scale = H, kv_rank + rot, cache.shape[1], scale
        # the keys of a row are shared out until the grid fills the GPU once (one CTA per SM, two for up to 16 heads)
        groups, per_sm = ((H + 31) // 32, 1) if H > 16 else (1, 2)
        d.nsplit = max(1, min(32, nv.workspace(q.device).num_sms * per_sm // (T * groups)))
        d.window = window
        if window > 0:                                       # (no share without a 64-key tile)
            d.nsplit = min(d.nsplit, window // 64 + 1)
        hold = None
        if d.nsplit > 1:
            n = T * H * d.nsplit
            hold = torch.empty(n * (kv_rank + 2), dtype=torch.float32, device=q.device)
            d.part_o, d.part_ml = _p(hold), hold.data_ptr() + 4 * n * kv_rank
        nv._check(lib.lx_latent_decode(ctypes.byref(d), kv_rank, T, nv._stream()), "lx_latent_decode")
        nv.launch_count += int(d.nsplit > 1)
        return out
    p = LatentAttnParams()
    p.q_lat, p.ld_ql, p.q, p.ldq, p.head, p.rot_off = _p(q_lat), q_lat.stride(0), _p(q), q.stride(0), head, rot_off
    p.cache, p.out, p.ldo, p.rows = _p(cache), _p(out), out.stride(0), step_rows(inp, T)
    p.H, p.KR, p.R, p.page, p.scale, p.window = H, kv_rank, kv_rank + rot, cache.shape[1], scale, window
    nv._check(nv.load().lx_latent_attn(ctypes.byref(p), T, _f32(q), nv._stream()), "lx_latent_attn")
    return out


# mean prompt tokens per sequence from which a prompt expands its latents to keys and values instead of being carried into the
# latent space row by row (the expansion costs a row of the context about as much as twenty queries save on it)
LATENT_EXPAND_MIN_ROWS = 24


def latent_prefill(q, cache, w_ukv, gate, out, H: int, dk: int, rot: int, dv: int, scale: float, inp, nd: int, window: int = 0,
                   wide_gate: bool = False) -> bool:
    """Gated attention outputs of the prompt rows [nd, T) into out[nd:, : H * dv] on the tensor-core kernel; False when this step is
    better (or only) served by the absorbed form."""
    T, B = q.shape[0] - nd, inp.cache_lens.shape[0]
    lib = nv.load()
    if q.dtype != torch.bfloat16 or T < LATENT_EXPAND_MIN_ROWS * B or not lib.lx_latent_prefill_supported(dk, rot, dv):
        return False
    ctx_off, rows = inp.contexts[window]
    KR, dev = cache.shape[2] - rot, q.device
    lat = torch.empty(rows, KR, dtype=q.dtype, device=dev)
    keys = torch.empty(rows, rot, dtype=q.dtype, device=dev)
    nv._check(lib.lx_latent_gather(_p(cache), _p(inp.block_tables), inp.block_tables.shape[1], _p(ctx_off), _p(inp.cache_lens), window, B, rows,
                                   cache.shape[1], KR, rot, _p(lat), _p(keys), nv._stream()), "lx_latent_gather")
    kv = nv.gemm(lat, w_ukv)
    y, g = out[nd:], gate[nd:]
    qp = q[nd:]
    nv._check(lib.lx_latent_prefill(_p(qp), qp.stride(0), T, _p(kv), _p(keys), rows, _p(ctx_off), _p(inp.cu_q), _p(inp.cache_lens),
                                    _p(inp.q128_seq), _p(inp.q128_q0), inp.q128_seq.shape[0], _p(g), g.stride(0), _p(y), y.stride(0), H, dk, rot,
                                    dv, scale, window, int(wide_gate), _p(nv.workspace(dev).status), nv._stream()), "lx_latent_prefill")
    return True


def qk_norm_kvwrite(qkv, H: int, G: int, dk: int, dv: int, n: int, q_norm, k_norm, eps: float, cache, slots, positions=None,
                    cos_sin=None, v_cos_sin=None):
    width = lambda t: t.shape[1] if t is not None else 0
    rows = min([t.shape[0] for t in (cos_sin, v_cos_sin) if t is not None] + [1 << 30])
    p = QkNormParams(_p(qkv), qkv.stride(0), _p(cache), _p(slots), _p(q_norm), _p(k_norm), qkv.shape[0], H, G, dk, dv,
                     cache.shape[2] // (dk + dv), 1.0 / n, eps, _p(positions), _p(cos_sin), _p(v_cos_sin), width(cos_sin), width(v_cos_sin), rows)
    nv._check(nv.load().lx_qk_norm_kvwrite(ctypes.byref(p), _f32(qkv), nv._stream()), "lx_qk_norm_kvwrite")


def _gqa_splits(ctas: int, window: int, max_blocks: int, page: int) -> int:
    """Parts the keys of one row and head group are cut into: one when the rows fill the GPU, else enough to do so with at least four
    pages each."""
    if ctas >= 96:
        return 1
    pages = min(max_blocks, (window + page - 1) // page + 1 if window > 0 else max_blocks)
    return max(1, min(8, 192 // max(1, ctas), pages // 4))


def gqa_attn(q, cache, H: int, G: int, dk: int, dv: int, scale: float, window: int, inp, out, softcap: float = 0.0, sink=None, gate=None,
             out_scale: float = 1.0, turn_back=None):
    T = q.shape[0]
    turn = (_p(turn_back), turn_back.shape[1], turn_back.shape[0]) if turn_back is not None else (None, 0, 0)
    lib, ws = nv.load(), nv.workspace(q.device)
    page = cache.shape[2] // (dk + dv)
    ldg = gate.stride(0) if gate is not None else 0
    if q.dtype == torch.float32:
        p = GqaF32Params(_p(q), q.stride(0), _p(cache), _p(out), out.stride(0), step_rows(inp, T), T, H, G, dk, dv, page, window, scale, softcap,
                         out_scale, _p(sink), _p(gate), ldg, *turn)
        nv._check(lib.lx_gqa_attn_f32(ctypes.byref(p), nv._stream()), "lx_gqa_attn_f32")
        return out
    if page != lib.lx_gqa_page_size():
        raise ValueError(f"the attention kernels take pages of {lib.lx_gqa_page_size()} tokens, not {page}")
    nd, dbt, _, ctx = inp.decode_view(T)
    if nd:
        nsplit = _gqa_splits(nd * G * ((H // G + 15) // 16), window, dbt.shape[1], page)
        part_o = part_lse = None
        if nsplit > 1:
            part_o = torch.empty(nd * H * nsplit * (dv + 1), dtype=torch.float32, device=q.device)
            part_lse = part_o[nd * H * nsplit * dv:]
        nv._check(lib.lx_gqa_decode(_p(q), q.stride(0), _p(cache), _p(dbt), dbt.shape[1], _p(ctx), _p(out), out.stride(0), _p(part_o), _p(part_lse),
                                    nd, H, G, dk, dv, window, scale, nsplit, softcap, _p(sink), _p(gate), ldg, out_scale, *turn, nv._stream()),
                  "lx_gqa_decode")
        nv.launch_count += int(nsplit > 1)
    if inp.is_prefill:
        qp, op, tiles = q[nd:], out[nd:], inp.tile_seq.shape[0]
        gp = gate[nd:] if gate is not None else None
        if nv.TC_PREFILL and dk == dv and lib.lx_attn_prefill_tc_supported(H, G, dk, q.stride(0), out.stride(0)):
            nv._check(lib.lx_gqa_prefill_tc(_p(qp), q.stride(0), T - nd, _p(cache), cache.shape[0], _p(inp.block_tables), inp.block_tables.shape[1],
                                            _p(inp.cu_q), _p(inp.cache_lens), _p(inp.tile_seq), _p(inp.tile_q0), tiles, _p(op), out.stride(0), H, G,
                                            dk, window, scale, softcap, _p(sink), _p(gp), ldg, out_scale, *turn, _p(ws.status), nv._stream()),
                      "lx_gqa_prefill_tc")
        else:
            nv._check(lib.lx_gqa_prefill(_p(qp), q.stride(0), _p(cache), _p(inp.block_tables), inp.block_tables.shape[1], _p(inp.cu_q),
                                         _p(inp.cache_lens), _p(inp.tile_seq), _p(inp.tile_q0), tiles, _p(op), out.stride(0), H, G, dk, dv, window,
                                         scale, softcap, _p(sink), _p(gp), ldg, out_scale, *turn, nv._stream()), "lx_gqa_prefill")
    return out
