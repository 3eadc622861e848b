"""Plain PyTorch statements of every operator.

They are the oracle for the CUDA kernels (tests compare a kernel against the fp32 version of the same
function) and the compute path of the engine on a machine without a GPU.  Signatures mirror
:mod:`lorax_b200.ops.native`.
"""

from __future__ import annotations

import math
from typing import NamedTuple, Optional

import torch
import torch.nn.functional as F


def gemm(x, w, bias=None, out=None, out_scale: float = 1.0, lora=None, **_):
    y = (x.float() @ w.float().t()) * out_scale
    if bias is not None:
        y = y + bias.float()
    if lora is not None:      # the CUDA kernel adds the delta in its epilogue, before the one rounding to bf16
        d = torch.zeros_like(y)
        lora_expand(lora.v, lora.tok_slot, lora.arena, lora.slot_base, lora.slot_rank, lora.unit_off, d, lora.n0, lora.n1)
        y = y + d
    y = y.to(x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


FP8_MAX = 448.0


def quantize_weight_fp8_block128(w: torch.Tensor):
    """[N, K] -> (e4m3 [N, K], fp32 scales [ceil(N/128), ceil(K/128)]): w ~= q * scale of its 128 x 128 block."""
    N, K = w.shape
    nb, kb = (N + 127) // 128, (K + 127) // 128
    wp = torch.zeros(nb * 128, kb * 128, dtype=torch.float32, device=w.device)
    wp[:N, :K] = w.float()
    blocks = wp.view(nb, 128, kb, 128)
    scale = blocks.abs().amax(dim=(1, 3)).clamp_min(1e-12) / FP8_MAX
    q = (blocks / scale[:, None, :, None]).clamp(-FP8_MAX, FP8_MAX).view(nb * 128, kb * 128)[:N, :K].to(torch.float8_e4m3fn)
    return q.contiguous(), scale.contiguous()


def dequantize_weight_fp8_block128(q: torch.Tensor, scale: torch.Tensor) -> torch.Tensor:
    N, K = q.shape
    s = scale.repeat_interleave(128, 0)[:N].repeat_interleave(128, 1)[:, :K]
    return q.view(torch.float8_e4m3fn).float() * s


def quant_act_fp8(x):
    """Per token and 128-wide K block: (e4m3 [T, K], scales [K/128, T])."""
    T, K = x.shape
    kb = (K + 127) // 128
    xp = torch.zeros(T, kb * 128, dtype=torch.float32, device=x.device)
    xp[:, :K] = x.float()
    b = xp.view(T, kb, 128)
    scale = b.abs().amax(dim=2).clamp_min(1e-12) / FP8_MAX
    q = (b / scale[:, :, None]).clamp(-FP8_MAX, FP8_MAX).view(T, kb * 128)[:, :K].to(torch.float8_e4m3fn)
    return q.contiguous(), scale.t().contiguous()


def gemm_wq(x, w, bias=None, out=None):
    """Oracle of the weight-only quantised GEMM: the packed matrix expanded to the activation dtype, then a plain product."""
    from ..utils.quant_formats import dequantize
    y = x.float() @ dequantize(w, torch.float32).to(x.dtype).float().t()
    if bias is not None:
        y = y + bias.float()
    y = y.to(x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


def gemm_fp8(x, wq, w_scale, bias=None, out=None):
    """Oracle of the block-scaled fp8 GEMM: both operands rounded to e4m3 with their scales, product in fp32."""
    xq, sa = quant_act_fp8(x)
    T, K = x.shape
    xd = xq.float() * sa.t().repeat_interleave(128, 1)[:, :K]
    y = xd @ dequantize_weight_fp8_block128(wq, w_scale).t()
    if bias is not None:
        y = y + bias.float()
    y = y.to(x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


def norm_residual(x, residual, weight, eps, bias=None, out=None, weight_offset: float = 0.0, x_scale: float = 1.0,
                  layernorm: bool = False):
    h = x.float() * x_scale
    if residual is not None:
        h = h + residual.float()
        residual.copy_(h.to(residual.dtype))
        h = residual.float()
    if layernorm:
        mean = h.mean(-1, keepdim=True)
        var = (h * h).mean(-1, keepdim=True) - mean * mean
        y = (h - mean) * torch.rsqrt(var.clamp_min(0) + eps)
    else:
        y = h * torch.rsqrt((h * h).mean(-1, keepdim=True) + eps)
    y = y * (weight.float() + weight_offset)
    if bias is not None:
        y = y + bias.float()
    y = y.to(x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


def apply_rope(x, cos, sin, rot):
    """x: [T, heads, d]; cos/sin: [T, rot/2].  Rotate-half convention on the first `rot` dims."""
    half = rot // 2
    x1, x2, rest = x[..., :half].float(), x[..., half:rot].float(), x[..., rot:]
    c, s = cos[:, None, :], sin[:, None, :]
    o1 = x1 * c - x2 * s
    o2 = x2 * c + x1 * s
    return torch.cat([o1.to(x.dtype), o2.to(x.dtype), rest], dim=-1)


def _to_e4m3_bytes(x, scale):
    """x / scale as e4m3 bytes, saturating at +-448 like the kernel."""
    return (x.float() / scale).clamp(-448.0, 448.0).to(torch.float8_e4m3fn).view(torch.uint8)


def rope_kvwrite(qkv, positions, cos_sin, kv_cache, slots, nh, nkv, d, rot, apply_rope_flag: bool = True, kv_scale=None):
    """In place on qkv [T, (nh+2nkv)*d]; kv_cache [blocks, nkv, 2, page, d] (bf16 / fp32, or e4m3 holding value / scale)."""
    T = qkv.shape[0]
    page = kv_cache.shape[3]
    q = qkv[:, : nh * d].view(T, nh, d)
    k = qkv[:, nh * d: (nh + nkv) * d].view(T, nkv, d)
    v = qkv[:, (nh + nkv) * d: (nh + 2 * nkv) * d].view(T, nkv, d)
    if apply_rope_flag:
        cs = cos_sin[positions.long()]
        cos, sin = cs[:, : rot // 2], cs[:, rot // 2: rot]
        q.copy_(apply_rope(q, cos, sin, rot))
        k.copy_(apply_rope(k, cos, sin, rot))
    if slots is not None:
        ok = slots >= 0
        s = slots[ok].long()
        blk, off = s // page, s % page
        if kv_cache.dtype == torch.float8_e4m3fn:
            ks, vs = kv_scale or (1.0, 1.0)
            raw = kv_cache.view(torch.uint8)
            raw[blk, :, 0, off, :] = _to_e4m3_bytes(k[ok], ks)
            raw[blk, :, 1, off, :] = _to_e4m3_bytes(v[ok], vs)
        else:
            kv_cache[blk, :, 0, off, :] = k[ok]
            kv_cache[blk, :, 1, off, :] = v[ok]


def _act(x, act):
    if act in ("silu", "swish"):
        return F.silu(x)
    if act == "gelu":
        return F.gelu(x)
    if act in ("gelu_new", "gelu_pytorch_tanh", "gelu_fast", "gelu_tanh"):
        return F.gelu(x, approximate="tanh")
    if act == "relu":
        return F.relu(x)
    if act == "relu2":
        return F.relu(x).square()
    raise ValueError(act)


CLAMPED_SWIGLU_ALPHA = 1.702


def act_mul(x, inter, act="silu", gated=True, out=None, limit: float = 0.0):
    """act(gate) * up of rows [gate | up], or act(gate).  "clamped_swiglu" (gated): gate at most `limit`, up within +-limit,
    gate * sigmoid(1.702 gate) * (up + 1)."""
    g = x[:, :inter].float()
    if act == "clamped_swiglu":
        g = g.clamp(max=limit)
        g = g * torch.sigmoid(CLAMPED_SWIGLU_ALPHA * g) * (x[:, inter: 2 * inter].float().clamp(-limit, limit) + 1.0)
    else:
        g = _act(g, act)
        if gated:
            g = g * x[:, inter: 2 * inter].float()
    g = g.to(x.dtype)
    if out is not None:
        out.copy_(g)
        return out
    return g


def embed(ids, table, v0=0, v1=None, mult=1.0, out=None):
    if v1 is None:
        v1 = v0 + table.shape[0]
    idl = ids.long()
    ok = (idl >= v0) & (idl < v1)
    y = table[(idl - v0).clamp(0, table.shape[0] - 1)]
    if mult != 1.0:
        y = (y.float() * mult).to(table.dtype)
    y = torch.where(ok[:, None], y, torch.zeros_like(y))
    if out is not None:
        out.copy_(y)
        return out
    return y


def argmax_logprob(logits, ids=None, logprobs=None, softcap: float = 0.0):
    x = logits.float()
    if softcap > 0:
        x = softcap * torch.tanh(x / softcap)
    i = x.argmax(-1)
    lp = torch.log_softmax(x, -1).gather(1, i[:, None])[:, 0]
    if ids is not None:
        ids.copy_(i.to(ids.dtype))
        logprobs.copy_(lp)
        return ids, logprobs
    return i.to(torch.int32), lp


def advance_decode(input_ids, next_ids, positions, ctx_lens, slots, block_tables, page):
    live = ctx_lens > 0
    input_ids[live] = next_ids[live].to(input_ids.dtype)
    positions[live] += 1
    ctx_lens[live] = positions[live] + 1
    pos = positions.long()
    blk = block_tables.gather(1, (pos // page).clamp(0, block_tables.shape[1] - 1)[:, None])[:, 0]
    new_slots = blk * page + (pos % page).to(blk.dtype)
    slots.copy_(torch.where(live, new_slots.to(slots.dtype), torch.full_like(slots, -1)))


def prefill_metadata(cu_q, cache_lens, seq_slot, block_tables, page, T):
    """-> (positions [T], slots [T], tok_slot [T]) int32 of a ragged prefill whose sequence b owns tokens [cu_q[b], cu_q[b+1])."""
    t = torch.arange(T, device=cu_q.device)
    b = torch.searchsorted(cu_q[1:].long().contiguous(), t, right=True).clamp(max=cache_lens.shape[0] - 1)
    pos = cache_lens.long()[b] + (t - cu_q.long()[b])
    blk = (pos // page).clamp(max=block_tables.shape[1] - 1)
    slots = block_tables.long()[b, blk] * page + pos % page
    return pos.to(torch.int32), slots.to(torch.int32), seq_slot[b].to(torch.int32)


def _gather_kv(kv_cache, block_table, n_keys, kvh, kv_scale=None):
    """-> K [n_keys, d], V [n_keys, d] for one sequence and kv head."""
    page = kv_cache.shape[3]
    nblk = (n_keys + page - 1) // page
    blocks = block_table[:nblk].long()
    if kv_cache.dtype == torch.float8_e4m3fn:
        ks, vs = kv_scale or (1.0, 1.0)
        raw = kv_cache.view(torch.uint8)
        k = raw[blocks, kvh, 0].reshape(-1, kv_cache.shape[-1])[:n_keys].view(torch.float8_e4m3fn).float() * ks
        v = raw[blocks, kvh, 1].reshape(-1, kv_cache.shape[-1])[:n_keys].view(torch.float8_e4m3fn).float() * vs
        return k, v
    k = kv_cache[blocks, kvh, 0].reshape(-1, kv_cache.shape[-1])[:n_keys]
    v = kv_cache[blocks, kvh, 1].reshape(-1, kv_cache.shape[-1])[:n_keys]
    return k, v


def _attend(q, k, v, q_pos, scale, window, softcap, slope=None):
    """q: [nq, d] at absolute positions q_pos [nq]; k, v: [nk, d] at positions 0..nk-1.  `slope` (scalar or [nq]) adds the
    ALiBi bias -slope * (query position - key position)."""
    s = (q.float() @ k.float().t()) * scale
    if softcap and softcap > 0:
        s = softcap * torch.tanh(s / softcap)
    kp = torch.arange(k.shape[0], device=q.device)[None, :]
    if slope is not None:
        sl = slope if torch.is_tensor(slope) and slope.dim() else torch.as_tensor(slope, device=q.device).reshape(1)
        s = s - sl.float().reshape(-1, 1) * (q_pos[:, None] - kp).float()
    mask = kp <= q_pos[:, None]
    if window and window > 0:
        mask &= kp > (q_pos[:, None] - window)
    s = s.masked_fill(~mask, float("-inf"))
    p = torch.softmax(s, -1)
    p = torch.nan_to_num(p, nan=0.0)
    return p @ v.float()


def attn_decode(q, kv_cache, block_tables, ctx_lens, nh, nkv, d, scale, window=0, softcap=0.0, nsplit=1, out=None, alibi=None,
                kv_scale=None):
    T = q.shape[0]
    res = torch.zeros(T, nh * d, dtype=q.dtype, device=q.device)
    g = nh // nkv
    for t in range(T):
        n = int(ctx_lens[t])
        if n <= 0:
            continue
        for kvh in range(nkv):
            k, v = _gather_kv(kv_cache, block_tables[t], n, kvh, kv_scale)
            qh = q[t, kvh * g * d: (kvh + 1) * g * d].view(g, d)
            o = _attend(qh, k, v, torch.full((g,), n - 1, device=q.device), scale, window, softcap,
                        None if alibi is None else alibi[kvh * g: (kvh + 1) * g])
            res[t, kvh * g * d: (kvh + 1) * g * d] = o.reshape(-1).to(q.dtype)
    if out is not None:
        out.copy_(res)
        return out
    return res


def attn_prefill(q, kv_cache, block_tables, cu_q, cache_lens, tile_seq, tile_q0, nh, nkv, d, scale, window=0, softcap=0.0,
                 out=None, alibi=None, kv_scale=None):
    T = q.shape[0]
    res = torch.zeros(T, nh * d, dtype=q.dtype, device=q.device)
    g = nh // nkv
    B = cache_lens.shape[0]
    for b in range(B):
        s, e = int(cu_q[b]), int(cu_q[b + 1])
        if e <= s:
            continue
        c = int(cache_lens[b])
        n = c + (e - s)
        pos = torch.arange(c, n, device=q.device)
        for kvh in range(nkv):
            k, v = _gather_kv(kv_cache, block_tables[b], n, kvh, kv_scale)
            for gi in range(g):
                h = kvh * g + gi
                o = _attend(q[s:e, h * d: (h + 1) * d], k, v, pos, scale, window, softcap, None if alibi is None else alibi[h])
                res[s:e, h * d: (h + 1) * d] = o.to(q.dtype)
    if out is not None:
        out.copy_(res)
        return out
    return res


def prefill_tiles(q_lens, tile: int = 64):
    """Host-side tile map for attn_prefill: (tile_seq, tile_q0) int32 lists."""
    seq, q0 = [], []
    for b, n in enumerate(q_lens):
        for s in range(0, n, tile):
            seq.append(b)
            q0.append(s)
    return seq, q0


def context_offsets(cache_lens, q_lens, window: int = 0):
    """First rows of the sequences' contexts laid end to end, and their total: what precedes a portion of q tokens and can be seen from
    it, then the portion (window: at most window - 1 tokens precede it)."""
    off = [0]
    for c, n in zip(cache_lens, q_lens):
        off.append(off[-1] + (min(c, window - 1) if window else c) + n)
    return off


def lora_shrink(x, tok_slot, arena, slot_base, slot_rank, unit_off, nparts, max_rank, v=None):
    T, K = x.shape
    if v is None:
        v = torch.zeros(T, nparts * max_rank, dtype=torch.float32, device=x.device)
    for t in range(T):
        s = int(tok_slot[t])
        if s < 0 or int(slot_base[s]) < 0:
            continue
        r = int(slot_rank[s])
        off = int(slot_base[s]) + r * unit_off
        A = arena[off: off + nparts * r * K].view(nparts * r, K)
        v[t, : nparts * r] = x[t].float() @ A.float().t()
    return v


def lora_expand(v, tok_slot, arena, slot_base, slot_rank, unit_off, y, n0, n1):
    T, N = y.shape
    bounds = [0, n0, n1, N]
    for t in range(T):
        s = int(tok_slot[t])
        if s < 0 or int(slot_base[s]) < 0:
            continue
        r = int(slot_rank[s])
        off = int(slot_base[s]) + r * unit_off
        B = arena[off: off + N * r].view(N, r).float()
        delta = torch.zeros(N, dtype=torch.float32, device=y.device)
        for part in range(3):
            a, b = bounds[part], bounds[part + 1]
            if b > a:
                delta[a:b] = B[a:b] @ v[t, part * r: (part + 1) * r].float()
        y[t] = (y[t].float() + delta).to(y.dtype)


def lora_shrink_tiles(x, tiles, num_tiles, max_tile_rows, arena, slot_base, slot_rank, unit_off, nparts, max_rank, v=None):
    """Tile-table form (tiles: int32 [n, 4] = slot, row0, nrows, -).  The CPU oracle reads A_cat straight from the
    arena; the CUDA kernel reads the same bytes through the per-slot tensor maps."""
    T, K = x.shape
    if v is None:
        v = torch.zeros(T, nparts * max_rank, dtype=torch.float32, device=x.device)
    for i in range(num_tiles):
        s, row0, n, _ = (int(q) for q in tiles[i])
        n = min(n, T - row0)                 # a table may be older than the batch: rows past T are gone
        if s < 0 or n <= 0 or int(slot_base[s]) < 0:
            continue
        r = int(slot_rank[s])
        off = int(slot_base[s]) + r * unit_off
        A = arena[off: off + nparts * r * K].view(nparts * r, K).float()
        v[row0:row0 + n, : nparts * r] = x[row0:row0 + n].float() @ A.t()
    return v


def lora_expand_tiles(v, tiles, num_tiles, max_tile_rows, arena, slot_base, slot_rank, unit_off, y, n0, n1):
    T, N = y.shape
    bounds = [0, n0, n1, N]
    for i in range(num_tiles):
        s, row0, n, _ = (int(q) for q in tiles[i])
        n = min(n, T - row0)
        if s < 0 or n <= 0 or int(slot_base[s]) < 0:
            continue
        r = int(slot_rank[s])
        off = int(slot_base[s]) + r * unit_off
        B = arena[off: off + N * r].view(N, r).float()
        delta = torch.zeros(n, N, dtype=torch.float32, device=y.device)
        for part in range(3):
            a, b = bounds[part], bounds[part + 1]
            if b > a:
                delta[:, a:b] = v[row0:row0 + n, part * r:(part + 1) * r].float() @ B[a:b].t()
        y[row0:row0 + n] = (y[row0:row0 + n].float() + delta).to(y.dtype)


def build_lora_tiles(slots_per_row, max_rows: int):
    """Host helper: rows with equal adapter slot that are adjacent form a segment; segments are cut into tiles of at
    most `max_rows` rows.  -> list of (slot, row0, nrows, 0); rows without adapter (slot < 0) get no tile."""
    tiles = []
    i, n = 0, len(slots_per_row)
    while i < n:
        s = slots_per_row[i]
        j = i
        while j < n and slots_per_row[j] == s:
            j += 1
        if s >= 0:
            for a in range(i, j, max_rows):
                tiles.append((s, a, min(max_rows, j - a), 0))
        i = j
    return tiles


def rope_cache(rot: int, max_pos: int, theta: float, scaling: Optional[dict] = None, device="cpu") -> torch.Tensor:
    """[max_pos, rot] fp32 table: cos in the first half, sin in the second.

    Scaling variants follow `server/lorax_server/utils/layers.py:484-816` of the reference: linear,
    dynamic NTK, YaRN, Su/LongRoPE and llama3.
    """
    inv_freq = 1.0 / (theta ** (torch.arange(0, rot, 2, dtype=torch.float32) / rot))
    mscale = 1.0
    t = torch.arange(max_pos, dtype=torch.float32)
    if scaling:
        kind = scaling.get("rope_type", scaling.get("type", "default"))
        factor = float(scaling.get("factor", 1.0))
        if kind == "linear":
            t = t / factor
        elif kind == "dynamic":
            orig = int(scaling.get("original_max_position_embeddings", max_pos))
            if max_pos > orig:
                base = theta * ((factor * max_pos / orig) - (factor - 1)) ** (rot / (rot - 2))
                inv_freq = 1.0 / (base ** (torch.arange(0, rot, 2, dtype=torch.float32) / rot))
        elif kind == "llama3":
            low = float(scaling.get("low_freq_factor", 1.0))
            high = float(scaling.get("high_freq_factor", 4.0))
            orig = float(scaling.get("original_max_position_embeddings", 8192))
            wavelen = 2 * math.pi / inv_freq
            smooth = ((orig / wavelen) - low) / (high - low)
            scaled = torch.where(wavelen > orig / low, inv_freq / factor, inv_freq)
            mid = (wavelen <= orig / low) & (wavelen >= orig / high)
            inv_freq = torch.where(mid, (1 - smooth) * inv_freq / factor + smooth * inv_freq, scaled)
        elif kind == "yarn":
            orig = float(scaling.get("original_max_position_embeddings", 4096))
            beta_fast, beta_slow = float(scaling.get("beta_fast", 32)), float(scaling.get("beta_slow", 1))

            def corr_dim(nrot):
                return (rot * math.log(orig / (nrot * 2 * math.pi))) / (2 * math.log(theta))

            lo = max(math.floor(corr_dim(beta_fast)), 0)
            hi = min(math.ceil(corr_dim(beta_slow)), rot - 1)
            ramp = ((torch.arange(rot // 2, dtype=torch.float32) - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
            inv_mask = 1 - ramp
            inv_freq = (inv_freq / factor) * (1 - inv_mask) + inv_freq * inv_mask
            mscale = float(scaling.get("attention_factor") or (0.1 * math.log(factor) + 1.0 if factor > 1 else 1.0))
        elif kind in ("su", "longrope"):
            orig = int(scaling.get("original_max_position_embeddings", max_pos))
            ext = torch.tensor(scaling["long_factor"] if max_pos > orig else scaling["short_factor"], dtype=torch.float32)
            inv_freq = inv_freq / ext
            sc = max_pos / orig
            mscale = 1.0 if sc <= 1 else math.sqrt(1 + math.log(sc) / math.log(orig))
    freqs = torch.outer(t, inv_freq)
    return torch.cat([freqs.cos() * mscale, freqs.sin() * mscale], dim=-1).to(device)


# ------------------------------------------------------------------------------------------------
# Layer-by-layer designs (models/mixers.py): fp32 residual stream, linear recurrences with per-request state, latent attention.
# `inp` is the StepInputs of the step: rows [0, nd) are decode rows, the rows after them ragged prompt tokens.
# ------------------------------------------------------------------------------------------------
def rope_table(rot: int, max_pos: int, base: float, device="cpu", scaling=None) -> torch.Tensor:
    """[max_pos, rot] fp32: cos of position * base^(-2i / rot) in the first half, sin in the second; angles formed in fp64.  `scaling`
    (factor, original, fast, slow): YaRN, which divides the frequencies of pairs that turn less than `slow` times over `original`
    positions by `factor`, leaves those that turn more than `fast` times, goes linearly between, and multiplies cos and sin by
    0.1 ln(factor) + 1.  `scaling` (factor, original, low, high): bands as in Llama 3.1, which divides the frequencies of pairs that turn less
    than `low` times over `original` positions by `factor`, leaves those that turn more than `high` times, and blends between."""
    f = torch.pow(torch.tensor(float(base), dtype=torch.float64), -torch.arange(0, rot, 2, dtype=torch.float64) / rot)
    mult = 1.0
    if scaling and "high" in scaling:
        factor, low, high = float(scaling["factor"]), float(scaling["low"]), float(scaling["high"])
        turns = float(scaling["original"]) * f / (2 * math.pi)
        keep = ((turns - low) / (high - low)).clamp(0, 1) if high != low else (turns >= low).double()
        f = torch.where(turns > high, f, torch.where(turns < low, f / factor, (1 - keep) * f / factor + keep * f))
    elif scaling:
        factor, original = float(scaling["factor"]), float(scaling["original"])
        pair = lambda turns: rot * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(pair(scaling["fast"])), 0), min(math.ceil(pair(scaling["slow"])), rot - 1)
        ramp = ((torch.arange(rot // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        f = f / factor * ramp + f * (1 - ramp)
        mult = 0.1 * math.log(factor) + 1.0
    a = torch.outer(torch.arange(max_pos, dtype=torch.float64), f)
    return (torch.cat([a.cos(), a.sin()], -1) * mult).float().to(device)


def _tokens_before(ids, pages, inp):
    """The token in front of every row's (-1: none), from the step itself or, in front of a sequence's first row, from the pages of token
    ids [blocks, page]; the step's own ids are left there."""
    T, page = ids.shape[0], pages.shape[1]
    prev = torch.full((T,), -1, dtype=torch.int64, device=ids.device)
    nd, dbt, _, ctx = inp.decode_view(T)
    spans = [(i, 1, dbt[i], int(ctx[i]) - 1) for i in range(nd) if int(ctx[i]) > 0]
    if inp.is_prefill:
        cu = [int(c) for c in inp.cu_q]
        spans += [(nd + cu[b], cu[b + 1] - cu[b], inp.block_tables[b], int(inp.cache_lens[b])) for b in range(len(cu) - 1) if cu[b + 1] > cu[b]]
    for r0, n, bt, before in spans:
        prev[r0 + 1: r0 + n] = ids[r0: r0 + n - 1].long()
        if before > 0:
            prev[r0] = pages[int(bt[(before - 1) // page]), (before - 1) % page].long()
    ok = inp.slots >= 0
    pages.view(-1)[inp.slots[ok].long()] = ids[ok].to(pages.dtype)
    return prev


def embed_stream(ids, table, mult=1.0, pos=None, positions=None, copy=None, bigram=None):
    """table[ids] * mult (+ pos[positions]) in fp32; `copy` takes the same values in its own dtype.  bigram = (vectors [buckets + 1, W],
    (buckets, mul_prev, mul_cur), pages of token ids, inp) adds the vector of (token before, token), the last one where none is before."""
    ids = ids.clamp(0, table.shape[0] - 1)
    x = table[ids.long().clamp(0, table.shape[0] - 1)].float() * mult
    if pos is not None:
        x = x + pos[positions.long().clamp(0, pos.shape[0] - 1)].float()
    if bigram is not None:
        vectors, (buckets, mul_prev, mul_cur), pages, inp = bigram
        prev = _tokens_before(ids, pages, inp)
        row = (prev * mul_prev + ids.long() * mul_cur) % buckets
        x = x + vectors[torch.where(prev < 0, torch.full_like(row, buckets), row)].float()
    if copy is not None:
        copy.copy_(x)
    return x


def _layer_norm(x, weight, bias, eps, n: int):
    """Layer norm over the first `n` columns; the padding behind them stays zero when weight and bias are zero there."""
    d = x - x[:, :n].mean(-1, keepdim=True)
    y = d * torch.rsqrt(d[:, :n].square().mean(-1, keepdim=True) + eps) * weight
    return y if bias is None else y + bias


def _weighted_rows(y, pairs, W: int):
    """Sum of every token's rows pos [T, k] (-1: none) of `y` with the weights w [T, k], in fp32."""
    pos, w = pairs
    return torch.einsum("tk,tkw->tw", torch.where(pos >= 0, w, torch.zeros_like(w)), y[pos.long().clamp(min=0)][:, :, :W].float())


def norm_add(residual, y, weight, bias, mult: float, eps, n: int, dtype, layernorm: bool = True, pairs=None, gate=None, next_weight=None,
             rows=None):
    """residual (fp32, in place) += mult * norm(y) over the first `n` columns; returns the new residual in `dtype`.  With `pairs` =
    (pos [T, k], w [T, k]) a token's y is the weighted sum of its rows pos (-1: none) of `y`.  gate [T, W]: y times its sigmoid.
    next_weight [W]: returns the new residual's RMS norm with this weight instead, of `rows` only when given (whether the residual's other
    rows still take the addition is open)."""
    W = residual.shape[1]
    x = y[:, :W].float() if pairs is None else _weighted_rows(y, pairs, W)
    if gate is not None:
        x = x * torch.sigmoid(gate[:, :W].float())
    if layernorm:
        x = _layer_norm(x, weight, bias, eps, n)
    else:
        x = x * torch.rsqrt((x * x).sum(-1, keepdim=True) / n + eps) * weight
        if bias is not None:
            x = x + bias
    residual += mult * x
    if next_weight is not None:
        return norm_stream(residual, None, next_weight, eps, 0.0, n, dtype, rows=rows)
    return residual if dtype == torch.float32 else residual.to(dtype)


def norm_stream(residual, pending, weight, eps, weight_offset: float, n: int, dtype, bias=None, layernorm: bool = False, rows=None, pairs=None):
    """residual (fp32, in place) += pending, with `pairs` a weighted sum of its rows as in `norm_add`; returns its RMS or layer norm (mean
    over the first `n` columns) in `dtype`, of `rows` only when given (whether the residual's other rows still take the addition is
    open: only the last norm of a pass takes `rows`)."""
    if pending is not None:
        residual += pending.float() if pairs is None else _weighted_rows(pending, pairs, residual.shape[1])
    if rows is not None:
        residual = residual[rows.long()]
    if layernorm:
        return _layer_norm(residual, weight + weight_offset, bias, eps, n).to(dtype)
    y = residual * torch.rsqrt((residual * residual).sum(-1, keepdim=True) / n + eps)
    return (y * (weight + weight_offset)).to(dtype)


def norm_gate(x, group: int, n: int, weight, gate, act: str, eps, out):
    """x [T, G * group] fp32: every group of columns divided by its root mean square (over `n` real columns), times `weight`
    [G * group], times act(gate); written to `out` in its dtype."""
    T, C = x.shape
    g = x.view(T, C // group, group)
    y = (g * torch.rsqrt((g * g).sum(-1, keepdim=True) / n + eps)).view(T, C) * weight
    z = gate[:, :C].float()
    y = y * (torch.sigmoid(z) if act == "sigmoid" else F.silu(z))
    out[:, :C] = y.to(out.dtype)
    return out


def _sequences(inp, T: int):
    """(first row, rows, state slot, tokens before the step) of every live sequence of the step."""
    nd, _, slots, ctx = inp.decode_view(T)
    out = [(i, 1, int(slots[i]), int(ctx[i]) - 1) for i in range(nd) if int(ctx[i]) > 0]
    if inp.is_prefill:
        cu = [int(c) for c in inp.cu_q]
        out += [(nd + cu[b], cu[b + 1] - cu[b], int(inp.state_slots[b]), int(inp.cache_lens[b])) for b in range(len(cu) - 1)
                if cu[b + 1] > cu[b]]
    return out


def linear_attn(q, k, v, H: int, d: int, dv: int, decay, state, inp):
    """Linear attention with one decay per head over silu(q), silu(k), silu(v) (row-strided views [T, H * d / dv]):
    S <- decay S + k v^T, o = S^T q.  `state` [slots, H, d, dv] fp32 is read and updated.  -> o [T, H * dv] fp32."""
    T = q.shape[0]
    qf, kf = F.silu(q.float()).view(T, H, d), F.silu(k.float()).view(T, H, d)
    vf = F.silu(v.float()).view(T, H, dv)
    if q.dtype != torch.float32:
        qf, kf, vf = (x.to(q.dtype).float() for x in (qf, kf, vf))
    out = torch.zeros(T, H * dv, dtype=torch.float32, device=q.device)
    for r0, n, slot, before in _sequences(inp, T):
        S = state[slot].clone() if before > 0 else torch.zeros_like(state[slot])
        for t in range(r0, r0 + n):
            S = decay[:, None, None] * S + kf[t][:, :, None] * vf[t][:, None, :]
            out[t] = torch.einsum("hij,hi->hj", S, qf[t]).reshape(-1)
        state[slot] = S
    return out


def token_shift(h, mu, shift, inp):
    """Interpolation with the previous token's input: row s of the result [n, T, W] is h + (h' - h) * mu[s]; h' of a sequence's
    first token comes from `shift` [slots, W] (zeros at position 0), which then takes the sequence's last row."""
    T = h.shape[0]
    prev = torch.zeros_like(h)
    last = []
    for r0, n, slot, before in _sequences(inp, T):
        prev[r0 + 1: r0 + n] = h[r0: r0 + n - 1]
        if before > 0:
            prev[r0] = shift[slot]
        last.append((slot, r0 + n - 1))
    for slot, r in last:
        shift[slot] = h[r]
    hf, pf = h.float(), prev.float()
    return torch.stack([(hf + (pf - hf) * mu[s]).to(h.dtype) for s in range(mu.shape[0])])


def gemm_stack(x, w):
    """x [n, T, K], w [n, N, K] -> [n, T, N]: one product per stacked pair."""
    return torch.stack([gemm(x[i], w[i]) for i in range(w.shape[0])])


def tanh_(x):
    x.copy_(torch.tanh(x.float()).to(x.dtype))
    return x


def wkv(r, k, v, z, w0, u, H: int, d: int, state, inp):
    """WKV recurrence with data-dependent decay w = exp(-exp(z + w0)) per key channel and a bonus u for the current token:
    o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T.  -> o [T, H * d] fp32; `state` [slots, H, d, d] is updated."""
    T = r.shape[0]
    rf, kf, vf = (x.float().reshape(T, H, d) for x in (r, k, v))
    w = torch.exp(-torch.exp(z.float() + w0)).view(T, H, d)
    out = torch.zeros(T, H * d, dtype=torch.float32, device=r.device)
    for r0, n, slot, before in _sequences(inp, T):
        S = state[slot].clone() if before > 0 else torch.zeros_like(state[slot])
        for t in range(r0, r0 + n):
            kv = kf[t][:, :, None] * vf[t][:, None, :]
            out[t] = torch.einsum("hij,hi->hj", S + u.view(H, d)[:, :, None] * kv, rf[t]).reshape(-1)
            S = w[t][:, :, None] * S + kv
        state[slot] = S
    return out


def _rotate_pairs(x, cos, sin):
    """x [..., rot] with interleaved pairs; cos / sin broadcastable [..., rot / 2]."""
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    return torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)


def latent_prep(dq, dkv, dq_norm, dkv_norm, q_rank: int, kv_rank: int, rot: int, eps, cos_sin, positions, slots, cache, q=None, heads: int = 0,
                head: int = 0, off: int = 0):
    """Down-projections of latent attention -> normalised query latent [T, q_rank padded] (returned) and cache rows
    [normalised key/value latent | rotated key part] (scattered into `cache` [blocks, page, kv_rank padded + rot padded]).  Without a query
    latent (dq None) the columns [off, off + rot) of every head of q [T, heads * head] are rotated in place."""
    dt = dkv.dtype
    kr = dkv_norm.shape[0]
    page = cache.shape[1]

    def rms(x, n, w):
        x = x.float()
        return (x * torch.rsqrt((x * x).sum(-1, keepdim=True) / n + eps) * w).to(dt)
    cq = rms(dq[:, : dq_norm.shape[0]], q_rank, dq_norm) if dq is not None else None
    if q is not None:
        rope_pairs(q, positions, cos_sin, heads, head, off, rot)
    row = torch.zeros(dkv.shape[0], cache.shape[2], dtype=dt, device=dkv.device)
    row[:, :kr] = rms(dkv[:, :kr], kv_rank, dkv_norm)
    cs = cos_sin[positions.long()]
    row[:, kr: kr + rot] = _rotate_pairs(dkv[:, kr: kr + rot], cs[:, : rot // 2], cs[:, rot // 2:]).to(dt)
    ok = slots >= 0
    s = slots[ok].long()
    cache[s // page, s % page] = row[ok]
    return cq


def rope_pairs(x, positions, cos_sin, H: int, head: int, off: int, rot: int):
    """Rotates columns [off, off + rot) of every head (width `head`) of x [T, H * head] in place, interleaved pairs."""
    T = x.shape[0]
    cs = cos_sin[positions.long()]
    part = x[:, : H * head].unflatten(1, (H, head))[:, :, off: off + rot]
    part.copy_(_rotate_pairs(part, cs[:, None, : rot // 2], cs[:, None, rot // 2:]).to(x.dtype))


def gemm_heads(x, w, out, x_head: int, gate=None, wide_gate: bool = False):
    """Per-head products: head h of `out` (width N) = columns [h * x_head, h * x_head + K) of x times w[h]^T (w [H, N, K]),
    optionally times sigmoid(gate[:, h]), or (wide_gate) times sigmoid of the gate column of every output column."""
    H, N, K = w.shape
    T = x.shape[0]
    xs = torch.stack([x[:, h * x_head: h * x_head + K] for h in range(H)], 1).float()
    y = torch.einsum("thk,hnk->thn", xs, w.float())
    if gate is not None:
        z = torch.sigmoid(gate[:, : H * N if wide_gate else H].float())
        y = y * (z.view(T, H, N) if wide_gate else z[:, :, None])
    out[:, : H * N] = y.reshape(T, H * N).to(out.dtype)
    return out


def latent_prefill(q, cache, w_ukv, gate, out, H: int, dk: int, rot: int, dv: int, scale: float, inp, nd: int, window: int = 0,
                   wide_gate: bool = False) -> bool:
    """The expanded form of prompt attention exists on the device only; False sends the rows through `latent_attn`."""
    return False


def latent_attn(q_lat, q, cache, H: int, kv_rank: int, head: int, rot_off: int, rot: int, scale: float, inp, window: int = 0):
    """Causal softmax attention in the latent space: head h's query is [q_lat[h] | q[h, rot_off : rot_off + rot]] against the
    cached rows [latent | rotated key], the last `window` of them (0: all).  -> weighted latents [T, H * kv_rank]."""
    T = q.shape[0]
    page = cache.shape[1]
    nd, dbt, _, ctx = inp.decode_view(T)
    ql, qr = q_lat.view(T, H, kv_rank).float(), q[:, : H * head].unflatten(1, (H, head))[:, :, rot_off: rot_off + rot].float()
    out = torch.zeros(T, H, kv_rank, dtype=q.dtype, device=q.device)
    spans = [(i, 1, dbt[i], int(ctx[i]) - 1) for i in range(nd) if int(ctx[i]) > 0]
    if inp.is_prefill:
        cu = [int(c) for c in inp.cu_q]
        spans += [(nd + cu[b], cu[b + 1] - cu[b], inp.block_tables[b], int(inp.cache_lens[b])) for b in range(len(cu) - 1) if cu[b + 1] > cu[b]]
    for r0, n, bt, before in spans:
        keys = before + n
        rows = cache[bt[: (keys + page - 1) // page].long()].reshape(-1, cache.shape[2])[:keys].float()
        s = torch.einsum("thc,sc->hts", ql[r0: r0 + n], rows[:, :kv_rank]) + torch.einsum("thc,sc->hts", qr[r0: r0 + n], rows[:, kv_rank: kv_rank + rot])
        pos, kp = torch.arange(before, keys, device=q.device)[:, None], torch.arange(keys, device=q.device)[None, :]
        hidden = kp > pos
        if window > 0:
            hidden |= kp <= pos - window
        s = (s * scale).masked_fill(hidden, float("-inf"))
        out[r0: r0 + n] = torch.einsum("hts,sc->thc", torch.softmax(s, -1), rows[:, :kv_rank]).to(q.dtype)
    return out.view(T, H * kv_rank)


def _conv_rows(x, w, state, inp):
    """Depthwise causal convolution of the step's rows: y_t = sum_j w[j] * u_(t - taps + 1 + j), u the rows of the sequence, zeros in
    front of it.  w [taps, C]; `state` [slots, taps - 1, C] holds the sequences' last rows and takes the new ones.  -> fp32 [T, C]"""
    T, taps = x.shape[0], w.shape[0]
    out = torch.zeros(T, x.shape[1], dtype=torch.float32, device=x.device)
    for r0, n, slot, before in _sequences(inp, T):
        u = x[r0: r0 + n]
        if taps > 1:
            old = state[slot] if before > 0 else torch.zeros_like(state[slot])
            u = torch.cat([old, u])
            state[slot] = u[u.shape[0] - (taps - 1):].clone()
        for j in range(taps):
            out[r0: r0 + n] += w[j] * u[j: j + n].float()
    return out


def causal_conv(x, w, b, act: str, state, inp):
    """act(convolution + b) of x [T, C] in x's dtype, in memory of its own."""
    y = _conv_rows(x, w, state, inp)
    if b is not None:
        y = y + b
    return (_act(y, act) if act else y).to(x.dtype)


def conv_rope_kvwrite(qkv, H: int, G: int, dk: int, dv: int, cos_sin, rot: int, positions, cache, inp, conv_w=None, conv_state=None):
    """Rows [q (H heads) | k (G) | v (G)] of padded widths dk, dk, dv (G 0: queries only), through the convolution when there is one:
    the first `rot` columns of every q and k head rotated in interleaved pairs, k and v to the cache.  -> q [T, H * dk], which without
    convolution is the front of `qkv` itself."""
    T = qkv.shape[0]
    x = qkv[:, : (H + G) * dk + G * dv].float() if conv_w is None else _conv_rows(qkv, conv_w, conv_state, inp)
    qk = x[:, : (H + G) * dk].reshape(T, H + G, dk).clone()
    if rot:
        cs = cos_sin[positions.long()]
        qk[:, :, :rot] = _rotate_pairs(qk[:, :, :rot], cs[:, None, : rot // 2], cs[:, None, rot // 2:])
    qk = qk.to(qkv.dtype)
    if G:
        page = cache.shape[2] // (dk + dv)
        ok = inp.slots >= 0
        s = inp.slots[ok].long()
        blk, off = s // page, s % page
        cache[:, :, : page * dk].view(cache.shape[0], G, page, dk)[blk, :, off] = qk[ok][:, H:]
        cache[:, :, page * dk:].view(cache.shape[0], G, page, dv)[blk, :, off] = x[ok][:, (H + G) * dk:].reshape(-1, G, dv).to(qkv.dtype)
    q = qk[:, :H].reshape(T, H * dk)
    if conv_w is None:
        qkv[:, : H * dk] = q
        return qkv[:, : H * dk]
    return q


def ssd(xbc, dt, H: int, G: int, n: int, p: int, dt_bias, A, D, state, inp):
    """Selective state space recurrence (Mamba-2) over rows [x (H heads of p) | B (G groups of n) | C (G)]: with s = softplus(dt + dt_bias)
    per token and head, S <- exp(A s) S + s B x^T, y = S^T C + D x.  `state` [slots, H, n, p] fp32 is read and updated.
    -> y [T, H * p] fp32"""
    T = xbc.shape[0]
    x = xbc[:, : H * p].float().reshape(T, H, p)
    B, C = (xbc[:, H * p + i * G * n: H * p + (i + 1) * G * n].float().reshape(T, G, n).repeat_interleave(H // G, 1) for i in (0, 1))
    s = F.softplus(dt[:, :H].float() + dt_bias)
    out = torch.zeros(T, H * p, dtype=torch.float32, device=xbc.device)
    for r0, rows, slot, before in _sequences(inp, T):
        S = state[slot].clone() if before > 0 else torch.zeros_like(state[slot])
        for t in range(r0, r0 + rows):
            S = torch.exp(A * s[t])[:, None, None] * S + (s[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
            out[t] = (torch.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * x[t]).reshape(-1)
        state[slot] = S
    return out


def gate_norm(y, z, H: int, p: int, parts: int, weight, eps, out):
    """y [T, H * p padded] fp32 times silu(z) (the same layout), the heads' real columns closed up to [T, H * p], every one of `parts`
    equal parts of a row divided by its root mean square, times `weight` [H * p]; columns of `out` behind them are zeroed."""
    T, pp = y.shape[0], y.shape[1] // H
    g = (y * F.silu(z[:, : H * pp].float())).view(T, H, pp)[:, :, :p].reshape(T, parts, -1)
    g = (g * torch.rsqrt(g.square().mean(-1, keepdim=True) + eps)).reshape(T, H * p) * weight
    out[:, : H * p] = g.to(out.dtype)
    out[:, H * p:] = 0
    return out


def _kv_planes(cache, blocks, dk: int, dv: int, keys: int):
    """Pages of a sequence -> K [keys, heads, dk], V [keys, heads, dv] (fp32)."""
    page = cache.shape[2] // (dk + dv)
    x = cache[blocks.long()].float()
    k = x[:, :, : page * dk].reshape(-1, cache.shape[1], page, dk).transpose(1, 2).reshape(-1, cache.shape[1], dk)
    v = x[:, :, page * dk:].reshape(-1, cache.shape[1], page, dv).transpose(1, 2).reshape(-1, cache.shape[1], dv)
    return k[:keys], v[:keys]


def qk_norm_kvwrite(qkv, H: int, G: int, dk: int, dv: int, n: int, q_norm, k_norm, eps, cache, slots, positions=None, cos_sin=None, v_cos_sin=None):
    """Rows [q (H heads) | k (G) | v (G)] of padded widths dk, dk, dv: q (in place) and k are divided by their root mean square over
    the first `n` columns of each head and multiplied by the norm's weight, and with cos_sin [P, rot] rotated in their first `rot` columns
    (interleaved pairs); with v_cos_sin v is rotated likewise.  k and v go to the cache."""
    T = qkv.shape[0]

    def turn(x, table):
        if table is None:
            return x
        rot, cs = table.shape[1], table[positions.long()][:, None]
        return torch.cat([_rotate_pairs(x[..., :rot], cs[..., : rot // 2], cs[..., rot // 2:]), x[..., rot:].float()], -1)

    def rms(x, heads, w):
        x = x.reshape(T, heads, dk).float()
        return turn(x * torch.rsqrt((x * x).sum(-1, keepdim=True) / n + eps) * w, cos_sin).to(qkv.dtype)
    q = rms(qkv[:, : H * dk], H, q_norm)
    qkv[:, : H * dk] = q.reshape(T, -1)
    k = rms(qkv[:, H * dk: (H + G) * dk], G, k_norm)
    v = turn(qkv[:, (H + G) * dk: (H + G) * dk + G * dv].reshape(T, G, dv), v_cos_sin).to(qkv.dtype)
    page = cache.shape[2] // (dk + dv)
    ok = slots >= 0
    s = slots[ok].long()
    blk, off = s // page, s % page
    cache[:, :, : page * dk].view(cache.shape[0], G, page, dk)[blk, :, off] = k[ok]
    cache[:, :, page * dk:].view(cache.shape[0], G, page, dv)[blk, :, off] = v[ok]


def gqa_attn(q, cache, H: int, G: int, dk: int, dv: int, scale: float, window: int, inp, out, softcap: float = 0.0, sink=None, gate=None,
             out_scale: float = 1.0, turn_back=None):
    """Softmax attention of a step's rows (queries in the first H * dk columns of q) over the cached keys and values; a token sees the
    last `window` tokens (0: all) including itself.  softcap: scores become cap * tanh(score / cap).  sink [H]: a score that counts in
    the denominator only.  turn_back [P, rot]: the first `rot` columns of every head's result are rotated back by the token's position
    (interleaved pairs).  The result is multiplied by `out_scale` and by sigmoid(gate) [T, H * dv].  -> out [T, H * dv]"""
    T = q.shape[0]
    page = cache.shape[2] // (dk + dv)
    nd, dbt, _, ctx = inp.decode_view(T)
    spans = [(i, 1, dbt[i], int(ctx[i]) - 1) for i in range(nd) if int(ctx[i]) > 0]
    if inp.is_prefill:
        cu = [int(c) for c in inp.cu_q]
        spans += [(nd + cu[b], cu[b + 1] - cu[b], inp.block_tables[b], int(inp.cache_lens[b])) for b in range(len(cu) - 1) if cu[b + 1] > cu[b]]
    out[:, : H * dv] = 0
    for r0, n, bt, before in spans:
        keys = before + n
        k, v = _kv_planes(cache, bt[: (keys + page - 1) // page], dk, dv, keys)
        pos, kp = torch.arange(before, keys, device=q.device)[:, None], torch.arange(keys, device=q.device)[None, :]
        hidden = kp > pos
        if window > 0:
            hidden |= kp <= pos - window
        qs = q[r0: r0 + n, : H * dk].reshape(n, G, H // G, dk).float()
        s = torch.einsum("tghd,sgd->ghts", qs, k) * scale
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(hidden, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.view(G, H // G, 1, 1).expand(-1, -1, n, 1)], -1)
        y = torch.einsum("ghts,sgd->tghd", torch.softmax(s, -1)[..., :keys], v).reshape(n, H, dv)
        if turn_back is not None:
            rot, cs = turn_back.shape[1], turn_back[before: keys][:, None]
            y = torch.cat([_rotate_pairs(y[..., :rot], cs[..., : rot // 2], -cs[..., rot // 2:]), y[..., rot:]], -1)
        y = y.reshape(n, H * dv) * out_scale
        if gate is not None:
            y = y * torch.sigmoid(gate[r0: r0 + n, : H * dv].float())
        out[r0: r0 + n, : H * dv] = y.to(out.dtype)
    return out


class MoeRouting(NamedTuple):
    topk_ids: torch.Tensor     # [T, k] int32
    topk_w: torch.Tensor       # [T, k + shared] fp32
    seg: torch.Tensor          # [experts + shared + 1] int32: rows of every expert in the sorted order
    pos: torch.Tensor          # [T, k + shared] int32: sorted row of (token, choice), -1 when the expert lives on another rank
    xg: torch.Tensor           # the tokens' rows in the sorted order; the rows of the shared experts are the same ones, held once


def moe_route(x, router_w, k: int, e0: int, e_local: int, experts=None, score: str = "softmax", correction=None, groups: int = 0,
              keep: int = 0, scale: float = 1.0, shared: int = 0, group_top: int = 2, renorm: bool = True, bias=None,
              shared_gate: bool = True) -> MoeRouting:
    """Routing of every token to `k` of the router's first `experts` rows by its scores, softmax over all of them or sigmoid (plus a
    correction that takes part in the choice only), within the best `keep` of `groups` groups (by the sum of a group's `group_top`
    largest; softmax: 1).  The weights are the scores, divided by their sum if `renorm`, times `scale`.  `bias` [experts] is added to the
    logits.  `shared` experts more take every token, with the weight sigmoid(router row `experts`), or without shared_gate one."""
    T, E = x.shape[0], experts or router_w.shape[0]
    z = x.float() @ router_w.float().t()
    if bias is not None:
        z[:, :E] += bias
    s = torch.softmax(z[:, :E], -1) if score == "softmax" else torch.sigmoid(z[:, :E])
    choice = s if correction is None else s + correction
    if groups:
        g = choice.view(T, groups, E // groups)
        best = g.topk(min(group_top, E // groups), -1).values.sum(-1).topk(keep, -1).indices
        kept = torch.zeros(T, groups, dtype=torch.bool, device=x.device).scatter_(1, best, True)
        choice = g.masked_fill(~kept[:, :, None], float("-inf")).reshape(T, E)
    ids = choice.topk(k, -1).indices
    w = s.gather(1, ids)
    if renorm:
        w = w / (w.sum(-1, keepdim=True) + (0.0 if score == "softmax" else 1e-20))
    w = w * scale
    local = ids - e0
    flat = torch.where((local >= 0) & (local < e_local), local, torch.full_like(local, e_local)).reshape(-1)
    order = torch.argsort(flat, stable=True)
    count = torch.bincount(flat, minlength=e_local + 1)[:e_local]
    total = int(count.sum())
    seg = [0] + torch.cumsum(count, 0).tolist() + [total + (i + 1) * T for i in range(shared)]
    pos = torch.empty_like(flat)
    pos[order] = torch.arange(flat.shape[0], device=x.device)
    pos = torch.where(flat < e_local, pos, torch.full_like(pos, -1)).view(T, k)
    xg = x[torch.div(order[:total], k, rounding_mode="floor")]
    if shared:
        t = torch.arange(T, device=x.device)
        pos = torch.cat([pos] + [(total + i * T + t)[:, None] for i in range(shared)], 1)
        w = torch.cat([w] + [torch.sigmoid(z[:, E: E + 1]) if shared_gate else torch.ones_like(w[:, :1])] * shared, 1)
        xg = torch.cat([xg, x])
    return MoeRouting(ids.to(torch.int32), w, torch.tensor(seg, dtype=torch.int32), pos.to(torch.int32), xg)


def moe_grouped_gemm(xg, w, seg, avg_rows: int, out=None, shared: int = 0, tokens: int = 0, act: str = ""):
    """out[q] = act(xg[q] @ w[e(q)]^T) for every sorted row q (e(q): the expert whose run [seg[e], seg[e + 1]) holds q).  The last
    `shared` experts all read the one set of `tokens` rows that stands where the first of them begins.  act "swiglu": the rows of w are
    gate and up in turn, and column i of the result is silu(column 2i) * column 2i + 1."""
    s = [int(v) for v in seg]
    n = len(s) - 1
    y = torch.zeros(s[-1], w.shape[1] // (2 if act == "swiglu" else 1), dtype=xg.dtype, device=xg.device)
    for e in range(n):
        back = max(0, e - (n - shared)) * tokens if shared else 0
        z = xg[s[e] - back: s[e + 1] - back].float() @ w[e].float().t()
        y[s[e]: s[e + 1]] = (F.silu(z[:, 0::2]) * z[:, 1::2] if act == "swiglu" else _act(z, act) if act else z).to(xg.dtype)
    return y
