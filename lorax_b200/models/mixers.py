"""Layers of designs that list their layers one by one, over an fp32 residual stream.  Four styles:

  parallel   a token mixer and an optional gated feed-forward side by side, both reading one RMS norm of the stream (`MixerLayer`)
  pre        the mixer, then the feed-forward (dense or routed experts), each reading an RMS norm of the stream of its own
             (`PreNormLayer`)
  post       the mixer, then the feed-forward (dense or routed experts), each reading the stream itself; the norm of its output is
             added to the stream (`PostNormLayer`)
  sandwich   the mixer, then the feed-forward, each reading an RMS norm of the stream of its own; its output, times the sigmoid of a
             projection of its input, goes through a second norm and is added (`SandwichLayer`)

A mixer declares its tensors (`shapes`), what it keeps per token or per request (`cache_shape`), which of its projections read the
layer's input (`in_parts`, one GEMM; in a parallel layer together with the feed-forward's gate and up projections) and its output
projection (`out_part`; in a parallel layer fused with the down projection into one GEMM: the sum of both sublayers is formed in the
accumulator).  All sizes are padded to
multiples of 16 with zero weights when the layer is loaded, so the kernels see aligned heads whatever the configuration says; a padded
channel stays exactly zero through every operation.

  lightning         linear attention, one constant decay per head, state [heads, dim, vdim] per request
  wkv               token-shifted linear recurrence with a data-dependent decay per key channel, state [heads, dim, dim] per request
                    plus the previous token's input
  latent_attention  softmax attention over a low-rank latent and one shared rotated key part per token, both paged; with or without a
                    low-rank query, a sliding window, an output gate per head or per element
  attention         grouped-query softmax attention over paged keys and values, with a choice of normed queries and keys, short
                    convolutions, rotation, rotated values, capped scores, sliding window, sink, output gate, keys and values of another
                    layer
  mamba2            selective state space recurrence behind a short convolution, state [heads, state, vdim] per request, gated norm
  parallel          two mixers that read the same rows, their outputs weighted and added
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

PAD = 16


def pad16(n: int) -> int:
    return (n + PAD - 1) // PAD * PAD


def _pad_to(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """Zero-pad every dimension at its end."""
    if tuple(t.shape) == tuple(shape):
        return t
    out = torch.zeros(*shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def pad_heads_rows(w: torch.Tensor, heads: int, d: int, K: int) -> torch.Tensor:
    """[heads * d, k] -> [heads * pad16(d), K]: every head's rows padded on their own."""
    return _pad_to(w.view(heads, d, -1), heads, pad16(d), K).reshape(heads * pad16(d), K)


def pad_heads_cols(w: torch.Tensor, heads: int, d: int, N: int) -> torch.Tensor:
    """[n, heads * d] -> [N, heads * pad16(d)]."""
    return _pad_to(w.view(w.shape[0], heads, d), N, heads, pad16(d)).reshape(N, heads * pad16(d))


def pad_heads_vec(v: torch.Tensor, heads: int, d: int) -> torch.Tensor:
    return _pad_to(v.reshape(heads, d), heads, pad16(d)).reshape(-1)


class Mixer:
    """Common part.  `get(name)` passed to `load` returns the checkpoint tensor of this mixer in fp32; `fin` brings a matrix to the
    model's dtype and device, `vec` a vector to fp32 on the device."""

    recurrent = False                                        # keeps something per request
    window = 0                                               # tokens that attention sees (0: all)
    gathers_context = False                                  # prompts are attended to over their contexts laid end to end
    parallelism = 1 << 20                                    # thread blocks that one sequence gives the recurrence kernels

    def __init__(self, params: dict, width: int):
        self.width, self.W = width, pad16(width)

    def shapes(self) -> Dict[str, Tuple[int, ...]]:
        raise NotImplementedError

    def in_parts(self, get) -> List[Tuple[str, torch.Tensor]]:
        """(name, [rows, W]) of the projections that read the layer's norm."""
        raise NotImplementedError

    def in_bias(self, get) -> Dict[str, torch.Tensor]:
        """Bias vectors [rows] of those that have one."""
        return {}

    def out_part(self, get) -> torch.Tensor:
        """Output projection [W, out_dim]."""
        raise NotImplementedError

    def load(self, get, fin, vec, model):
        raise NotImplementedError

    def cache_shape(self, model) -> dict:
        """{"paged": width per token}, {"kv": (heads, key width, value width)} and / or {"state": {name: (shape per request, dtype)}},
        {"share_layer": the layer whose entry this one reads}, or {"parts": {name: one of these}}."""
        raise NotImplementedError

    def run(self, model, h, proj, y, inp, cache):
        """Mixes the step's rows: h [T, W] the layer's norm, proj name -> view of the fused projection, y [T, out_dim] the result."""
        raise NotImplementedError


class LightningMixer(Mixer):
    recurrent = True

    def __init__(self, params: dict, width: int):
        super().__init__(params, width)
        self.H, self.d, self.dv = int(params["heads"]), int(params["dim"]), int(params["vdim"])
        self.decay_values = [float(x) for x in params["decay"]]
        if len(self.decay_values) != self.H:
            raise ValueError(f"{len(self.decay_values)} decays for {self.H} heads")
        self.dp, self.dvp = pad16(self.d), pad16(self.dv)
        self.out_dim = self.H * self.dvp
        self.parallelism = self.H * ((self.dvp + 63) // 64)

    def shapes(self):
        H, d, dv, w = self.H, self.d, self.dv, self.width
        return {"q": (H * d, w), "k": (H * d, w), "v": (H * dv, w), "g": (H * dv, w), "o": (w, H * dv), "norm": (H * dv,)}

    def in_parts(self, get):
        H, d, dv, W = self.H, self.d, self.dv, self.W
        return [(n, pad_heads_rows(get(n), H, dd, W)) for n, dd in (("q", d), ("k", d), ("v", dv), ("g", dv))]

    def out_part(self, get):
        return pad_heads_cols(get("o"), self.H, self.dv, self.W)

    def load(self, get, fin, vec, model):
        self.norm = vec(pad_heads_vec(get("norm"), self.H, self.dv))
        self.decay = vec(torch.tensor(self.decay_values, dtype=torch.float64))

    def cache_shape(self, model):
        return {"state": {"S": ((self.H, self.dp, self.dvp), torch.float32)}}

    def run(self, model, h, proj, y, inp, cache):
        ops = model.ops
        o = ops.linear_attn(proj["q"], proj["k"], proj["v"], self.H, self.dp, self.dvp, self.decay, cache["S"], inp)
        ops.norm_gate(o, self.out_dim, self.H * self.dv, self.norm, proj["g"], "sigmoid", model.eps, y)


class WkvMixer(Mixer):
    recurrent = True
    STREAMS = ("r", "k", "v", "g", "w")

    def __init__(self, params: dict, width: int):
        super().__init__(params, width)
        self.H, self.d = int(params["heads"]), int(params["dim"])
        self.dp = pad16(self.d)
        self.out_dim = self.H * self.dp
        self.parallelism = self.H * ((self.dp + 63) // 64)
        self.rank: Optional[int] = params.get("rank")      # of the decay's low-rank map; the checkpoint's own shape decides

    def shapes(self):
        hd, w, r = self.H * self.d, self.width, int(self.rank or max(16, self.width // 64))
        out = {"mu." + s: (w,) for s in self.STREAMS}
        out.update({s: (hd, w) for s in "rkvg"})
        out.update({"w1": (r, w), "w2": (hd, r), "w0": (hd,), "u": (self.H, self.d), "norm": (hd,), "o": (w, hd)})
        return out

    def in_parts(self, get):
        return []                                           # every projection reads a shifted mix of its own

    def out_part(self, get):
        return pad_heads_cols(get("o"), self.H, self.d, self.W)

    def load(self, get, fin, vec, model):
        H, d, W = self.H, self.d, self.W
        self.mu = vec(torch.stack([_pad_to(get("mu." + s), W) for s in self.STREAMS]))
        self.rkvg = fin(torch.stack([pad_heads_rows(get(s), H, d, W) for s in "rkvg"]))          # [4, H * dp, W]
        w1, w2 = get("w1"), get("w2")
        rp = pad16(w1.shape[0])
        self.w1 = fin(_pad_to(w1, rp, W))
        self.w2 = fin(pad_heads_rows(w2, H, d, rp))
        self.w0 = vec(pad_heads_vec(get("w0"), H, d))
        self.u = vec(pad_heads_vec(get("u"), H, d))
        self.norm = vec(pad_heads_vec(get("norm"), H, d))

    def cache_shape(self, model):
        return {"state": {"S": ((self.H, self.dp, self.dp), torch.float32), "shift": ((self.W,), model.dtype)}}

    def run(self, model, h, proj, y, inp, cache):
        ops = model.ops
        mix = ops.token_shift(h, self.mu, cache["shift"], inp)                 # [5, T, W]
        r, k, v, g = ops.gemm_stack(mix[:4], self.rkvg)
        z = ops.gemm(ops.tanh_(ops.gemm(mix[4], self.w1)), self.w2)
        o = ops.wkv(r, k, v, z, self.w0, self.u, self.H, self.dp, cache["S"], inp)
        ops.norm_gate(o, self.dp, self.d, self.norm, g, "silu", model.eps, y)


class LatentAttentionMixer(Mixer):
    """What a design has of the following is a parameter:

      q_rank      queries come from a normed latent of this rank of their own (none: from the layer's input)
      mask.size   token i sees the last `size` tokens including itself (no mask: all before it)
      rot_layout  "interleaved": pairs of neighbours; "halves": dimension i with i + rot_dim / 2.  Scores do not change when the rotated
                  dimensions of queries and keys are put in another order, so halves are brought to pairs when the weights are loaded
      gate        the heads times sigmoid of a projection of the input: one number per "head" or one per "element" """

    gathers_context = True

    def __init__(self, params: dict, width: int):
        super().__init__(params, width)
        p = params
        self.H, self.d, self.rot, self.dv = int(p["heads"]), int(p["dim"]), int(p["rot_dim"]), int(p["vdim"])
        self.q_rank, self.kv_rank, self.scale = int(p.get("q_rank") or 0), int(p["kv_rank"]), float(p["scale"])
        self.rot_spec, mask = p["rot"], p.get("mask")
        if int(self.rot_spec.get("dims", self.rot)) != self.rot:
            raise NotImplementedError("latent attention rotates the whole rotated key part")
        if self.rot % 2:
            raise ValueError(f"rotation of {self.rot} dimensions")
        self.window = int(mask["size"]) if mask else 0
        if mask and self.window < 1:
            raise ValueError(f"a window of {self.window} tokens")
        self.gate, self.layout = p.get("gate", "head"), p.get("rot_layout", "interleaved")
        self.dp, self.rp, self.dvp = pad16(self.d), pad16(self.rot), pad16(self.dv)
        self.qrp, self.kvp, self.gp = pad16(self.q_rank), pad16(self.kv_rank), pad16(self.H)
        self.head = self.dp + self.rp
        self.out_dim = self.H * self.dvp

    def shapes(self):
        H, d, r, dv, w = self.H, self.d, self.rot, self.dv, self.width
        q = ({"dq": (self.q_rank, w), "dq.norm": (self.q_rank,), "uq": (H * (d + r), self.q_rank)} if self.q_rank else {"q": (H * (d + r), w)})
        return {**q, "dkv": (self.kv_rank + r, w), "dkv.norm": (self.kv_rank,), "uk": (H * d, self.kv_rank), "uv": (H * dv, self.kv_rank),
                "g": (H if self.gate == "head" else H * dv, w), "o": (w, H * dv)}

    def _pairs(self, t):
        """Rows of a rotated part [..., rot, n] in the order of interleaved pairs."""
        return t if self.layout == "interleaved" else t[..., torch.arange(self.rot).view(2, -1).t().reshape(-1), :]

    def _q_rows(self, t, cols):
        """Rows of every query head, unrotated and rotated part padded on their own."""
        t = t.view(self.H, self.d + self.rot, -1)
        return torch.cat([_pad_to(t[:, : self.d], self.H, self.dp, cols), _pad_to(self._pairs(t[:, self.d:]), self.H, self.rp, cols)],
                         1).reshape(self.H * self.head, cols)

    def in_parts(self, get):
        dkv, W = get("dkv"), self.W
        dkv = torch.cat([_pad_to(dkv[: self.kv_rank], self.kvp, W), _pad_to(self._pairs(dkv[self.kv_rank:]), self.rp, W)])
        g = _pad_to(get("g"), self.gp, W) if self.gate == "head" else pad_heads_rows(get("g"), self.H, self.dv, W)
        q = ("dq", _pad_to(get("dq"), self.qrp, W)) if self.q_rank else ("q", self._q_rows(get("q"), W))
        return [q, ("dkv", dkv), ("g", g)]

    def out_part(self, get):
        return pad_heads_cols(get("o"), self.H, self.dv, self.W)

    def load(self, get, fin, vec, model):
        H, d, dv = self.H, self.d, self.dv
        if self.q_rank:
            self.uq, self.dq_norm = fin(self._q_rows(get("uq"), self.qrp)), vec(_pad_to(get("dq.norm"), self.qrp))
        self.uk_t = fin(_pad_to(get("uk").view(H, d, self.kv_rank).transpose(1, 2), H, self.kvp, self.dp))     # [H, kv_rank, dim]
        self.uv = fin(_pad_to(get("uv").view(H, dv, self.kv_rank), H, self.dvp, self.kvp))                     # [H, vdim, kv_rank]
        # the expansion of prompts: every head's key rows, then its value rows
        self.ukv = fin(torch.cat([_pad_to(get("uk").view(H, d, self.kv_rank), H, self.dp, self.kvp),
                                  _pad_to(get("uv").view(H, dv, self.kv_rank), H, self.dvp, self.kvp)], 1)
                       .reshape(H * (self.dp + self.dvp), self.kvp))
        self.dkv_norm = vec(_pad_to(get("dkv.norm"), self.kvp))
        self.cos_sin = model.rope_table(self.rot, float(self.rot_spec["base"]), self.rot_spec.get("scaling"))

    def cache_shape(self, model):
        return {"paged": self.kvp + self.rp}

    def run(self, model, h, proj, y, inp, cache):
        ops = model.ops
        prep = lambda dq, norm, **q: ops.latent_prep(dq, proj["dkv"], norm, self.dkv_norm, self.q_rank, self.kv_rank, self.rot, model.eps, self.cos_sin,
                                                     inp.positions, inp.slots, cache, **q)
        if self.q_rank:
            q = ops.gemm(prep(proj["dq"], self.dq_norm), self.uq)
            ops.rope_pairs(q, inp.positions, self.cos_sin, self.H, self.head, self.dp, self.rot)
        else:
            q = proj["q"]
            prep(None, None, q=q, heads=self.H, head=self.head, off=self.dp)
        gate, wide = proj["g"], self.gate == "element"
        if inp.is_prefill and ops.latent_prefill(q, cache, self.ukv, gate, y, self.H, self.dp, self.rp, self.dvp, self.scale, inp, inp.n_decode,
                                                 window=self.window, wide_gate=wide):
            if inp.n_decode == 0:
                return
            inp = inp.decode_rows()                          # the decode rows of a mixed step are left
            n = inp.input_ids.shape[0]
            q, gate, y = q[:n], gate[:n], y[:n]
        q_lat = torch.empty(q.shape[0], self.H * self.kvp, dtype=q.dtype, device=q.device)
        ops.gemm_heads(q, self.uk_t, q_lat, self.head)
        o_lat = ops.latent_attn(q_lat, q, cache, self.H, self.kvp, self.head, self.dp, self.rp, self.scale, inp, window=self.window)
        ops.gemm_heads(o_lat, self.uv, y, self.kvp, gate=gate, wide_gate=wide)


class AttentionMixer(Mixer):
    """Grouped-query attention over paged keys and values.  What a design or layer has of the following is a parameter:

      mask.size   token i sees the last `size` tokens including itself (no mask: all before it)
      qk_norm     queries and keys divided by their root mean square per head (weights shared by the heads)
      bias        biases of the projections
      conv        short causal convolution of this many taps on every channel of q, k and v, in front of the rotation
      rot         rotation of the first `dims` dimensions of q and k, interleaved pairs, `base`, optionally `scaling` of the frequencies
      rot_values  values rotated by their position over all `vdim` dimensions (`base`, no scaling), the result back by the query's
      softcap     scores s become softcap * tanh(s / softcap)
      sink        "learned": a score per head that only the denominator contains; "unit": the denominator plus one
      gate        the heads times sigmoid of a projection of the same input
      out_scale   factor of the output
      kv_from     the layer whose keys and values it uses in place of its own"""

    HEAD_SIZES = (64, 128, 256)                              # of the attention kernels; a head is padded to the next one
    MAX_TAPS = 9                                             # of the convolution kernel

    def __init__(self, params: dict, width: int):
        super().__init__(params, width)
        self.H, self.G, self.d, self.dv = (int(params[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
        if self.H % self.G:
            raise ValueError(f"{self.H} query heads over {self.G} key/value heads")
        mask, self.rot, self.sink = params.get("mask"), params.get("rot"), params.get("sink")
        self.scale, self.window = float(params["scale"]), int(mask["size"]) if mask else 0
        if mask and self.window < 1:
            raise ValueError(f"a window of {self.window} tokens")
        self.sign, self.scale = (-1.0 if self.scale < 0 else 1.0), abs(self.scale)      # (the kernels take scores that grow with the products)
        self.softcap, self.out_scale = float(params.get("softcap") or 0.0), float(params.get("out_scale", 1.0))
        self.qk_norm, self.bias, self.gate, self.rot_values = (bool(params.get(n)) for n in ("qk_norm", "bias", "gate", "rot_values"))
        self.taps, self.kv_from = int(params.get("conv") or 0), params.get("kv_from")
        self.rot_dims = int(self.rot["dims"]) if self.rot else 0
        if self.rot_dims % 2 or self.rot_dims > self.d:
            raise ValueError(f"rotation of {self.rot_dims} of {self.d} dimensions")
        if self.taps > self.MAX_TAPS:
            raise NotImplementedError(f"convolutions of {self.taps} taps (up to {self.MAX_TAPS})")
        if self.qk_norm and (self.taps or self.kv_from is not None):
            raise NotImplementedError("normed queries and keys with a convolution or another layer's keys")
        if self.rot_values and not self.qk_norm:
            raise NotImplementedError("rotated values without normed queries and keys")
        if self.rot_values and self.dv % 2:
            raise ValueError(f"rotation of {self.dv} dimensions")
        if self.kv_from is not None and self.taps:
            raise NotImplementedError("another layer's keys with a convolution")
        self.recurrent = self.taps > 1
        self.dp, self.dvp = self._padded(self.d), self._padded(self.dv)
        self.out_dim = self.H * self.dvp
        # projections: name, heads, width of a head, padded width
        own = [("k", self.G, self.d, self.dp), ("v", self.G, self.dv, self.dvp)] if self.kv_from is None else []
        self.projections = [("q", self.H, self.d, self.dp)] + own

    def _padded(self, n: int) -> int:
        for size in self.HEAD_SIZES:
            if n <= size:
                return size
        raise NotImplementedError(f"attention heads of {n} (up to {self.HEAD_SIZES[-1]})")

    def shapes(self):
        w, out = self.width, {}
        for n, heads, d, _ in self.projections:
            out[n] = (heads * d, w)
            if self.bias:
                out[n + ".b"] = (heads * d,)
            if self.taps:
                out[n + ".conv"] = (heads * d, self.taps)
        if self.qk_norm:
            out.update({"q.norm": (self.d,), "k.norm": (self.d,)})
        if self.sink == "learned":
            out["sink"] = (self.H,)
        if self.gate:
            out["g"] = (self.H * self.dv, w)
        out["o"] = (w, self.H * self.dv)
        return out

    def _q_sign(self, name):
        return self.sign if name == "q" else 1.0

    def _rows(self, t, heads, d, dp, cols):
        return _pad_to(t.view(heads, d, -1), heads, dp, cols).reshape(heads * dp, cols)

    def in_parts(self, get):
        out = [("qkv", torch.cat([self._q_sign(n) * self._rows(get(n), heads, d, dp, self.W) for n, heads, d, dp in self.projections]))]
        return out + ([("g", self._rows(get("g"), self.H, self.dv, self.dvp, self.W))] if self.gate else [])

    def in_bias(self, get):
        if not self.bias:
            return {}
        return {"qkv": torch.cat([self._q_sign(n) * self._rows(get(n + ".b"), heads, d, dp, 1)[:, 0] for n, heads, d, dp in self.projections])}

    def out_part(self, get):
        o = get("o")
        return _pad_to(o.view(o.shape[0], self.H, self.dv), self.W, self.H, self.dvp).reshape(self.W, self.out_dim)

    def load(self, get, fin, vec, model):
        if self.qk_norm:
            self.q_norm, self.k_norm = (vec(_pad_to(get(n), self.dp)) for n in ("q.norm", "k.norm"))      # (the norm keeps the sign of q)
        self.sinks = vec(get("sink")) if self.sink == "learned" else vec(torch.zeros(self.H)) if self.sink == "unit" else None
        self.conv_w = None
        if self.taps:                                        # [taps, channels]
            self.conv_w = vec(torch.cat([self._rows(get(n + ".conv"), heads, d, dp, self.taps) for n, heads, d, dp in self.projections]).t())
        self.cos_sin = model.rope_table(self.rot_dims, float(self.rot["base"]), self.rot.get("scaling")) if self.rot_dims else None
        self.v_cos_sin = model.rope_table(self.dv, float(self.rot["base"])) if self.rot_values else None
        if self.kv_from is not None:
            self._check_source(model)

    def _check_source(self, model):
        """The layers in front of this one are there already."""
        src = model.layers[self.kv_from].mixer if 0 <= self.kv_from < len(model.layers) else None
        src = getattr(src, "kv_mixer", src)
        if not isinstance(src, AttentionMixer) or src.kv_from is not None:
            raise ValueError(f"layer {self.kv_from} has no keys and values of its own in front of the layer that uses them")
        if (src.G, src.d, src.dv) != (self.G, self.d, self.dv):
            raise ValueError(f"layer {self.kv_from} has other key/value heads than the layer that uses them")

    def cache_shape(self, model):
        if self.kv_from is not None:
            return {"share_layer": self.kv_from}
        out = {"kv": (self.G, self.dp, self.dvp)}
        if self.recurrent:
            out["state"] = {"conv": ((self.taps - 1, self.conv_w.shape[1]), model.dtype)}
        return out

    def run(self, model, h, proj, y, inp, cache):
        qkv, ops, conv = proj["qkv"], model.ops, None
        while isinstance(cache, dict):                       # pages beside a state, or those of a mixer within a layer
            conv, cache = cache.get("conv"), cache["kv"] if "kv" in cache else cache["left"]
        if self.qk_norm:
            q = qkv
            ops.qk_norm_kvwrite(qkv, self.H, self.G, self.dp, self.dvp, self.d, self.q_norm, self.k_norm, model.eps, cache, inp.slots,
                                positions=inp.positions, cos_sin=self.cos_sin, v_cos_sin=self.v_cos_sin)
        else:
            own = self.G if self.kv_from is None else 0
            q = ops.conv_rope_kvwrite(qkv, self.H, own, self.dp, self.dvp, self.cos_sin, self.rot_dims, inp.positions, cache, inp, self.conv_w, conv)
        ops.gqa_attn(q, cache, self.H, self.G, self.dp, self.dvp, self.scale, self.window, inp, y, softcap=self.softcap, sink=self.sinks,
                     gate=proj.get("g"), out_scale=self.out_scale, turn_back=self.v_cos_sin)


class Mamba2Mixer(Mixer):
    """Selective state space recurrence: x, B and C through a short causal convolution and silu, a decay and a step size per token and
    head, the state [state, vdim] of a head, then the gate and an RMS norm of `norm_groups` equal parts."""

    recurrent = True
    MAX_STATE = 256                                          # of the recurrence kernels

    def __init__(self, params: dict, width: int):
        super().__init__(params, width)
        self.H, self.dv, self.n, self.G = (int(params[k]) for k in ("heads", "vdim", "state", "groups"))
        self.taps, self.parts, self.out_scale = int(params["conv"]), int(params["norm_groups"]), float(params.get("out_scale", 1.0))
        self.inner = self.H * self.dv
        if self.H % self.G or self.inner % self.parts:
            raise ValueError(f"{self.H} heads of {self.dv} in {self.G} groups, normed in {self.parts} parts")
        if not 1 <= self.taps <= AttentionMixer.MAX_TAPS or self.n > self.MAX_STATE:
            raise NotImplementedError(f"a state of {self.n} (up to {self.MAX_STATE}) behind {self.taps} taps (1 to {AttentionMixer.MAX_TAPS})")
        self.np, self.dvp = pad16(self.n), pad16(self.dv)
        self.out_dim = pad16(self.inner)
        self.channels = self.H * self.dvp + 2 * self.G * self.np
        self.parallelism = self.H * ((self.dvp + 63) // 64)

    def shapes(self):
        c = self.inner + 2 * self.G * self.n
        return {"in": (self.inner + c + self.H, self.width), "conv": (c, self.taps), "conv.b": (c,), "dt_bias": (self.H,), "A_log": (self.H,),
                "D": (self.H,), "norm": (self.inner,), "o": (self.width, self.inner)}

    def _channels(self, t, cols):
        """Rows [x | B | C], every head and group padded on its own."""
        x, b, c = torch.split(t.reshape(t.shape[0], -1), [self.inner, self.G * self.n, self.G * self.n])
        pad = lambda u, heads, d: _pad_to(u.reshape(heads, d, -1), heads, pad16(d), cols).reshape(heads * pad16(d), cols)
        return torch.cat([pad(x, self.H, self.dv), pad(b, self.G, self.n), pad(c, self.G, self.n)])

    def in_parts(self, get):
        z, xbc, dt = torch.split(get("in"), [self.inner, self.inner + 2 * self.G * self.n, self.H])
        return [("z", pad_heads_rows(z, self.H, self.dv, self.W)), ("xbc", self._channels(xbc, self.W)), ("dt", _pad_to(dt, pad16(self.H), self.W))]

    def out_part(self, get):
        return _pad_to(get("o"), self.W, self.out_dim)

    def load(self, get, fin, vec, model):
        self.conv_w = vec(self._channels(get("conv"), self.taps).t())              # [taps, channels]
        self.conv_b = vec(self._channels(get("conv.b"), 1)[:, 0])
        self.dt_bias, self.D = vec(get("dt_bias")), vec(get("D"))
        self.A = vec(-torch.exp(get("A_log")))
        self.norm = vec(get("norm") * self.out_scale)

    def cache_shape(self, model):
        return {"state": {"S": ((self.H, self.np, self.dvp), torch.float32), "conv": ((self.taps - 1, self.channels), model.dtype)}}

    def run(self, model, h, proj, y, inp, cache):
        ops = model.ops
        xbc = ops.causal_conv(proj["xbc"], self.conv_w, self.conv_b, "silu", cache["conv"], inp)
        o = ops.ssd(xbc, proj["dt"], self.H, self.G, self.np, self.dvp, self.dt_bias, self.A, self.D, cache["S"], inp)
        ops.gate_norm(o, proj["z"], self.H, self.dv, self.parts, self.norm, model.eps, y)


class ParallelMixer(Mixer):
    """left_scale * left(h) + right_scale * right(h).  Both write side by side into one buffer, already scaled, and their output
    projections are one product whose K runs over both."""

    SIDES = ("left", "right")

    def __init__(self, params: dict, width: int):
        super().__init__(params, width)
        sub = lambda side: dict({k: v for k, v in params[side].items() if k != "type"}, out_scale=float(params.get(side + "_scale", 1.0)))
        self.sides = {s: _mixer_class(params[s]["type"])(sub(s), width) for s in self.SIDES}
        for m in self.sides.values():
            if not hasattr(m, "out_scale"):
                raise NotImplementedError(f"{type(m).__name__} beside another mixer")
        self.recurrent = any(m.recurrent for m in self.sides.values())
        self.parallelism = min(m.parallelism for m in self.sides.values())
        self.out_dim = sum(m.out_dim for m in self.sides.values())
        self.kv_mixer = self.sides["left"]

    def _each(self, get):
        return ((s, m, lambda name, s=s: get(f"{s}.{name}")) for s, m in self.sides.items())

    def shapes(self):
        return {f"{s}.{n}": shape for s, m in self.sides.items() for n, shape in m.shapes().items()}

    def in_parts(self, get):
        return [(f"{s}.{n}", t) for s, m, sub in self._each(get) for n, t in m.in_parts(sub)]

    def in_bias(self, get):
        return {f"{s}.{n}": t for s, m, sub in self._each(get) for n, t in m.in_bias(sub).items()}

    def out_part(self, get):
        return torch.cat([m.out_part(sub) for _, m, sub in self._each(get)], 1)

    def load(self, get, fin, vec, model):
        for _, m, sub in self._each(get):
            m.load(sub, fin, vec, model)

    def cache_shape(self, model):
        return {"parts": {s: m.cache_shape(model) for s, m in self.sides.items()}}

    def run(self, model, h, proj, y, inp, cache):
        at = 0
        for s, m in self.sides.items():
            m.run(model, h, {n[len(s) + 1:]: v for n, v in proj.items() if n.startswith(s + ".")}, y[:, at: at + m.out_dim], inp, cache[s])
            at += m.out_dim


MIXERS = {"lightning": LightningMixer, "wkv": WkvMixer, "latent_attention": LatentAttentionMixer, "attention": AttentionMixer,
          "mamba2": Mamba2Mixer, "parallel": ParallelMixer}


def _mixer_class(name: str):
    if name not in MIXERS:
        raise NotImplementedError(f"no mixer {name!r}; known: {sorted(MIXERS)}")
    return MIXERS[name]


def make_mixer(spec, width: int) -> Mixer:
    return _mixer_class(spec.mixer)(spec.params, width)


@dataclass
class MixerLayer:
    """One layer: its norm, its mixer and the two fused projections."""
    mixer: Mixer
    ff: int                                                  # padded width of the feed-forward (0: none)
    norm: Optional[torch.Tensor] = None                      # fp32 [W], stored around zero
    in_w: Optional[torch.Tensor] = None                      # [rows, W]: the mixer's input projections, then gate and up
    out_w: Optional[torch.Tensor] = None                     # [W, mixer out_dim + ff]
    parts: Dict[str, Tuple[int, int]] = field(default_factory=dict)

    def forward(self, model, residual, pending, inp, cache):
        """residual (fp32) += pending; returns this layer's contribution, to be added by whoever norms the residual next."""
        ops, m = model.ops, self.mixer
        h = ops.norm_stream(residual, pending, self.norm, model.eps, model.config.norm_weight_offset, model.hidden, model.dtype)
        T = h.shape[0]
        proj = ops.gemm(h, self.in_w) if self.in_w is not None else None
        views = {n: proj[:, a:b] for n, (a, b) in self.parts.items()}
        y = torch.empty(T, m.out_dim + self.ff, dtype=h.dtype, device=h.device)
        m.run(model, h, views, y, inp, cache)
        if self.ff:
            ops.act_mul(views["mlp"], self.ff, model.config.hidden_act, gated=True, out=y[:, m.out_dim:])
        return ops.gemm(y, self.out_w)


class DenseMlp:
    """down(act(up(h))), or gated: down(act(gate(h)) * up(h)).  `act`: an activation of its own in place of the model's, with its limit."""

    def __init__(self, ff: int, width: int, gated: bool, act: str = "", limit: float = 0.0):
        self.ff, self.width, self.W, self.gated = ff, width, pad16(width), gated
        self.fp = pad16(ff)
        self.names = ("gate", "up") if gated else ("up",)
        self.act, self.act_args = act, dict(limit=limit) if act else {}

    def shapes(self):
        return dict({n: (self.ff, self.width) for n in self.names}, down=(self.width, self.ff))

    def load(self, get, fin, vec, model, beside=None):
        """`beside`: (weight [n, W], bias [n]) of a further projection of the same input, which rides in the first product."""
        rows, self.up_b = [_pad_to(get(n), self.fp, self.W) for n in self.names], None
        if beside is not None:
            self.up_b = fin(torch.cat([torch.zeros(len(rows) * self.fp, device=beside[1].device), beside[1]]))
            rows.append(beside[0])
        self.up = fin(torch.cat(rows))
        self.down = fin(_pad_to(get("down"), self.W, self.fp))

    def run(self, model, h):
        """-> (rows, None): one row per token."""
        return self.run_beside(model, h)[:2]

    def run_beside(self, model, h):
        """-> the same and the projection beside (or None)."""
        ops, n = model.ops, len(self.names) * self.fp
        u = ops.gemm(h, self.up, bias=self.up_b)
        a = ops.act_mul(u, self.fp, self.act or model.config.hidden_act, gated=self.gated, **self.act_args)
        return ops.gemm(a, self.down), None, u[:, n:] if self.up_b is not None else None


class MoeMlp:
    """Routed experts down(act(up(h))), or gated: down(silu(gate(h)) * up(h)), with the rows of gate and up taking turns in one matrix, so
    that the product's epilogue has both.  How the experts are chosen and weighted is in the MoeSpec.

    The shared expert is cut into slices of an expert's (padded) width; every token takes each slice with the weight
    sigmoid(sg . h), or one, so the slices ride in the grouped products as further experts, and `sg` is one more row of the router."""

    TILE = 128                                               # features per work item of the grouped products

    def __init__(self, spec, width: int):
        self.spec, self.width, self.W = spec, width, pad16(width)
        self.names = ("gate", "up") if spec.gated else ("up",)
        up = lambda n, tile=self.TILE: (n + tile - 1) // tile * tile
        self.fp, self.Wp = up(spec.ff, self.TILE // len(self.names)), up(self.W)
        self.slices = (spec.shared_ff + self.fp - 1) // self.fp
        if spec.experts > 256 or spec.top > 32 or self.slices > 32:      # tables of the routing kernels
            raise NotImplementedError(f"{spec.experts} experts, {spec.top} per token, a shared expert of {self.slices} expert widths")
        if spec.score == "softmax" and (spec.group_top != 1 and spec.groups):
            raise NotImplementedError("groups of softmax scores by more than their largest")

    def shapes(self):
        s, w = self.spec, self.width
        out = {"router": (s.experts, w)}
        if s.score == "sigmoid":
            out["correction"] = (s.experts,)
        if s.bias:
            out["router.b"] = (s.experts,)
        for e in range(s.experts):
            out.update({f"e{e}.{n}": (s.ff, w) for n in self.names})
            out[f"e{e}.down"] = (w, s.ff)
        if s.shared_ff:
            out.update({f"shared.{n}": (s.shared_ff, w) for n in self.names})
            out["shared.down"] = (w, s.shared_ff)
            if s.shared_gate:
                out["shared.sg"] = (1, w)
        return out

    def load(self, get, fin, vec, model, beside=None):
        s, n, step = self.spec, self.spec.experts + self.slices, len(self.names)
        if s.gated and model.config.hidden_act != "silu":
            raise NotImplementedError(f"gated experts with {model.config.hidden_act}")
        new = lambda *shape: torch.zeros(*shape, dtype=model.dtype, device=model.device)
        self.up, self.down = new(n, step * self.fp, self.W), new(n, self.Wp, self.fp)
        for e in range(s.experts):
            for i, name in enumerate(self.names):
                self.up[e, i: step * s.ff: step, : self.width] = fin(get(f"e{e}.{name}"))
            self.down[e, : self.width, : s.ff] = fin(get(f"e{e}.down"))
        router = [get("router")]
        if s.shared_ff:
            ups, down = [fin(get("shared." + name)) for name in self.names], fin(get("shared.down"))
            for i in range(self.slices):
                a, b = i * self.fp, min((i + 1) * self.fp, s.shared_ff)
                for j, up in enumerate(ups):
                    self.up[s.experts + i, j: step * (b - a): step, : self.width] = up[a:b]
                self.down[s.experts + i, : self.width, : b - a] = down[:, a:b]
            if s.shared_gate:
                router.append(get("shared.sg"))
        self.router = fin(_pad_to(torch.cat(router), (s.experts + 8) // 8 * 8, self.W))      # (whole tiles of the router kernel)
        self.correction = vec(get("correction")) if s.score == "sigmoid" else None
        self.router_b = vec(get("router.b")) if s.bias else None
        self.beside = (fin(beside[0]), fin(beside[1])) if beside is not None else None

    def run(self, model, h):
        """-> (rows of every (token, expert) pair, (row, weight) of each token's pairs)."""
        return self.run_beside(model, h)[:2]

    def run_beside(self, model, h):
        """-> the same and the projection beside (or None)."""
        s, ops = self.spec, model.ops
        r = ops.moe_route(h, self.router, s.top, 0, s.experts, experts=s.experts, score=s.score, correction=self.correction, groups=s.groups,
                          keep=s.keep, scale=s.scale, shared=self.slices, group_top=s.group_top, renorm=s.renorm, bias=self.router_b,
                          shared_gate=s.shared_gate)
        avg = max(1, (h.shape[0] * s.top + s.experts - 1) // s.experts)
        a = ops.moe_grouped_gemm(r.xg, self.up, r.seg, avg, shared=self.slices, tokens=h.shape[0],
                                 act="swiglu" if s.gated else model.config.hidden_act)
        beside = ops.gemm(h, self.beside[0], bias=self.beside[1]) if self.beside is not None else None
        return ops.moe_grouped_gemm(a, self.down, r.seg, avg), (r.pos, r.topk_w), beside


@dataclass
class PreNormLayer:
    """x += mixer(norm1(x)), then x += ff(norm2(x)).  The stream is fp32; what a sublayer adds (`pending`: rows, and with experts the
    (row, weight) pairs of every token) is added by the norm that reads the stream next."""
    mixer: Mixer
    mlp: Optional[object]                                    # DenseMlp, MoeMlp or None
    norm1: torch.Tensor = None                               # fp32 [W]
    norm2: Optional[torch.Tensor] = None
    in_w: Optional[torch.Tensor] = None                      # [rows, W]
    in_b: Optional[torch.Tensor] = None                      # [rows]
    out_w: Optional[torch.Tensor] = None                     # [W, mixer out_dim]
    parts: Dict[str, Tuple[int, int]] = field(default_factory=dict)

    def forward(self, model, residual, pending, inp, cache):
        ops, m, c = model.ops, self.mixer, model.config
        norm = lambda pending, w: ops.norm_stream(residual, pending[0], w, model.eps, c.norm_weight_offset, model.hidden, model.dtype, pairs=pending[1])
        h = norm(pending, self.norm1)
        proj = ops.gemm(h, self.in_w, bias=self.in_b)
        y = torch.empty(h.shape[0], m.out_dim, dtype=h.dtype, device=h.device)
        m.run(model, h, {n: proj[:, a:b] for n, (a, b) in self.parts.items()}, y, inp, cache)
        pending = ops.gemm(y, self.out_w), None
        return pending if self.mlp is None else self.mlp.run(model, norm(pending, self.norm2))


@dataclass
class PostNormLayer:
    """x += mult * norm1(mixer(x)), then x += mult * norm2(ff(x)).  The stream is fp32; `h` is its copy in the model's dtype that the
    products read, written by whoever last added to the stream."""
    mixer: Mixer
    mlp: Optional[object]                                    # DenseMlp, MoeMlp or None
    norm1: Tuple[torch.Tensor, torch.Tensor] = None          # weight, bias: fp32 [W]
    norm2: Optional[Tuple[torch.Tensor, torch.Tensor]] = None
    in_w: Optional[torch.Tensor] = None
    out_w: Optional[torch.Tensor] = None
    parts: Dict[str, Tuple[int, int]] = field(default_factory=dict)

    def forward(self, model, residual, h, inp, cache):
        """Adds both sublayers to `residual`; -> its new copy."""
        ops, m, c = model.ops, self.mixer, model.config
        proj = ops.gemm(h, self.in_w)
        y = torch.empty(h.shape[0], m.out_dim, dtype=h.dtype, device=h.device)
        m.run(model, h, {n: proj[:, a:b] for n, (a, b) in self.parts.items()}, y, inp, cache)
        add = lambda rows, norm, pairs=None: ops.norm_add(residual, rows, norm[0], norm[1], c.residual_multiplier, model.eps, model.hidden,
                                                          model.dtype, layernorm=True, pairs=pairs)
        h = add(ops.gemm(y, self.out_w), self.norm1)
        if self.mlp is not None:
            rows, pairs = self.mlp.run(model, h)
            h = add(rows, self.norm2, pairs)
        return h


@dataclass
class SandwichLayer:
    """x += scale1 * norm1b(mixer(norm1(x)) * gate1), then x += scale2 * norm2b(ff(norm2(x)) * gate2), a gate being the sigmoid of a
    projection (with bias) of what its sublayer reads.  The gates' projections ride in the products that read the same rows.  The stream
    is fp32; `h` is its norm that the next sublayer reads, written by whoever last added to the stream."""
    mixer: Mixer
    mlp: Optional[object]                                    # DenseMlp, MoeMlp or None
    norm1: torch.Tensor = None                               # fp32 [W]
    norm2: Optional[torch.Tensor] = None
    add1: torch.Tensor = None                                # fp32 [W]: weight of the output's norm times the layer scale
    add2: Optional[torch.Tensor] = None
    in_w: Optional[torch.Tensor] = None                      # [rows, W]
    in_b: Optional[torch.Tensor] = None                      # [rows]
    out_w: Optional[torch.Tensor] = None                     # [W, mixer out_dim]
    parts: Dict[str, Tuple[int, int]] = field(default_factory=dict)

    def forward(self, model, residual, h, inp, cache, next_norm, rows=None):
        """Adds both sublayers to `residual`; -> its norm by `next_norm` (of `rows` only when given: the stream's other rows are then
        not needed any more)."""
        ops, m, c = model.ops, self.mixer, model.config
        add = lambda y, w, gate, nxt, rows, pairs=None: ops.norm_add(residual, y, w, None, c.residual_multiplier, model.eps, model.hidden, model.dtype,
                                                                     layernorm=False, pairs=pairs, gate=gate, next_weight=nxt, rows=rows)
        proj = ops.gemm(h, self.in_w, bias=self.in_b)
        views = {n: proj[:, a:b] for n, (a, b) in self.parts.items()}
        y = torch.empty(h.shape[0], m.out_dim, dtype=h.dtype, device=h.device)
        m.run(model, h, views, y, inp, cache)
        y, gate = ops.gemm(y, self.out_w), views.get("residual_gate")
        if self.mlp is None:
            return add(y, self.add1, gate, next_norm, rows)
        h = add(y, self.add1, gate, self.norm2, None)
        y, pairs, gate = self.mlp.run_beside(model, h)
        return add(y, self.add2, gate, next_norm, rows, pairs)


LAYER_KINDS = {"pre": PreNormLayer, "post": PostNormLayer, "sandwich": SandwichLayer}


def make_mlp(spec, width: int):
    if spec.moe is not None:
        return MoeMlp(spec.moe, width)
    return DenseMlp(spec.ff, width, spec.gated, spec.act, spec.limit) if spec.ff else None


def _parts(layer, rows):
    """Row ranges of the fused input projection -> layer.parts."""
    o = 0
    for name, t in rows:
        layer.parts[name] = (o, o + t.shape[0])
        o += t.shape[0]


def load_mixer_layers(m, w):
    """Tensors of a layer-by-layer checkpoint -> `m` (a DecoderModel): `embed`, `pos`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`,
    `l<i>.mlp.*`, `final.norm`, `head`; a layer norm's bias is called like its weight with `.b` added.  Also, where the design has them:
    `bigram`; `l<i>.norm1b`, `l<i>.norm2b` (norms of the sublayers' outputs), `l<i>.ls1`, `l<i>.ls2` (their scale) and `l<i>.rg1`, `l<i>.rg2`
    with `.b` (their gate)."""
    c, dt, dev = m.config, m.dtype, m.device
    if m.tp.world_size > 1:
        raise ValueError(f"{c.model_type} is served on one shard")
    W = pad16(c.hidden_size)

    def get(name):
        return w.get_tensor(name).float()

    def fin(t):
        return t.to(dt).to(dev).contiguous()

    def vec(t):
        return t.to(torch.float32).to(dev).contiguous()

    m.embed = fin(_pad_to(get("embed"), c.vocab_size, W))
    m.lm_head = fin(_pad_to(get("head"), pad16(c.vocab_size), W))
    stream_vec = lambda t: vec(_pad_to(t.expand(c.hidden_size), W))          # (a single number counts for every column)
    m.final_norm = stream_vec(get("final.norm"))
    if c.bigram:
        m.bigram_embed = fin(_pad_to(get("bigram"), c.bigram[0] + 1, W))
    if c.learned_positions:
        m.pos_embed = fin(_pad_to(get("pos"), c.max_position_embeddings, W))
    if c.norm_type == "layernorm":
        m.final_norm_b = vec(_pad_to(get("final.norm.b"), W))
    m.layers = []
    if c.layer_style in LAYER_KINDS:
        norm = lambda name: stream_vec(get(name))
        if c.layer_style == "post":
            norm = lambda name: (vec(_pad_to(get(name), W)), vec(_pad_to(get(name + ".b"), W)))
        for i, spec in enumerate(c.layer_specs):
            if spec.weights_of is not None:
                m.layers.append(None)
                continue
            layer = LAYER_KINDS[c.layer_style](make_mixer(spec, c.hidden_size), make_mlp(spec, c.hidden_size), norm(f"l{i}.norm1"))
            sub = lambda name, i=i: get(f"l{i}.mix.{name}")
            rows, bias = layer.mixer.in_parts(sub), layer.mixer.in_bias(sub)
            beside = None
            if c.layer_style == "sandwich":
                out_norm = lambda n, i=i: stream_vec(get(f"l{i}.norm{n}b") * (get(f"l{i}.ls{n}") if c.layer_scale else 1.0))
                layer.add1 = out_norm(1)
                if c.residual_gate:
                    gate = lambda n, i=i: (_pad_to(get(f"l{i}.rg{n}"), W, W), _pad_to(get(f"l{i}.rg{n}.b"), W))
                    w_gate, bias["residual_gate"] = gate(1)
                    rows.append(("residual_gate", w_gate))
                if layer.mlp is not None:
                    layer.add2, beside = out_norm(2), gate(2) if c.residual_gate else None
            _parts(layer, rows)
            layer.in_w, layer.out_w = fin(torch.cat([t for _, t in rows])), fin(layer.mixer.out_part(sub))
            if bias:
                layer.in_b = fin(torch.cat([bias[n] if n in bias else torch.zeros_like(t[:, 0]) for n, t in rows]))
            layer.mixer.load(sub, fin, vec, m)
            if layer.mlp is not None:
                layer.norm2 = norm(f"l{i}.norm2")
                layer.mlp.load(lambda name, i=i: get(f"l{i}.mlp.{name}"), fin, vec, m, **(dict(beside=beside) if beside is not None else {}))
            m.layers.append(layer)
        for i, spec in enumerate(c.layer_specs):
            if spec.weights_of is not None:
                m.layers[i] = m.layers[spec.weights_of]
        return
    for i, spec in enumerate(c.layer_specs):
        mx = make_mixer(spec, c.hidden_size)
        ff = pad16(spec.ff) if spec.ff else 0
        layer = MixerLayer(mx, ff, norm=vec(_pad_to(get(f"l{i}.norm1"), W)))
        sub = lambda name, i=i: get(f"l{i}.mix.{name}")
        rows = mx.in_parts(sub)
        out = [mx.out_part(sub)]
        if ff:
            rows.append(("mlp", torch.cat([_pad_to(get(f"l{i}.mlp.{n}"), ff, W) for n in ("gate", "up")])))
            out.append(_pad_to(get(f"l{i}.mlp.down"), W, ff))
        _parts(layer, rows)
        layer.in_w = fin(torch.cat([t for _, t in rows])) if rows else None
        layer.out_w = fin(torch.cat(out, 1))
        mx.load(sub, fin, vec, m)
        m.layers.append(layer)


def tensor_shapes(c) -> Dict[str, Tuple[int, ...]]:
    """Name -> shape of every tensor of a layer-by-layer checkpoint of this configuration."""
    w = c.hidden_size
    stream = () if c.norm_scalar else (w,)
    out = {"embed": (c.vocab_size, w), "head": (c.vocab_size, w), "final.norm": stream}
    if c.bigram:
        out["bigram"] = (c.bigram[0] + 1, w)
    if c.layer_style in LAYER_KINDS:
        if c.learned_positions:
            out["pos"] = (c.max_position_embeddings, w)
        if c.norm_type == "layernorm":
            out["final.norm.b"] = (w,)
        for i, spec in enumerate(c.layer_specs):
            if spec.weights_of is not None:
                continue
            mlp = make_mlp(spec, w)
            for n in (1, 2) if mlp is not None else (1,):
                out[f"l{i}.norm{n}"] = stream
                if c.norm_type == "layernorm":
                    out[f"l{i}.norm{n}.b"] = (w,)
                if c.layer_style == "sandwich":
                    out[f"l{i}.norm{n}b"] = stream
                    out.update({f"l{i}.ls{n}": (w,)} if c.layer_scale else {})
                    out.update({f"l{i}.rg{n}": (w, w), f"l{i}.rg{n}.b": (w,)} if c.residual_gate else {})
            out.update({f"l{i}.mix.{n}": s for n, s in make_mixer(spec, w).shapes().items()})
            out.update({f"l{i}.mlp.{n}": s for n, s in (mlp.shapes() if mlp is not None else {}).items()})
        return out
    for i, spec in enumerate(c.layer_specs):
        out[f"l{i}.norm1"] = (w,)
        out.update({f"l{i}.mix.{n}": s for n, s in make_mixer(spec, w).shapes().items()})
        if spec.ff:
            out.update({f"l{i}.mlp.gate": (spec.ff, w), f"l{i}.mlp.up": (spec.ff, w), f"l{i}.mlp.down": (w, spec.ff)})
    return out


class RandomWeights:
    """Random tensors of `tensor_shapes`, drawn one at a time on `device` when the loader asks for them (benchmarks, tests)."""
    quant = None

    def __init__(self, c, device="cpu", seed: int = 0):
        self.shapes, self.device, self.seed = tensor_shapes(c), device, seed
        self.order = {n: i for i, n in enumerate(self.shapes)}
        self.plain_norm = 1.0 - c.norm_weight_offset         # a norm weight that scales by one

    def has_tensor(self, name):
        return name in self.shapes

    def get_tensor(self, name):
        shape = self.shapes[name]
        g = torch.Generator(device=self.device).manual_seed(self.seed * 100003 + self.order[name])
        t = torch.randn(shape, generator=g, device=self.device, dtype=torch.float32)
        leaf = name.rsplit(".", 1)[-1]
        if ".mu." in name:
            return torch.sigmoid(t)
        if name.endswith(("dq.norm", "dkv.norm", "mix.norm")):
            return 1.0 + 0.1 * t
        if leaf == "w0":
            return -2.0 + 1.5 * t
        if leaf in ("norm1", "norm2", "norm", "norm1b", "norm2b", "ls1", "ls2"):
            return self.plain_norm + 0.1 * t
        if leaf == "b":
            return 0.1 * t
        if leaf == "correction":
            return 0.2 * t
        if leaf in ("u", "A_log"):
            return 0.5 * t
        if leaf == "D":
            return 1.0 + 0.1 * t
        if leaf == "dt_bias":
            return -1.5 + t
        if leaf == "sink":
            return t
        return t if name in ("embed", "pos", "bigram") else t * shape[-1] ** -0.5
