"""Prefill and decode throughput of a layer-by-layer design (random weights, layers of a real model's size) beside the closest
uniform decoder of this framework at equal size, and the device time of every kernel of both with its share of the roofline.

    python bench.py --design vabunex|sapudra|saredra|fegolorn [--design-size small,base] [--steps K] [--warmup W]

"Equal size": for Vabunex a llama-style decoder with the same width, feed-forward width, number of layer runs and attention heads of
128; for Sapudra a Mixtral-style decoder with the same width, heads, window, layers and experts, whose gated experts (three matrices)
have two thirds of the width, and which takes one expert more per token in place of the shared one; where the size has no experts, a
Mistral-style decoder likewise; for Saredra two designs whose kernels are its kernels' closest relatives: Sapudra with the same width,
heads, window, layers and experts (not gated, of 3/2 the width: the same bytes), and Vabunex with as many layers of linear attention
whose state has the size of the state space mixer's; for Fegolorn likewise Sapudra with the same width, heads (no window), layers and
experts, and Vabunex with as many layers of latent attention (no window, a low-rank query) and its dense feed-forward.
Throughput: prefill is one eager forward pass over ragged prompts, decode one CUDA-graph replay per token, both through
`ModelRunner`, timed with CUDA events.  Kernel times: CUDA events around every operator of an eager pass, L2 flushed in front of it,
median of the passes.  Rooflines: the measured copy bandwidth and bf16 rate of MEASURED_PEAKS.json, whichever bounds the operator.
"""

from __future__ import annotations

import json
import os
import statistics
import time

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

VABUNEX_SIZES = {
    # width, ff, recurrent heads x dim, wkv heads x dim, latent heads, q rank, kv rank, rot
    "small": dict(width=2048, ff=8192, lin=(16, 128), wkv=(32, 64), heads=16, q_rank=1024, kv_rank=512, rot=64),
    "base": dict(width=4096, ff=14336, lin=(32, 128), wkv=(64, 64), heads=32, q_rank=1536, kv_rank=512, rot=64),
}
SAPUDRA_SIZES = {
    # width, layers, heads and key/value heads of 128, window; experts, per token, groups and groups kept, width of an expert (or of the
    # dense feed-forward)
    "small": dict(width=2048, layers=4, heads=16, kv=4, window=1024, experts=64, top=6, groups=(8, 4), ff=1536),
    "base": dict(width=4096, layers=4, heads=32, kv=8, window=1024, experts=32, top=4, groups=(4, 2), ff=6144),
    "dense": dict(width=4096, layers=4, heads=32, kv=8, window=1024, experts=0, ff=21504),
}
SAREDRA_SIZES = {
    # width, layer triples (parallel, attention, attention over the keys of the one before), heads and key/value heads of 128, window;
    # state space heads of 64, their groups and parts of the norm, state; experts, per token, groups and groups kept, width of an expert
    # (or of the dense feed-forward)
    "small": dict(width=2048, triples=2, heads=16, kv=4, window=1024, ssm=64, ssm_groups=1, parts=1, state=128, experts=64, top=6, groups=(8, 4), ff=1024),
    "base": dict(width=4096, triples=1, heads=32, kv=8, window=1024, ssm=128, ssm_groups=8, parts=8, state=128, experts=32, top=4, groups=(4, 2), ff=4096),
    "dense": dict(width=4096, triples=1, heads=32, kv=8, window=1024, ssm=128, ssm_groups=8, parts=8, state=128, experts=0, ff=14336),
}
FEGOLORN_SIZES = {
    # width, layer pairs (latent attention with a dense feed-forward, attention with experts); heads of 128, key/value heads; rank of the
    # latent, rotated part, window of the latent layers; width of the dense feed-forward; experts, per token, width of an expert and of the
    # shared one (0 experts: dense in every layer)
    "small": dict(width=2048, pairs=2, heads=16, kv=4, rank=512, rot=64, latent_window=1024, dense=8192, experts=64, top=6, ff=1024),
    "base": dict(width=4096, pairs=2, heads=32, kv=8, rank=512, rot=64, latent_window=1024, dense=14336, experts=32, top=4, ff=4096),
    "dense": dict(width=4096, pairs=2, heads=32, kv=8, rank=512, rot=64, latent_window=1024, dense=14336, experts=0, ff=14336),
}
PREFILL = [(1, 4096), (4, 2048), (1, 16384)]           # (prompts, tokens each)
DECODE = [(16, 2048), (64, 2048), (256, 2048)]         # (rows, tokens of context)


def vabunex_config(s, vocab=32000):
    H, d = s["lin"]
    wh, wd = s["wkv"]
    decay = [1.0 - 2.0 ** (-3 - 7 * h / max(H - 1, 1)) for h in range(H)]
    lin = dict(type="lightning", mixer=dict(heads=H, dim=d, vdim=d, decay=decay), mlp=dict(kind="dense", ff=s["ff"]))
    wkv = dict(type="wkv", mixer=dict(heads=wh, dim=wd), mlp=dict(kind="dense", ff=s["ff"]))
    lat = dict(type="latent_attention", mlp=dict(kind="dense", ff=s["ff"]),
               mixer=dict(heads=s["heads"], dim=128, rot_dim=s["rot"], vdim=128, q_rank=s["q_rank"], kv_rank=s["kv_rank"],
                          scale=(128 + s["rot"]) ** -0.5, rot=dict(base=10000.0, dims=s["rot"])))
    return dict(architecture="Vabunex", vocab=vocab, width=s["width"], norm=dict(eps=1e-5), embedding=dict(scale=1.0),
                layers=[lin, wkv, lat, wkv], loop=dict(start=1, stop=3, times=2))


def llama_like(s, runs, vocab=32000):
    from lorax_b200.config import ModelConfig
    heads = s["width"] // 128
    return ModelConfig(model_type="llama", vocab_size=vocab, hidden_size=s["width"], intermediate_size=s["ff"], num_hidden_layers=runs,
                       num_attention_heads=heads, num_key_value_heads=max(heads // 4, 1), head_dim=128, max_position_embeddings=32768)


def sapudra_config(s, vocab=32000):
    if s["experts"]:
        mlp = dict(kind="moe", expert=dict(ff=s["ff"]), shared=dict(ff=s["ff"]),
                   router=dict(experts=s["experts"], top=s["top"], scale=2.5, groups=dict(count=s["groups"][0], keep=s["groups"][1])))
    else:
        mlp = dict(kind="dense", ff=s["ff"])
    layer = dict(type="attention", mlp=mlp, mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5))
    if s.get("window"):
        layer["mixer"]["mask"] = dict(size=s["window"])
    return dict(architecture="Sapudra", vocab=vocab, width=s["width"], norm=dict(eps=1e-5), residual_mult=0.3, logit_softcap=30.0,
                max_positions=20000, layers=[layer] * s["layers"])


def mixtral_like(s, runs, vocab=32000):
    from lorax_b200.config import ModelConfig
    moe = dict(num_local_experts=s["experts"], num_experts_per_tok=s["top"] + 1) if s["experts"] else {}
    return ModelConfig(model_type="mixtral" if moe else "mistral", vocab_size=vocab, hidden_size=s["width"], intermediate_size=s["ff"] * 2 // 3,
                       num_hidden_layers=runs, num_attention_heads=s["heads"], num_key_value_heads=s["kv"], head_dim=128,
                       max_position_embeddings=32768, sliding_window=s["window"], **moe)


def saredra_config(s, vocab=32000):
    if s["experts"]:
        mlp = dict(kind="moe", expert=dict(ff=s["ff"]),
                   router=dict(experts=s["experts"], top=s["top"], groups=dict(count=s["groups"][0], keep=s["groups"][1])))
    else:
        mlp = dict(kind="dense", ff=s["ff"])
    heads = lambda **rot: dict(heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5, softcap=50.0, mask=dict(size=s["window"]),
                               rot=dict(base=500000.0, dims=64, **rot))
    yarn = dict(factor=4.0, original=8192, fast=32.0, slow=1.0)
    right = dict(heads=s["ssm"], vdim=64, state=s["state"], groups=s["ssm_groups"], norm_groups=s["parts"], conv=4)
    layers = []
    for i in range(s["triples"]):
        layers.append(dict(type="parallel", mlp=mlp, mixer=dict(left=dict(heads(scaling=yarn), conv=4), right=right, left_scale=0.7, right_scale=0.7)))
        layers.append(dict(type="attention", mlp=mlp, mixer=heads()))
        layers.append(dict(type="attention", mlp=mlp, mixer=dict(heads(), kv_from=3 * i + 1)))
    return dict(architecture="Saredra", vocab=vocab, width=s["width"], norm=dict(eps=1e-5), layers=layers)


def sapudra_of_that_size(s, runs, vocab=32000):
    from lorax_b200.config import ModelConfig
    d = sapudra_config(dict(s, layers=runs, ff=s["ff"] * 3 // 2), vocab)
    for layer in d["layers"]:
        layer["mlp"].pop("shared", None)
    return ModelConfig.from_dict(d)


def linear_attention_of_that_size(s, runs, vocab=32000):
    from lorax_b200.config import ModelConfig
    H, d = s["ssm"], s["state"]
    lin = dict(type="lightning", mixer=dict(heads=H, dim=d, vdim=64, decay=[1.0 - 2.0 ** (-3 - 7 * h / max(H - 1, 1)) for h in range(H)]),
               mlp=dict(kind="dense", ff=2 * s["width"]))
    return ModelConfig.from_dict(dict(architecture="Vabunex", vocab=vocab, width=s["width"], norm=dict(eps=1e-5), embedding=dict(scale=1.0),
                                      layers=[lin] * runs))


def fegolorn_config(s, vocab=32000):
    dense = dict(kind="dense", ff=s["dense"], limit=7.0)
    mlp = dict(kind="moe", expert=dict(ff=s["ff"]), shared=dict(ff=s["ff"]), router=dict(experts=s["experts"], top=s["top"])) if s["experts"] else dense
    bands = dict(factor=8.0, low=1.0, high=4.0, original=8192)
    lat = dict(type="latent_attention", mlp=dense, mixer=dict(heads=s["heads"], dim=128, rot_dim=s["rot"], vdim=128, kv_rank=s["rank"],
                                                              scale=(128 + s["rot"]) ** -0.5, mask=dict(size=s["latent_window"]),
                                                              rot=dict(base=10000.0, dims=s["rot"])))
    att = dict(type="attention", mlp=mlp, mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5,
                                                     rot=dict(base=500000.0, dims=128, scaling=bands)))
    return dict(architecture="Fegolorn", vocab=vocab, width=s["width"], norm=dict(eps=1e-5), logit_softcap=30.0, layers=[lat, att] * s["pairs"],
                embedding=dict(scale=1.0, bigram=dict(buckets=16381, mul_prev=8191, mul_cur=127)))


def sapudra_with_those_experts(s, runs, vocab=32000):
    from lorax_b200.config import ModelConfig
    return ModelConfig.from_dict(sapudra_config(dict(s, layers=runs, ff=s["ff"] * 3 // 2, groups=(1, 1)), vocab))


def latent_attention_of_that_size(s, runs, vocab=32000):
    from lorax_b200.config import ModelConfig
    lat = dict(type="latent_attention", mlp=dict(kind="dense", ff=s["dense"]),
               mixer=dict(heads=s["heads"], dim=128, rot_dim=s["rot"], vdim=128, q_rank=s["width"] // 2, kv_rank=s["rank"],
                          scale=(128 + s["rot"]) ** -0.5, rot=dict(base=10000.0, dims=s["rot"])))
    return ModelConfig.from_dict(dict(architecture="Vabunex", vocab=vocab, width=s["width"], norm=dict(eps=1e-5), embedding=dict(scale=1.0),
                                      layers=[lat] * runs))


# sizes, configuration of the design, and what runs beside it
DESIGNS = {"vabunex": (VABUNEX_SIZES, vabunex_config, [("llama-like", llama_like)]),
           "sapudra": (SAPUDRA_SIZES, sapudra_config, [("mixtral-like", mixtral_like)]),
           "saredra": (SAREDRA_SIZES, saredra_config, [("sapudra", sapudra_of_that_size), ("linear-attention", linear_attention_of_that_size)]),
           "fegolorn": (FEGOLORN_SIZES, fegolorn_config, [("sapudra", sapudra_with_those_experts), ("latent-attention", latent_attention_of_that_size)])}


def peaks():
    try:
        with open(os.path.join(REPO, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "of measured"
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15, "of fallback"


class OpTimer:
    """Wraps the operators of `ops.native` for eager passes: flush L2, event, call, event; knows each operator's algorithmic bytes
    and FLOPs."""

    FLUSH_BYTES = 256 << 20

    def __init__(self, native, names, inp_info):
        import torch
        self.nv, self.names, self.info = native, names, inp_info
        self.flush = torch.empty(self.FLUSH_BYTES, dtype=torch.uint8, device="cuda")
        self.records, self.saved = [], {}

    def __enter__(self):
        import torch
        self.inside = False

        def wrap(name, fn):
            def timed(*a, **kw):
                if self.inside:                             # an operator inside another one belongs to that one's time
                    return fn(*a, **kw)
                self.inside = True
                self.flush.zero_()
                s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                s.record()
                out = fn(*a, **kw)
                e.record()
                self.inside = False
                if out is False:                            # (the operator declined; nothing was launched)
                    return out
                self.records.append((name, self.cost(name, a, kw), s, e))
                return out
            return timed
        for n in self.names:
            self.saved[n] = getattr(self.nv, n)
            setattr(self.nv, n, wrap(n, self.saved[n]))
        return self

    def __exit__(self, *exc):
        for n, fn in self.saved.items():
            setattr(self.nv, n, fn)

    def cost(self, name, a, kw):
        """(label, bytes, flops) of one call."""
        nb = lambda *ts: sum(t.numel() * t.element_size() for t in ts if t is not None)
        q = self.info                                       # sequences, their tokens, decode?, window of a uniform model

        def pairs(window):
            """(query, key) pairs of the step, a decode row's keys counting once."""
            n, w = q["length"], window if window and window > 0 else 1 << 30
            if q["decode"]:
                return q["seqs"] * min(n, w)
            out = max(0, n - w)
            return q["seqs"] * (n * (n + 1) // 2 - out * (out + 1) // 2)
        if name == "gemm":
            x, w = a[0], a[1]
            return (f"gemm [{x.shape[0]}, {w.shape[1]}] x [{w.shape[0]}]", nb(x, w) + x.shape[0] * w.shape[0] * 2, 2 * x.shape[0] * w.numel())
        if name == "gemm_stack":
            x, w = a
            return ("gemm_stack", nb(x, w) + x.shape[0] * x.shape[1] * w.shape[1] * 2, 2 * x.shape[1] * w.numel())
        if name == "gemm_heads":
            x, w, out = a[:3]
            H, N, K = w.shape
            return (f"gemm_heads {N}x{K}", nb(w) + x.shape[0] * H * (N + K) * 2, 2 * x.shape[0] * w.numel())
        if name in ("linear_attn", "wkv"):
            H, d = (a[3], a[4]) if name == "linear_attn" else (a[6], a[7])
            dv = a[5] if name == "linear_attn" else d
            T = a[0].shape[0]
            io = T * H * (2 * d + dv) * 2 + T * H * dv * 4 + (T * H * d * 2 if name == "wkv" else 0)
            st = q["seqs"] * H * d * dv * 4 * (2 if q["decode"] else 1)
            return (name, io + st, 0)
        if name == "ssd":
            T, H, G, n, p = a[0].shape[0], *a[2:6]
            st = q["seqs"] * H * n * p * 4 * (2 if q["decode"] else 1)
            return (name, T * (H * p + 2 * G * n + H) * 2 + T * H * p * 4 + st, 0)
        if name == "causal_conv":
            taps, C = a[1].shape
            return (name, a[0].shape[0] * C * 4 + q["seqs"] * (taps - 1) * C * (4 if q["decode"] else 2), 0)
        if name == "conv_rope_kvwrite":
            T, H, G, dk, dv = a[0].shape[0], *a[1:5]
            w = a[10] if len(a) > 10 else None
            kept = q["seqs"] * (w.shape[0] - 1) * w.shape[1] * (4 if q["decode"] else 2) if w is not None else 0
            return (name + (" with conv" if w is not None else ""), T * 2 * (H * dk + G * (dk + dv)) * 2 + kept, 0)
        if name == "gate_norm":
            T, H, p = a[0].shape[0], a[2], a[3]
            return (name, T * H * p * (4 + 2 + 2), 0)
        if name == "latent_attn":
            H, kv, rot = a[3], a[4], a[7]
            T = a[0].shape[0]
            ctx = pairs(kw.get("window"))
            if q["decode"]:                                 # absorbed: rows of the cache against every head
                return (name, ctx * (kv + rot) * 2 + T * H * (2 * kv + rot) * 2, 2 * ctx * H * (2 * kv + rot))
            return (name, 0, 2 * ctx * H * (128 + rot + 128))       # the products of plain multi-head attention
        if name == "latent_prefill":                        # expansion of the contexts, then multi-head attention
            w, H, dk, rot, dv = a[2], *a[5:9]
            return (name, 0, 2 * q["seqs"] * q["length"] * w.numel() + 2 * pairs(kw.get("window")) * H * (dk + rot + dv))
        if name == "attn_decode":
            nh, nkv, d = a[4], a[5], a[6]
            ctx = pairs(q["window"])
            return (name, ctx * nkv * 2 * d * 2 + a[0].shape[0] * nh * d * 4, 4 * ctx * nh * d)
        if name == "attn_prefill":
            nh, d = a[7], a[9]
            return (name, 0, 4 * pairs(q["window"]) * nh * d)
        if name == "gqa_attn":
            H, G, dk, dv = a[2:6]
            ctx = pairs(a[7])
            if q["decode"]:
                return (name, ctx * G * (dk + dv) * 2 + a[0].shape[0] * H * (dk + dv) * 2, 2 * ctx * H * (dk + dv))
            return (name, 0, 2 * ctx * H * (dk + dv))
        if name == "qk_norm_kvwrite":
            T, H, G, dk, dv = a[0].shape[0], *a[1:5]
            return (name, T * 2 * (H * dk + G * (dk + dv)) * 2, 0)
        if name == "norm_add":
            r, y, pr, z = a[0], a[1], kw.get("pairs"), kw.get("gate")
            n = (kw["rows"] if kw.get("rows") is not None else r).shape[0] * r.shape[1]
            per = 2 * (pr[0].shape[1] if pr is not None else 1) + (2 if z is not None else 0) + (4 if kw.get("rows") is not None else 8) + 2
            return ("norm_add" + (" of experts" if pr is not None else "") + (" with gate and next norm" if z is not None else ""), n * per, 0)
        if name == "moe_route":
            x, w, k = a[:3]
            rows = k + (1 if kw.get("shared") else 0)
            return (name, nb(x, w) + nb(x) * rows, 2 * x.shape[0] * w.numel())
        if name == "moe_grouped_gemm":
            xg, w, seg = a[:3]
            sizes = seg.diff()
            rows = int(sizes.sum())
            cols = w.shape[1] // (2 if kw.get("act") == "swiglu" else 1)
            return (f"moe_grouped_gemm {w.shape[1]}x{w.shape[2]}", nb(xg) + int((sizes > 0).sum()) * w[0].numel() * 2 + rows * cols * 2,
                    2 * rows * w[0].numel())
        if name == "moe_combine":
            y, k, out = a[0], a[3], a[4]
            return (name, nb(out) * (k + 1), 0)
        if name == "norm_stream":
            r, pend = a[0] if kw.get("rows") is None else a[0][: kw["rows"].shape[0]], a[1]
            pairs = kw.get("pairs")
            more = 0 if pend is None else r.numel() * pend.element_size() * (pairs[0].shape[1] if pairs is not None else 1)
            return (name + (" of experts" if pairs is not None else ""), nb(r) * (2 if pend is not None else 1) + more + r.numel() * 2, 0)
        if name == "norm_residual":
            return (name, nb(a[0]) * 2 + nb(a[1]) * 2, 0)
        if name == "norm_gate":
            return (name, nb(a[0]) + a[0].numel() * 4, 0)
        if name == "token_shift":
            return (name, nb(a[0]) * (1 + a[1].shape[0]), 0)
        if name == "act_mul":
            return (name, a[0].shape[0] * a[1] * (6 if kw.get("gated", True) else 4), 0)
        if name == "rope_kvwrite":
            T, nh, nkv, d = a[0].shape[0], a[5], a[6], a[7]
            return (name, T * (2 * (nh + nkv) * d + 3 * nkv * d) * 2, 0)
        if name == "latent_prep":
            cq, q_rot = a[2].shape[0] if a[2] is not None else 0, kw.get("heads", 0) * a[6]
            return (name, a[1].shape[0] * (cq + a[3].shape[0] + a[6] + q_rot) * 4, 0)
        if name == "rope_pairs":
            return (name, a[0].shape[0] * a[3] * a[6] * 4, 0)
        if name in ("embed", "embed_stream"):
            per = 4 if name == "embed" else 6 + (2 if kw.get("pos") is not None else 0) + (2 if kw.get("copy") is not None else 0) + (2 if kw.get("bigram") is not None else 0)
            return (name, a[0].shape[0] * a[1].shape[1] * per, 0)
        return (name, nb(*[t for t in a if hasattr(t, "numel")]), 0)

    def report(self, bw, fl):
        import torch
        torch.cuda.synchronize()
        agg = {}
        for name, (label, nbytes, flops), s, e in self.records:
            agg.setdefault(label, []).append((s.elapsed_time(e) * 1e3, nbytes, flops))
        rows = []
        for label, xs in agg.items():
            us = statistics.median(x[0] for x in xs)
            best = max(xs[0][1] / bw, xs[0][2] / fl) * 1e6
            rows.append((label, len(xs), round(us, 1), round(best / us, 3)))
        return sorted(rows, key=lambda r: -r[1] * r[2])


OPS = ("gemm", "norm_residual", "rope_kvwrite", "act_mul", "embed", "attn_decode", "attn_prefill", "embed_stream", "norm_stream", "norm_gate",
       "tanh_", "gemm_heads", "gemm_stack", "linear_attn", "wkv", "token_shift", "latent_prep", "rope_pairs", "latent_attn", "latent_prefill", "argmax_logprob", "gqa_attn",
       "qk_norm_kvwrite", "conv_rope_kvwrite", "causal_conv", "ssd", "gate_norm", "norm_add", "moe_route", "moe_grouped_gemm", "moe_combine")


def main(args):
    import torch
    from lorax_b200.config import EngineConfig, ModelConfig
    from lorax_b200.models.decoder import DecoderModel
    from lorax_b200.ops import native
    from lorax_b200.runtime.kv_cache import make_cache
    from lorax_b200.runtime.runner import ModelRunner, PrefillItem
    if not torch.cuda.is_available():
        print(json.dumps({"error": "bench.py needs a CUDA device"}))
        return 1
    dev = torch.device("cuda", 0)
    bw, fl, of = peaks()
    steps, warm = min(args.steps, 50), max(3, min(args.warmup, 10))
    from bench import ClockSampler
    results = []
    sizes, config_of, likes = DESIGNS[args.design]
    with torch.inference_mode():
        for size in args.design_size.split(","):
            s = sizes[size]
            ours = ModelConfig.from_dict(config_of(s))
            window = s.get("window", 0)
            for name, cfg in [(args.design, ours)] + [(n, like(s, len(ours.layer_schedule))) for n, like in likes]:
                model = DecoderModel.random_init_on_device(cfg, dev, torch.bfloat16, seed=0, max_positions=20000)
                model.use_native_layers = True
                for kind, cases in (("prefill", PREFILL), ("decode", DECODE)):
                    for n, length in cases:
                        total = length + (8 + 2 * (steps + warm) if kind == "decode" else 0)
                        pages = (total + 31) // 32 + 1
                        kv = make_cache(model, EngineConfig(), n * pages + 1, n, num_slots=n + 1)
                        run = ModelRunner(model, kv, max_batch=n, max_seq_tokens=total + 32, max_prefill_tokens=max(n * length, 64))
                        blocks = [list(range(1 + i * pages, 1 + (i + 1) * pages)) for i in range(n)]
                        g = torch.Generator().manual_seed(1)
                        items = [PrefillItem(torch.randint(0, cfg.vocab_size, (length,), generator=g).tolist(), 0, blocks[i], state_slot=i + 1)
                                 for i in range(n)]
                        if kind == "decode":
                            # (the contents of caches and states do not matter for the time: no prompt is run)
                            rows = [run.state.take_row(i) for i in range(n)]
                            run.install(rows, torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist(), [length] * n, blocks, [0] * n, list(range(1, n + 1)))
                            run.resort()
                            step = lambda: run.decode()
                            info = dict(decode=True, seqs=n, length=length, window=window)
                            toks = n
                        else:
                            inp, _ = run._prefill_inputs(items)
                            step = lambda: model.forward(inp, kv.layers)
                            info = dict(decode=False, seqs=n, length=length, window=window)
                            toks = n * length
                        time.sleep(1.0)                      # no case inherits the heat of the one before
                        for _ in range(warm):
                            step()
                        torch.cuda.synchronize()
                        clk = ClockSampler(0, 0.05)
                        clk.start()
                        k = steps if kind == "decode" else max(3, min(steps, 10))
                        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                        e0.record()
                        for _ in range(k):
                            step()
                        e1.record()
                        torch.cuda.synchronize()
                        clocks = clk.stop()
                        ms = e0.elapsed_time(e1) / k
                        # per operator, eager, one launch at a time
                        model.use_native_layers = False
                        graphs, run.use_graphs = run.use_graphs, False
                        with OpTimer(native, OPS, info) as tm:
                            for _ in range(3):
                                step()
                            kernels = tm.report(bw, fl)
                        run.use_graphs, model.use_native_layers = graphs, True
                        native.workspace(dev).check_status()
                        r = {"design": name, "size": size, "kind": kind, "sequences": n, "tokens": length, "ms": round(ms, 3),
                             "tok_s": round(toks / ms * 1e3, 1), "layer_runs": len(model.schedule), "roofline": of,
                             "clocks": {c: clocks[c] for c in ("sm_mhz", "sm_max_mhz", "reasons")},
                             "kernels": [dict(op=a, calls=b // 3, us=c, roofline=d) for a, b, c, d in kernels]}
                        results.append(r)
                        print(json.dumps(r), flush=True)
                        del run, kv, step
                        torch.cuda.empty_cache()
                del model
                torch.cuda.empty_cache()
    return 0
