"""Plain, slow statement of the Fegolorn decoder, one function per mechanism, for the tests.

Everything is float64 over one whole sequence; nothing is shared with `lorax_b200`.  Weights come as a dict of tensor name ->
tensor with linear maps stored [out, in]; the configuration is the parsed config.json.
"""

import math

import torch

F64 = torch.float64


def linear(w, x):
    return x @ w.t()


def rms_norm(x, w, eps):
    """Over the last dimension; w is a vector or one number for all of it."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def embed(tokens, W, e):
    """Scaled token vectors plus a vector looked up by the pair (token before, token); nothing before the first token has a row of its own."""
    ids = [int(t) for t in tokens]
    x = W["embed"][torch.tensor(ids)] * e["scale"]
    b = e.get("bigram")
    if b:
        rows = [b["buckets"]] + [(p * b["mul_prev"] + t * b["mul_cur"]) % b["buckets"] for p, t in zip(ids, ids[1:])]
        x = x + W["bigram"][torch.tensor(rows)]
    return x


def frequencies(n, base, scaling=None):
    """Angle per position of every pair.  Scaling: short wavelengths are kept, long ones divided by the factor, blended in between."""
    out = []
    for i in range(n // 2):
        f = base ** (-2.0 * i / n)
        if scaling:
            length, slow = 2 * math.pi / f, f / scaling["factor"]
            if length >= scaling["original"] / scaling["high"]:
                if length > scaling["original"] / scaling["low"]:
                    f = slow
                else:
                    s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                    f = (1.0 - s) * slow + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def turn(x, n, f, first=0, halves=False, back=False):
    """x [T, heads, dim]: the first n dimensions rotated by position * f per pair, pairs being neighbours, or (halves) i and i + n / 2.
    back: the other way round."""
    a = torch.arange(first, first + x.shape[0], dtype=F64)[:, None, None] * f * (-1.0 if back else 1.0)
    cos, sin = a.cos(), a.sin()
    one, two = (slice(0, n // 2), slice(n // 2, n)) if halves else (slice(0, n, 2), slice(1, n, 2))
    y = x.clone()
    u, v = x[..., one], x[..., two]
    y[..., one], y[..., two] = u * cos - v * sin, v * cos + u * sin
    return y


def visible(T, size=None):
    """[T, T] bool: query i sees the keys i - size + 1 .. i (all before it without a size)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < (size or T))


def softmax(s):
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attend(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]"""
    per = q.shape[1] // k.shape[1]
    out = []
    for h in range(q.shape[1]):
        s = (q[:, h] @ k[:, h // per].t() * scale).masked_fill(~mask, float("-inf"))
        out.append(softmax(s) @ v[:, h // per])
    return torch.stack(out, 1)


def grouped_attention(h, W, p, m, eps):
    """Normed queries and keys, turned; values turned to their place and the result turned back from the query's.  -> [T, H * vdim]"""
    T, H, G, rot, dv = h.shape[0], m["heads"], m["kv_heads"], m["rot"], m["vdim"]
    q = rms_norm(linear(W[p + "q"], h).view(T, H, -1), W[p + "q.norm"], eps)
    k = rms_norm(linear(W[p + "k"], h).view(T, G, -1), W[p + "k.norm"], eps)
    f = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    fv = frequencies(dv, rot["base"])
    v = turn(linear(W[p + "v"], h).view(T, G, dv), dv, fv)
    y = attend(turn(q, rot["dims"], f), turn(k, rot["dims"], f), v, m["scale"], visible(T, (m.get("mask") or {}).get("size")))
    return turn(y, dv, fv, back=True).reshape(T, -1)


def latent_attention(h, W, p, m, eps):
    """Keys and values expanded from a normed latent, beside one turned key part for all heads; gated.  -> [T, H * vdim]"""
    T, H, d, r, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    f = frequencies(r, m["rot"]["base"], m["rot"].get("scaling"))
    q = linear(W[p + "q"], h).view(T, H, d + r)
    down = linear(W[p + "dkv"], h)
    c = rms_norm(down[:, :rank], W[p + "dkv.norm"], eps)
    shared = turn(down[:, None, rank:], r, f, halves=True).expand(T, H, r)
    q = torch.cat([q[..., :d], turn(q[..., d:], r, f, halves=True)], -1)
    k = torch.cat([linear(W[p + "uk"], c).view(T, H, d), shared], -1)
    v = linear(W[p + "uv"], c).view(T, H, m["vdim"])
    y = attend(q, k, v, m["scale"], visible(T, (m.get("mask") or {}).get("size"))).reshape(T, -1)
    return y * sigmoid(linear(W[p + "g"], h))


def mixer(h, W, p, spec, eps):
    y = {"attention": grouped_attention, "latent_attention": latent_attention}[spec["type"]](h, W, p, spec["mixer"], eps)
    return linear(W[p + "o"], y)


def clamped_feed_forward(h, W, p, limit):
    g = linear(W[p + "gate"], h).clamp(max=limit)
    u = linear(W[p + "up"], h).clamp(-limit, limit)
    return linear(W[p + "down"], g * sigmoid(1.702 * g) * (u + 1.0))


def expert(h, W, p):
    return linear(W[p + "down"], silu(linear(W[p + "gate"], h)) * linear(W[p + "up"], h))


def route(z, top):
    """Router logits z [T, E] -> (chosen experts [T, top], their weights, which sum to one)."""
    best = z.topk(top, -1)
    return best.indices, softmax(best.values)


def mixture(h, W, p, mlp):
    ids, w = route(linear(W[p + "router"], h) + W[p + "router.b"], mlp["router"]["top"])
    out = expert(h, W, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        at = (ids == e).nonzero()
        if len(at):
            t, j = at[:, 0], at[:, 1]
            out.index_add_(0, t, w[t, j][:, None] * expert(h[t], W, p + f"e{e}."))
    return out


def feed_forward(h, W, p, mlp):
    return clamped_feed_forward(h, W, p, mlp["limit"]) if mlp["kind"] == "dense" else mixture(h, W, p, mlp)


def sublayer(x, W, p, n, inner, eps):
    """The stream plus inner(normed stream), which is gated, normed and scaled on its way."""
    h = rms_norm(x, W[f"{p}norm{n}"], eps)
    y = inner(h) * sigmoid(linear(W[f"{p}rg{n}"], h) + W[f"{p}rg{n}.b"])
    return x + rms_norm(y, W[f"{p}norm{n}b"], eps) * W[f"{p}ls{n}"]


def forward(cfg, weights, tokens, layers_out=None):
    """-> logits [T, vocab] (float64) of one whole sequence; `layers_out` collects the residual after every layer."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, W, cfg["embedding"])
    for i, spec in enumerate(cfg["layers"]):
        while cfg["layers"][i].get("weights_of") is not None:
            i = cfg["layers"][i]["weights_of"]
        p = f"l{i}."
        x = sublayer(x, W, p, 1, lambda h: mixer(h, W, p + "mix.", spec, eps), eps)
        if spec.get("mlp"):
            x = sublayer(x, W, p, 2, lambda h: feed_forward(h, W, p + "mlp.", spec["mlp"]), eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = linear(W["head"], rms_norm(x, W["final.norm"], eps))
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def is_greedy(cfg, weights, prompt, out):
    """Whether every token of `out` is the arg-max behind the prompt and the tokens before it."""
    best = forward(cfg, weights, list(prompt) + list(out[:-1])).argmax(-1)[len(prompt) - 1:]
    return best.tolist() == list(out)
