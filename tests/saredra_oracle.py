"""Plain, slow statement of the Saredra decoder, one function per mechanism, for the tests.

Everything is float64 over one whole sequence; nothing is shared with `lorax_b200`.  Weights come as a dict of tensor name ->
tensor with linear maps stored [out, in]; the configuration is the parsed config.json.
"""

import math

import torch

F64 = torch.float64


def linear(w, x, b=None):
    y = x @ w.t()
    return y if b is None else y + b


def rms_norm(x, w, eps):
    """Over the last dimension, with a plain weight."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def causal_conv(u, w, b=None):
    """u [T, C], w [C, taps]: the last tap belongs to the token itself, tokens before the first are zero."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for back in range(min(taps, t + 1)):
            y[t] += w[:, taps - 1 - back] * u[t - back]
    return y if b is None else y + b


def frequencies(rot):
    """-> (angle per position of every pair, factor on cos and sin)"""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=F64), 1.0
    turns = lambda t: n * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, rot, first=0):
    """x [T, heads, dim]: pairs of neighbours among the first rot.dims dimensions."""
    f, mult = frequencies(rot)
    a = torch.arange(first, first + x.shape[0], dtype=F64)[:, None, None] * f
    cos, sin = a.cos() * mult, a.sin() * mult
    y = x.clone()
    n = rot["dims"]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2], y[..., 1:n:2] = u * cos - v * sin, v * cos + u * sin
    return y


def window_mask(T, size):
    """[T, T] bool: query i sees the keys i - size + 1 .. i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def attend(q, k, v, scale, size, cap, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; sink [H]: a score that is in the denominator only.  -> [T, H, dv]"""
    T, H, _ = q.shape
    per = H // k.shape[1]
    mask = window_mask(T, size)
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // per].t() * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        s = s.masked_fill(~mask, float("-inf"))
        m = torch.maximum(s.max(-1).values, sink[h])[:, None]
        e = torch.exp(s - m)
        out.append(e @ v[:, h // per] / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - m)))
    return torch.stack(out, 1)


def window_attention(h, W, p, m, kv=None):
    """The left mixer and the attention mixer.  Which of the branches apply shows in the tensors there are: biases, convolutions, a
    learned sink, an output gate.  kv: keys and values of another layer.  -> (output before its projection, own keys and values)"""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]

    def project(name, heads):
        u = linear(W[p + name], h, W.get(p + name + ".b"))
        if p + name + ".conv" in W:
            u = causal_conv(u, W[p + name + ".conv"])
        return u.view(T, heads, -1)
    q = rotate(project("q", H), m["rot"])
    if kv is None:
        kv = rotate(project("k", G), m["rot"]), project("v", G)
    sink = W[p + "sink"] if p + "sink" in W else torch.zeros(H, dtype=F64)
    size = m["mask"]["size"] if m.get("mask") else T
    y = attend(q, kv[0], kv[1], m["scale"], size, m.get("softcap"), sink).reshape(T, -1)
    if p + "g" in W:
        y = y * sigmoid(linear(W[p + "g"], h))
    return y, kv


def ssd(x, B, C, dt, A_log, D):
    """x [T, H, P], B, C [T, G, N], dt [T, H] (after softplus): the recurrence token by token.  -> y [T, H, P]"""
    T, H, P = x.shape
    group = [h // (H // B.shape[1]) for h in range(H)]
    y, S = torch.zeros_like(x), torch.zeros(H, B.shape[2], P, dtype=F64)
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + (dt[t][:, None] * B[t, group])[:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t, group][:, :, None]).sum(1) + D[:, None] * x[t]
    return y


def gated_group_norm(y, z, w, groups, eps):
    """The gate first, then every one of `groups` equal parts divided by its own root mean square."""
    y = (y * silu(z)).view(y.shape[0], groups, -1)
    y = y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)
    return y.reshape(y.shape[0], -1) * w


def mamba2(h, W, p, m, eps):
    """-> output before its projection"""
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xBC, dt = torch.split(linear(W[p + "in"], h), [inner, inner + 2 * G * N, H], -1)
    xBC = silu(causal_conv(xBC, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = torch.split(xBC, [inner, G * N, G * N], -1)
    dt = softplus(dt + W[p + "dt_bias"])
    y = ssd(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), dt, W[p + "A_log"], W[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, W[p + "norm"], m["norm_groups"], eps)


def feed_forward(h, W, p):
    return linear(W[p + "down"], silu(linear(W[p + "gate"], h)) * linear(W[p + "up"], h))


def route(z, router):
    """Router logits z [T, E] -> (chosen experts [T, top], their weights)."""
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    choice, groups = s, router.get("groups")
    if groups:
        T, E = z.shape
        g = s.view(T, groups["count"], E // groups["count"])
        best = g.max(-1).values.topk(groups["keep"], -1).indices
        keep = torch.zeros(T, groups["count"], dtype=torch.bool)
        for t in range(T):
            keep[t, best[t]] = True
        choice = g.masked_fill(~keep[:, :, None], float("-inf")).view(T, E)
    ids = choice.topk(router["top"], -1).indices
    return ids, torch.gather(s, 1, ids)


def mixture(h, W, p, mlp):
    ids, w = route(linear(W[p + "router"], h), mlp["router"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        at = (ids == e).nonzero()
        if len(at):
            t, j = at[:, 0], at[:, 1]
            out.index_add_(0, t, w[t, j][:, None] * feed_forward(h[t], W, p + f"e{e}."))
    return out


def mix(h, W, p, spec, eps, kv_of, i):
    m = spec["mixer"]
    if spec["type"] == "parallel":
        left, kv_of[i] = window_attention(h, W, p + "left.", m["left"])
        right = mamba2(h, W, p + "right.", m["right"], eps)
        return m["left_scale"] * linear(W[p + "left.o"], left) + m["right_scale"] * linear(W[p + "right.o"], right)
    y, kv_of[i] = window_attention(h, W, p, m, kv_of[m["kv_from"]] if m.get("kv_from") is not None else None)
    return linear(W[p + "o"], y)


def forward(cfg, weights, tokens, layers_out=None):
    """-> logits [T, vocab] (float64) of one whole sequence; `layers_out` collects the residual after every layer."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps, kv_of = cfg["norm"]["eps"], {}
    x = W["embed"][torch.as_tensor(tokens)]
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mix(rms_norm(x, W[p + "norm1"], eps), W, p + "mix.", spec, eps, kv_of, i)
        mlp = spec.get("mlp")
        if mlp:
            h = rms_norm(x, W[p + "norm2"], eps)
            x = x + (feed_forward(h, W, p + "mlp.") if mlp["kind"] == "dense" else mixture(h, W, p + "mlp.", mlp))
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(W["head"], rms_norm(x, W["final.norm"], eps))


def is_greedy(cfg, weights, prompt, out):
    """Whether every token of `out` is the arg-max behind the prompt and the tokens before it."""
    best = forward(cfg, weights, list(prompt) + list(out[:-1])).argmax(-1)[len(prompt) - 1:]
    return best.tolist() == list(out)
