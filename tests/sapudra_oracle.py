"""Plain, slow statement of the Sapudra decoder, one function per mechanism, for the tests.

Everything is float64 over one whole sequence; nothing is shared with `lorax_b200`.  Weights come as a dict of tensor name ->
tensor with linear maps stored [out, in]; the configuration is the parsed config.json.
"""

import torch

F64 = torch.float64


def linear(w, x):
    return x @ w.t()


def rms_norm(x, w, eps):
    """Over the last dimension, with a plain weight."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def relu2(z):
    return torch.clamp(z, min=0.0) ** 2


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def embed(W, tokens, first=0):
    ids = torch.as_tensor(tokens)
    return W["embed"][ids] + W["pos"][first: first + len(ids)]


def window_mask(T, size):
    """[T, T] bool: query i sees the keys i - size + 1 .. i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def attend(q, k, v, scale, size):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h reads key/value head h // (H / G).  -> [T, H, dv]"""
    T, H, _ = q.shape
    per = H // k.shape[1]
    mask = window_mask(T, size)
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // per].t() * scale
        out.append(torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ v[:, h // per])
    return torch.stack(out, 1)


def attention(h, W, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(linear(W[p + "q"], h).view(T, H, d), W[p + "q.norm"], eps)
    k = rms_norm(linear(W[p + "k"], h).view(T, G, d), W[p + "k.norm"], eps)
    v = linear(W[p + "v"], h).view(T, G, dv)
    return linear(W[p + "o"], attend(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, H * dv))


def feed_forward(h, W, p):
    return linear(W[p + "down"], relu2(linear(W[p + "up"], h)))


def route(z, correction, router):
    """Router logits z [T, E] -> (chosen experts [T, top], their weights)."""
    s = sigmoid(z)
    choice = s + correction
    groups = router.get("groups")
    if groups:
        T, E = z.shape
        g = choice.view(T, groups["count"], E // groups["count"])
        score = g.sort(-1, descending=True).values[:, :, :2].sum(-1)
        best = score.topk(groups["keep"], -1).indices
        keep = torch.zeros_like(score, dtype=torch.bool)
        for t in range(T):
            keep[t, best[t]] = True
        choice = g.masked_fill(~keep[:, :, None], float("-inf")).view(T, E)
    ids = choice.topk(router["top"], -1).indices
    w = torch.gather(s, 1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def mixture(h, W, p, mlp):
    ids, w = route(linear(W[p + "router"], h), W[p + "correction"], mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(ids[t].tolist(), w[t]):
            out[t] += we * feed_forward(h[t:t + 1], W, p + f"e{e}.")[0]
    if mlp.get("shared"):
        out = out + sigmoid(linear(W[p + "shared.sg"], h)) * feed_forward(h, W, p + "shared.")
    return out


def forward(cfg, weights, tokens, layers_out=None):
    """-> logits [T, vocab] (float64) of one whole sequence; `layers_out` collects the residual after every layer."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embed(W, tokens)
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + m * layer_norm(attention(x, W, p + "mix.", spec["mixer"], eps), W[p + "norm1"], W[p + "norm1.b"], eps)
        mlp = spec.get("mlp")
        if mlp:
            y = feed_forward(x, W, p + "mlp.") if mlp["kind"] == "dense" else mixture(x, W, p + "mlp.", mlp)
            x = x + m * layer_norm(y, W[p + "norm2"], W[p + "norm2.b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    z = linear(W["head"], layer_norm(x, W["final.norm"], W["final.norm.b"], eps))
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z


def greedy(cfg, weights, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, weights, ids)[-1].argmax()))
    return ids[len(prompt):]
