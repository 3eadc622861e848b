"""Plain, slow statement of the Vabunex decoder, one function per mechanism, for the tests.

Everything is float64 and runs token by token over one sequence; nothing is shared with `lorax_b200`.  Weights come as
a dict of tensor name -> tensor with linear maps stored [out, in]; the configuration is the parsed config.json.
"""

import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def linear(w, x):
    return x @ w.t()


def rotate_pairs(x, pos, base):
    """x [..., dims]: elements (2i, 2i + 1) turned by pos * base^(-2i / dims)."""
    dims = x.shape[-1]
    out = x.clone()
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(a) - v * math.sin(a)
        out[..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def linear_attention_scan(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, dv], decay [H].  S <- decay S + k v^T, o = S^T q.  -> (o [T, H, dv], S [H, d, dv])"""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def wkv_scan(r, k, v, w, u, state=None):
    """r, k, w [T, H, d], v [T, H, d], u [H, d].  o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=r.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1))
        S = w[t][:, :, None] * S + kv
    return torch.stack(out), S


def mixer_lightning(h, W, p, m, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(linear(W[p + "q"], h)).view(T, H, d)
    k = silu(linear(W[p + "k"], h)).view(T, H, d)
    v = silu(linear(W[p + "v"], h)).view(T, H, dv)
    o, _ = linear_attention_scan(q, k, v, torch.tensor(m["decay"], dtype=F64))
    o = rms(o.reshape(T, H * dv), eps) * W[p + "norm"]
    return linear(W[p + "o"], o / (1.0 + torch.exp(-linear(W[p + "g"], h))))


def mixer_wkv(h, W, p, m, eps):
    H, d = m["heads"], m["dim"]
    T = h.shape[0]
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    mix = {s: h + (prev - h) * W[p + "mu." + s] for s in "rkvgw"}
    r, k, v = (linear(W[p + s], mix[s]).view(T, H, d) for s in "rkv")
    gate = silu(linear(W[p + "g"], mix["g"]))
    w = torch.exp(-torch.exp(linear(W[p + "w2"], torch.tanh(linear(W[p + "w1"], mix["w"]))) + W[p + "w0"])).view(T, H, d)
    o, _ = wkv_scan(r, k, v, w, W[p + "u"])
    o = rms(o, eps).reshape(T, H * d)
    return linear(W[p + "o"], o * W[p + "norm"] * gate)


def mixer_latent_attention(h, W, p, m, eps):
    H, d, rd, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    T = h.shape[0]
    cq = rms(linear(W[p + "dq"], h), eps) * W[p + "dq.norm"]
    q = linear(W[p + "uq"], cq).view(T, H, d + rd)
    dkv = linear(W[p + "dkv"], h)
    c = rms(dkv[:, :kr], eps) * W[p + "dkv.norm"]
    qr = torch.stack([rotate_pairs(q[t, :, d:], t, base) for t in range(T)])
    kr_ = torch.stack([rotate_pairs(dkv[t, kr:], t, base) for t in range(T)])
    k = linear(W[p + "uk"], c).view(T, H, d)
    v = linear(W[p + "uv"], c).view(T, H, dv)
    s = torch.einsum("thd,shd->hts", q[:, :, :d], k) + torch.einsum("thd,sd->hts", qr, kr_)
    s = s * m["scale"]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    o = torch.einsum("hts,shd->thd", torch.softmax(s, -1), v)
    o = o / (1.0 + torch.exp(-linear(W[p + "g"], h)))[:, :, None]
    return linear(W[p + "o"], o.reshape(T, H * dv))


MIXERS = {"lightning": mixer_lightning, "wkv": mixer_wkv, "latent_attention": mixer_latent_attention}


def feed_forward(h, W, p):
    return linear(W[p + "down"], gelu_tanh(linear(W[p + "gate"], h)) * linear(W[p + "up"], h))


def schedule(cfg):
    """Layer indices in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, k = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * k + list(range(b, n))


def forward(cfg, weights, tokens, layers_out=None):
    """-> logits [T, vocab] (float64) of one whole sequence; `layers_out` collects the residual after every layer run."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i in schedule(cfg):
        spec = cfg["layers"][i]
        h = rms(x, eps) * (1.0 + W[f"l{i}.norm1"])
        y = MIXERS[spec["type"]](h, W, f"l{i}.mix.", spec["mixer"], eps)
        if spec.get("mlp"):
            y = y + feed_forward(h, W, f"l{i}.mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(W["head"], rms(x, eps) * (1.0 + W["final.norm"]))


def greedy(cfg, weights, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, weights, ids)[-1].argmax()))
    return ids[len(prompt):]
