"""A plain, slow statement of the Ravenex decoder in double precision, one function per mechanism, for comparison in
tests.  It keeps no cache: every function takes a whole sequence [T, ...] from its first token, keys and values are made in
full for every head, and experts run one token at a time.  Nothing of the package is imported here."""
import math

import torch

F64 = torch.float64


def d(t):
    return t.to(F64)


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * d(w)


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def rotate(x, base):
    """x [T, ..., n] at positions 0..T-1: the pair (2i, 2i+1) turns by position * base^(-2i/n)."""
    T, n = x.shape[0], x.shape[-1]
    freq = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=F64)
    a = (torch.arange(T, dtype=F64)[:, None] * freq).view((T,) + (1,) * (x.dim() - 2) + (n // 2,))
    u, v = x[..., 0::2], x[..., 1::2]
    y = torch.empty_like(x)
    y[..., 0::2] = u * torch.cos(a) - v * torch.sin(a)
    y[..., 1::2] = v * torch.cos(a) + u * torch.sin(a)
    return y


def windowed_softmax(score, window):
    """score [H, T, T] -> weights: query i sees keys i - window + 1 .. i (window None: all up to i)."""
    T = score.shape[-1]
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = gap >= 0
    if window is not None:
        seen &= gap < window
    return torch.softmax(score.masked_fill(~seen, -math.inf), -1)


def latent(w, p, cfg, eps, h):
    """What a layer keeps of its tokens: the normed latent [T, rank] and the rotated key part [T, rot] all heads share."""
    y = h @ d(w[p + "dkv"]).t()
    r = cfg["kv_rank"]
    return rms(y[:, :r], eps, w[p + "dkv.norm"]), rotate(y[:, r:], cfg["rot"]["base"])


def latent_attention(w, p, cfg, h, c, k_rot):
    T, H, D, R, E = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"]
    q = (h @ d(w[p + "q"]).t()).view(T, H, D + R)
    q_rot = rotate(q[..., D:], cfg["rot"]["base"])
    k = (c @ d(w[p + "uk"]).t()).view(T, H, D)
    v = (c @ d(w[p + "uv"]).t()).view(T, H, E)
    score = torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    a = windowed_softmax(score * cfg["scale"], (cfg.get("mask") or {}).get("size"))
    return torch.einsum("hij,jhe->ihe", a, v).reshape(T, H * E) @ d(w[p + "o"]).t()


def gated(w, p, h, act):
    return (act(h @ d(w[p + "gate"]).t()) * (h @ d(w[p + "up"]).t())) @ d(w[p + "down"]).t()


def route(z, correction, top):
    """Logits of one token -> (chosen experts, their weights): the correction takes part in the choice only."""
    s = 1 / (1 + torch.exp(-z))
    chosen = torch.argsort(s + d(correction), descending=True, stable=True)[:top]
    return chosen, s[chosen]


def mixture(w, p, cfg, h):
    out = torch.zeros_like(h)
    z = h @ d(w[p + "router"]).t()
    for t in range(h.shape[0]):
        chosen, weight = route(z[t], w[p + "correction"], cfg["router"]["top"])
        for e, a in zip(chosen.tolist(), weight):
            out[t] += a * gated(w, p + "e%d." % e, h[t], silu)
    if cfg.get("shared"):
        out = out + gated(w, p + "shared.", h, silu)
    return out


def feed_forward(w, p, cfg, h):
    return gated(w, p, h, gelu) if cfg["kind"] == "dense" else mixture(w, p, cfg, h)


def token_side(w, p, i, dim, eps, x, tokens):
    """The layer's own slice of the second embedding, gated by the residual and brought back to the model's width."""
    e = d(w["side.embed"])[tokens][:, i * dim:(i + 1) * dim]
    y = (gelu(x @ d(w[p + "side.gate"]).t()) * e) @ d(w[p + "side.proj"]).t()
    return rms(y, eps, w[p + "side.norm"])


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    tokens = torch.as_tensor(list(tokens), dtype=torch.long)
    x = d(w["embed"])[tokens]
    kept = {}
    for i, lay in enumerate(cfg["layers"]):
        p, mix = "l%d." % i, lay["mixer"]
        h = rms(x, eps, w[p + "norm1"])
        src = mix.get("kv_from")
        if src is None:
            src = i
            kept[i] = latent(w, p + "mix.", mix, eps, h)
        x = x + m * rms(latent_attention(w, p + "mix.", mix, h, *kept[src]), eps, w[p + "norm1b"])
        if lay["mlp"] is not None:
            y = feed_forward(w, p + "mlp.", lay["mlp"], rms(x, eps, w[p + "norm2"]))
            x = x + m * rms(y, eps, w[p + "norm2b"])
        if cfg.get("token_side"):
            x = x + m * token_side(w, p, i, cfg["token_side"]["dim"], eps, x, tokens)
        if layers_out is not None:
            layers_out.append(x)
    return rms(x, eps, w["final.norm"]) @ d(w["head"]).t()
