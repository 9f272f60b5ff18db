"""A plain, slow statement of the Safuvik decoder in double precision, one function per mechanism, for comparison in
tests.  It keeps no cache and no state between calls: every function takes a whole sequence [T, ...] from its first
token, and recurrences are walked one token at a time.  Nothing of the package is imported here."""
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


def inverse_frequencies(rot):
    """One angle per token and pair: base^(-2i/n), stretched by YaRN when the configuration has a scaling."""
    n, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(freq, dtype=F64), 1.0

    def turn(t):
        return n * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(turn(sc["fast"])), 0)
    hi = min(math.ceil(turn(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * r + f * (1 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, dim] at positions 0..T-1: neighbouring pairs (2i, 2i+1) of the first rot.dims dimensions turn."""
    freq, gain = inverse_frequencies(rot)
    n = rot["dims"]
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * freq[None, :]
    c, s = (torch.cos(a) * gain)[:, None, :], (torch.sin(a) * gain)[:, None, :]
    y = x.clone()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2] = u * c - v * s
    y[..., 1:n:2] = v * c + u * s
    return y


def window_attention(q, k, v, scale, window):
    """q [T, H, D], k [T, G, D], v [T, G, E]: softmax over the `window` newest keys, the query's own included."""
    T, H, _ = q.shape
    k, v = (t.repeat_interleave(H // t.shape[1], 1) for t in (k, v))
    score = torch.einsum("ihd,jhd->hij", q, k) * scale
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    score = score.masked_fill(~((gap >= 0) & (gap < window)), -math.inf)
    return torch.einsum("hij,jhe->ihe", torch.softmax(score, -1), v)


def gated_window_attention(w, p, cfg, eps, h):
    T = h.shape[0]
    H, G, D, E = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = rms(h @ d(w[p + "q"]).t(), eps, w[p + "q.norm"]).view(T, H, D)
    k = rms(h @ d(w[p + "k"]).t(), eps, w[p + "k.norm"]).view(T, G, D)
    v = (h @ d(w[p + "v"]).t()).view(T, G, E)
    o = window_attention(rotate(q, cfg["rot"]), rotate(k, cfg["rot"]), v, cfg["scale"], cfg["mask"]["size"])
    o = o * torch.sigmoid(h @ d(w[p + "g"]).t())[..., None]
    return o.reshape(T, H * E) @ d(w[p + "o"]).t()


def causal_conv(x, weight, bias):
    """x [T, C], weight [C, taps]: the last tap meets the current token, zeros before the first."""
    T, C = x.shape
    taps = weight.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x])
    return sum(pad[j:j + T] * d(weight)[:, j] for j in range(taps)) + d(bias)


def block_diagonal(x, weight, bias):
    """x [T, C], weight [B, C/B, C/B] as [block, out, in]."""
    B = weight.shape[0]
    y = torch.einsum("tbi,boi->tbo", x.view(x.shape[0], B, -1), d(weight)) + d(bias)
    return y.reshape(x.shape[0], -1)


def gated_linear_recurrence(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -8 r_t softplus(lam), S = 0 at the start."""
    log_a = -8.0 * r * torch.log1p(torch.exp(d(lam)))
    s, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        s = torch.exp(log_a[t]) * s + torch.sqrt(1 - torch.exp(2 * log_a[t])) * i[t] * u[t]
        out.append(s)
    return torch.stack(out)


def recurrent_block(w, p, h):
    y = gelu(h @ d(w[p + "y"]).t() + d(w[p + "y.b"]))
    u = causal_conv(h @ d(w[p + "x"]).t() + d(w[p + "x.b"]), w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_diagonal(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_diagonal(u, w[p + "ri"], w[p + "ri.b"]))
    return (gated_linear_recurrence(u, r, i, w[p + "lam"]) * y) @ d(w[p + "o"]).t()


def parallel_mixer(w, p, cfg, eps, h):
    left = gated_window_attention(w, p + "left.", cfg["left"], eps, h)
    right = recurrent_block(w, p + "right.", h)
    return 0.5 * (rms(left, eps, w[p + "left.out"]) + rms(right, eps, w[p + "right.out"]))


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, E], log gates i, f [T, H]; the running maximum starts at 0.  Returns [T, H, E]."""
    T, H, D = q.shape
    S, n, m = torch.zeros(H, D, v.shape[-1], dtype=F64), torch.zeros(H, D, dtype=F64), torch.zeros(H, dtype=F64)
    out = []
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm_gates(w, p, cap, h):
    i = cap * torch.tanh((h @ d(w[p + "i"]).t() + d(w[p + "i.b"])) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ d(w[p + "f"]).t() + d(w[p + "f.b"])) / cap))
    return i, f


def mlstm_mixer(w, p, cfg, eps, h):
    T, H, D, E = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"]
    q = (h @ d(w[p + "q"]).t()).view(T, H, D) * D ** -0.5
    k = (h @ d(w[p + "k"]).t()).view(T, H, D)
    v = (h @ d(w[p + "v"]).t()).view(T, H, E)
    i, f = mlstm_gates(w, p, cfg["gate_cap"], h)
    o = rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * E) * d(w[p + "norm"])
    return (o * torch.sigmoid(h @ d(w[p + "g"]).t())) @ d(w[p + "o"]).t()


def clamped_glu(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def feed_forward(w, p, cfg, h):
    y = clamped_glu(h @ d(w[p + "gate"]).t(), h @ d(w[p + "up"]).t(), cfg["limit"])
    return y @ d(w[p + "down"]).t()


def hyper_sublayer(w, p, xs, sublayer):
    """xs [T, streams, W]; mix is indexed [from, to]."""
    u = torch.einsum("s,tsw->tw", d(w[p + "in"]), xs)
    y = sublayer(u)
    return torch.einsum("st,nsw->ntw", d(w[p + "mix"]), xs) + d(w[p + "out"])[None, :, None] * y[:, None, :]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence."""
    eps = cfg["norm"]["eps"]
    x = d(w["embed"])[torch.as_tensor(list(tokens), dtype=torch.long)]
    xs = x[:, None, :].repeat(1, cfg["streams"], 1)
    for n, lay in enumerate(cfg["layers"]):
        p = "l%d." % n
        mixer = {"parallel": parallel_mixer, "mlstm": mlstm_mixer}[lay["type"]]
        xs = hyper_sublayer(w, p + "hc1.", xs, lambda u: mixer(w, p + "mix.", lay["mixer"], eps, rms(u, eps, w[p + "norm1"])))
        if lay["mlp"] is not None:
            xs = hyper_sublayer(w, p + "hc2.", xs, lambda u: feed_forward(w, p + "mlp.", lay["mlp"], rms(u, eps, w[p + "norm2"])))
        if layers_out is not None:
            layers_out.append(xs.sum(1))
    return rms(xs.sum(1), eps, w["final.norm"]) @ d(w["head"]).t() * cfg["logit_scale"]
