"""Plain-PyTorch twins of the kernel front-end in `kernels.py`, with the same names, arguments and in-place effects.

`LlamaEngine` and the weight providers pick this module when their tensors live on the CPU, so that the
hand-written forward/backward schedule, the sharding layouts and the collective logic run as gloo ranks in the
test-suite without a GPU (the reference tests its distributed code the same way, by forking CPU ranks:
tests/distributed_test.cpp).  Nothing here is used on a CUDA device.  Arithmetic is done in fp32 and rounded to
the dtype of the output buffer, which is what the kernels do.
"""
from __future__ import annotations

import math

import torch

_launches = [0]


def launch_count() -> int:
    return 0


def reset_launch_count():
    pass


def status_fetch() -> int:
    return 0


def check_status():
    pass


def gemm(a, b, *, a_major=0, b_major=0, out=None, out_dtype=None, bias=None, residual=None, act=0, accumulate=False,
         alpha=1.0, block_n=0, max_ctas=0):
    A = a.float() if a_major == 0 else a.float().t()
    B = b.float().t() if b_major == 0 else b.float()
    y = (A @ B) * alpha
    if bias is not None:
        y = y + bias.float()
    if act == 1:
        y = torch.nn.functional.gelu(y, approximate="tanh")
    if residual is not None:
        y = y + residual.float()
    if out is None:
        return y.to(out_dtype or a.dtype)
    if accumulate:
        out.copy_((out.float() + y).to(out.dtype))
    else:
        out.copy_(y.to(out.dtype))
    return out


def norm_fwd(x, weight, bias=None, residual=None, *, layer_norm=False, eps=1e-5, want_sum=True, out=None):
    xf = x.float()
    s = None
    if residual is not None:
        xf = xf + residual.float()
        s = xf.to(x.dtype) if want_sum else None
        xf = xf.to(x.dtype).float()
    mean = None
    if layer_norm:
        mean = xf.mean(-1)
        xc = xf - mean[:, None]
    else:
        xc = xf
    rstd = torch.rsqrt(xc.pow(2).mean(-1) + eps)
    y = xc * rstd[:, None] * weight.float()
    if bias is not None:
        y = y + bias.float()
    if out is not None:
        out.copy_(y.to(x.dtype))
        return out, s, mean, rstd
    return y.to(x.dtype), s, mean, rstd


def norm_bwd(dy, x, weight, mean, rstd, *, layer_norm=False, dres=None, dw=None, db=None, accumulate=False, out=None):
    xf, g = x.float(), dy.float()
    xc = xf - mean[:, None] if layer_norm else xf
    xhat = xc * rstd[:, None]
    gw = g * weight.float()
    D = x.shape[1]
    if layer_norm:
        dx = (gw - gw.mean(-1, keepdim=True) - xhat * (gw * xhat).mean(-1, keepdim=True)) * rstd[:, None]
    else:
        dx = (gw - xhat * (gw * xhat).sum(-1, keepdim=True) / D) * rstd[:, None]
    if dres is not None:
        dx = dx + dres.float()
    dwv = (g * xhat).sum(0)
    if dw is None:
        dw = dwv.to(weight.dtype)
    elif accumulate:
        dw.copy_((dw.float() + dwv).to(dw.dtype))
    else:
        dw.copy_(dwv.to(dw.dtype))
    if layer_norm:
        dbv = g.sum(0)
        if db is None:
            db = dbv.to(weight.dtype)
        elif accumulate:
            db.copy_((db.float() + dbv).to(db.dtype))
        else:
            db.copy_(dbv.to(db.dtype))
    if out is not None:
        out.copy_(dx.to(x.dtype))
        return out, dw, db
    return dx.to(x.dtype), dw, db


def rope_(x2d, cos, sin, T, heads, head_dim, *, col_offset=0, positions=None, backward=False):
    rows = x2d.shape[0]
    pos = positions.to(torch.int64) if positions is not None else torch.arange(rows, device=x2d.device) % T
    c = cos[pos][:, None, :]
    s = sin[pos][:, None, :]
    if backward:
        s = -s
    blk = x2d[:, col_offset:col_offset + heads * head_dim].float().reshape(rows, heads, head_dim // 2, 2)
    x0, x1 = blk[..., 0], blk[..., 1]
    out = torch.stack([x0 * c - x1 * s, x0 * s + x1 * c], dim=-1).reshape(rows, heads * head_dim)
    x2d[:, col_offset:col_offset + heads * head_dim] = out.to(x2d.dtype)
    return x2d


def swiglu_fwd(gu):
    F = gu.shape[1] // 2
    g, u = gu[:, :F].float(), gu[:, F:].float()
    return (torch.nn.functional.silu(g) * u).to(gu.dtype)


def swiglu_bwd(gu, dh, inplace=True):
    F = gu.shape[1] // 2
    g, u, d = gu[:, :F].float(), gu[:, F:].float(), dh.float()
    sg = torch.sigmoid(g)
    dg = d * u * (sg + g * sg * (1 - sg))
    du = d * g * sg
    out = gu if inplace else torch.empty_like(gu)
    out[:, :F] = dg.to(gu.dtype)
    out[:, F:] = du.to(gu.dtype)
    return out


def embedding_fwd(idx, table):
    idx = idx.reshape(-1).to(torch.int64).clamp(0, table.shape[0] - 1)
    return table[idx].contiguous()


def embedding_bwd(idx, dout, dtable):
    idx = idx.reshape(-1).to(torch.int64)
    ok = (idx >= 0) & (idx < dtable.shape[0])
    acc = dtable.float()
    acc.index_add_(0, idx[ok], dout[ok].float())
    dtable.copy_(acc.to(dtable.dtype))
    return dtable


def ce_stats(logits, targets, vocab_start=0):
    lf = logits.float()
    V = lf.shape[1]
    m = lf.amax(-1)
    s = torch.exp(lf - m[:, None]).sum(-1)
    loc = targets.to(torch.int64) - vocab_start
    inside = (loc >= 0) & (loc < V)
    tl = torch.where(inside, lf.gather(1, loc.clamp(0, V - 1)[:, None])[:, 0], torch.zeros_like(m))
    return torch.stack([m, s, tl], 1).contiguous()


def ce_finish(logits, targets, gstats, *, vocab_start=0, grad_scale=1.0, ignore_index=-100, write_grad=True):
    N, V = logits.shape
    tgt = targets.to(torch.int64)
    valid = tgt != ignore_index
    rows = torch.where(valid, torch.log(gstats[:, 1]) + gstats[:, 0] - gstats[:, 2], torch.zeros_like(gstats[:, 0]))
    if write_grad:
        p = torch.exp(logits.float() - gstats[:, 0:1]) / gstats[:, 1:2]
        loc = tgt - vocab_start
        inside = (loc >= 0) & (loc < V) & valid
        p[torch.arange(N, device=p.device)[inside], loc[inside]] -= 1.0
        p = p * valid[:, None] * grad_scale
        logits.copy_(p.to(logits.dtype))
    return rows


def _expand_kv(k, Hq):
    B, T, Hkv, D = k.shape
    return k if Hkv == Hq else k[:, :, :, None, :].expand(B, T, Hkv, Hq // Hkv, D).reshape(B, T, Hq, D)


def flash_fwd(q, k, v, *, causal=True, scale=None, window=0):
    B, Tq, Hq, D = q.shape
    Tk = k.shape[1]
    scale = (D ** -0.5) if scale is None else scale
    qf = q.float().permute(0, 2, 1, 3)
    kf = _expand_kv(k.float(), Hq).permute(0, 2, 1, 3)
    vf = _expand_kv(v.float(), Hq).permute(0, 2, 1, 3)
    s = qf @ kf.transpose(-1, -2) * scale
    if causal:
        mask = torch.ones(Tq, Tk, dtype=torch.bool, device=q.device).tril(Tk - Tq)
        if window > 0:
            mask = mask.triu(Tk - Tq - window + 1)
        s = s.masked_fill(~mask, float("-inf"))
    lse = torch.logsumexp(s, -1)
    o = torch.exp(s - lse[..., None]) @ vf
    return o.permute(0, 2, 1, 3).contiguous().to(q.dtype), lse.contiguous()


def flash_bwd(q, k, v, o, lse, do, *, causal=True, scale=None, dq=None, dk=None, dv=None):
    B, Tq, Hq, D = q.shape
    _, Tk, Hkv, _ = k.shape
    scale = (D ** -0.5) if scale is None else scale
    qf = q.float().permute(0, 2, 1, 3)
    kf = _expand_kv(k.float(), Hq).permute(0, 2, 1, 3)
    vf = _expand_kv(v.float(), Hq).permute(0, 2, 1, 3)
    dof = do.float().permute(0, 2, 1, 3)
    of = o.float().permute(0, 2, 1, 3)
    s = qf @ kf.transpose(-1, -2) * scale
    if causal:
        mask = torch.ones(Tq, Tk, dtype=torch.bool, device=q.device).tril(Tk - Tq)
        s = s.masked_fill(~mask, float("-inf"))
    p = torch.exp(s - lse[..., None])
    dvf = p.transpose(-1, -2) @ dof
    dp = dof @ vf.transpose(-1, -2)
    delta = (dof * of).sum(-1, keepdim=True)
    ds = p * (dp - delta) * scale
    dqf = ds @ kf
    dkf = ds.transpose(-1, -2) @ qf
    g = Hq // Hkv
    dkf = dkf.reshape(B, Hkv, g, Tk, D).sum(2)
    dvf = dvf.reshape(B, Hkv, g, Tk, D).sum(2)
    res = []
    for buf, val in ((dq, dqf), (dk, dkf), (dv, dvf)):
        val = val.permute(0, 2, 1, 3)
        if buf is None:
            res.append(val.contiguous().to(q.dtype))
        else:
            buf.copy_(val.to(buf.dtype))
            res.append(buf)
    return tuple(res)


def adam_flat(master, grad, m, v, param_bf16, *, lr, beta1, beta2, eps, wd, step, adamw=True, dyn=None):
    g = grad.float()
    if dyn is not None:
        if float(dyn[1]) != 0.0:
            return
        g = g * float(dyn[0])
    bc1 = 1.0 - beta1 ** step
    bc2 = 1.0 - beta2 ** step
    if not adamw and wd != 0.0:
        g = g + wd * master
    m.mul_(beta1).add_(g, alpha=1 - beta1)
    v.mul_(beta2).addcmul_(g, g, value=1 - beta2)
    if adamw:
        master.mul_(1.0 - lr * wd)
    master.addcdiv_(m / bc1, (v / bc2).sqrt() + eps, value=-lr)
    if param_bf16 is not None:
        param_bf16.copy_(master.to(param_bf16.dtype))


def sumsq(x, out):
    out[0] += x.float().pow(2).sum()
    out[1] += (~torch.isfinite(x.float())).sum()
    return out


def clip_coef(stats, dyn, max_norm, inv_scale=1.0):
    norm = math.sqrt(float(stats[0])) * inv_scale
    coef = min(1.0, max_norm / (norm + 1e-6)) if max_norm > 0 else 1.0
    dyn[0] = coef * inv_scale
    dyn[1] = 1.0 if float(stats[1]) != 0.0 else 0.0
    dyn[2] = norm
    return dyn


# ------------------------------------------------------------------------------------------------ hybrid decoders
def clamped_glu(gu, limit, slope=1.702):
    g, u = gu.float().chunk(2, -1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return (g * torch.sigmoid(slope * g) * (u + 1)).to(gu.dtype)


def linear(x, w, out_dtype=None, alpha=1.0):
    return (x.float() @ w.float().t() * alpha).to(out_dtype or x.dtype)


def block_diag(x, w):
    B, N, Kd = w.shape
    return torch.matmul(x.float().view(-1, B, 1, Kd), w.float().transpose(1, 2)).reshape(x.shape[0], B * N)


def rows_dot(x, w):
    return x.float() @ w.float().t()


def _rms(x, eps, w=None):
    y = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def hyper_norm(x, norm, eps, *, dtype, inn=None, tokens=None, embed=None, y=None, y_norm=None, y2=None, y2_norm=None, mix=None,
               out=None, rows=None, write=True):
    xs = x if embed is None else embed[tokens.long()].float()[:, None].expand(x.shape)
    if y is not None:
        y = y.float() if y2 is None else 0.5 * (_rms(y.float(), eps, y_norm) + _rms(y2.float(), eps, y2_norm))
    if rows is not None:
        xs = xs[rows.long()]
        y = None if y is None else y[rows.long()]
    if y is not None:
        xs = torch.matmul(mix.t(), xs) + out[:, None] * y[:, None]
    if write:
        x.copy_(xs)
    u = xs.sum(1) if inn is None else torch.matmul(inn, xs)
    return _rms(u, eps, norm).to(dtype)


def qkv_rope(proj, q_off, k_off, v_off, H, G, D, E, positions, slots, k_cache, v_cache, *, freq, rot_dims, gain=1.0, q_norm=None,
             k_norm=None, eps=1e-6, lin=None):
    N = proj.shape[0]
    bs, DP, EP = k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    angle = positions.double()[:, None] * freq[None]
    c, s = (torch.cos(angle) * gain).float()[:, None], (torch.sin(angle) * gain).float()[:, None]

    def take(off, heads, w):
        t = proj[:, off:off + heads * D].float()
        t = (t if w is None else _rms(t, eps, w)).reshape(N, heads, D).clone()
        u, v = t[..., 0:rot_dims:2].clone(), t[..., 1:rot_dims:2].clone()
        t[..., 0:rot_dims:2], t[..., 1:rot_dims:2] = u * c - v * s, v * c + u * s
        return torch.nn.functional.pad(t, (0, DP - D)).to(proj.dtype)

    q, k = take(q_off, H, q_norm), take(k_off, G, k_norm)
    v = torch.nn.functional.pad(proj[:, v_off:v_off + G * E].reshape(N, G, E), (0, EP - E))
    blk, off = slots.long() // bs, slots.long() % bs
    k_cache[blk, :, off] = k
    v_cache[blk, :, off] = v
    if lin is not None:
        lin[0].copy_(k)
        lin[1].copy_(v)
    return q


def kv_gather(k_cache, v_cache, table, pos0, n, k_lin, v_lin):
    p = torch.arange(pos0, pos0 + n)
    blk, off = table.long()[p // k_cache.shape[2]], p % k_cache.shape[2]
    k_lin.copy_(k_cache[blk, :, off].view_as(k_lin))
    if v_cache is not None:
        v_lin.copy_(v_cache[blk, :, off].view_as(v_lin))


def window_attn(q, k_cache, v_cache, tables, positions, *, D, E, window, scale, gate=None):
    N, H, _ = q.shape
    G, bs = k_cache.shape[1], k_cache.shape[2]
    o = torch.empty(N, H, E, dtype=torch.float32)
    for i in range(N):
        pos = int(positions[i])
        p = torch.arange(max(0, pos - window + 1) if window > 0 else 0, pos + 1)
        t = tables if tables.dim() == 1 else tables[i]
        blk = t.long()[p // bs]
        k = k_cache[blk, :, p % bs][..., :D].float().repeat_interleave(H // G, 1)
        v = v_cache[blk, :, p % bs][..., :E].float().repeat_interleave(H // G, 1)
        w = torch.softmax(torch.einsum("hd,jhd->hj", q[i, :, :D].float(), k) * scale, -1)
        o[i] = torch.einsum("hj,jhe->he", w, v)
    if gate is not None:
        o = o * torch.sigmoid(gate.float())[..., None]
    return o.to(q.dtype)


def head_gate(o, gate, E):
    return (o[..., :E].float() * torch.sigmoid(gate.float())[..., None]).to(o.dtype)


def conv_causal(x, xb, w, b, ring, start):
    N, C = x.shape
    taps = w.shape[1]
    xin = x.float() if xb is None else x.float() + xb
    head = torch.zeros(taps - 1, C)
    for k in range(taps - 1):
        pos = start - (taps - 1) + k
        if pos >= 0:
            head[k] = ring[pos % taps]
    full = torch.cat([head, xin])
    return (sum(full[k:k + N] * w[:, k] for k in range(taps)) + b).to(x.dtype)


def _rglru_coefficients(r, i, u, sp):
    log_a = -8.0 * torch.sigmoid(r) * sp
    return torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * torch.sigmoid(i) * u.float()


def rglru_scan(u, gates, rb, ib, sp, y, yb, x, xb, state, ring, taps, start):
    N, C = u.shape
    B, bw = rb.shape
    g = gates.view(N, B, 2, bw)
    a, b = _rglru_coefficients((g[:, :, 0] + rb).reshape(N, C), (g[:, :, 1] + ib).reshape(N, C), u, sp)
    s = state.clone() if start > 0 else torch.zeros(C)
    out = torch.empty(N, C)
    for t in range(N):
        s = a[t] * s + b[t]
        out[t] = s
    state.copy_(s)
    for t in range(max(0, N - taps), N):
        ring[(start + t) % taps] = x[t].float() + (0 if xb is None else xb)
    return (out * torch.nn.functional.gelu(y.float() + yb, approximate="tanh")).to(u.dtype)


def rglru_step(x, xb, conv_w, conv_b, gates, rb, ib, sp, y, yb, state, ring, slots, positions):
    rows = []
    for s in range(x.shape[0]):
        slot, pos = int(slots[s]), int(positions[s])
        u = conv_causal(x[s:s + 1], xb, conv_w, conv_b, ring[slot], pos)
        rows.append(rglru_scan(u, block_diag(u, gates), rb, ib, sp, y[s:s + 1], yb, x[s:s + 1], xb, state[slot], ring[slot], conv_w.shape[1], pos))
    return torch.cat(rows)


def mlstm_prefill(q, k, v, logits, ib, fb, cap, norm, eps, gate, S, n, m, D, E, start):
    N, H = q.shape[0], S.shape[0]
    i = cap * torch.tanh((logits[:, :H] + ib) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((logits[:, H:] + fb) / cap))
    qf, kf, vf = q.reshape(N, H, D).float() * D ** -0.5, k.reshape(N, H, D).float(), v.reshape(N, H, E).float()
    bank = start & 1
    Sc, nc, mc = (S.clone(), n[bank].clone(), m[bank].clone()) if start > 0 else (torch.zeros_like(S), torch.zeros(H, D), torch.zeros(H))
    o = torch.empty(N, H, E)
    for t in range(N):
        m1 = torch.maximum(f[t] + mc, i[t])
        keep, add = torch.exp(f[t] + mc - m1), torch.exp(i[t] - m1)
        Sc = keep[:, None, None] * Sc + (add[:, None] * kf[t])[:, :, None] * vf[t][:, None, :]
        nc = keep[:, None] * nc + add[:, None] * kf[t]
        mc = m1
        den = torch.maximum((nc * qf[t]).sum(-1).abs(), torch.exp(-mc)) + 1e-6
        o[t] = torch.einsum("hd,hde->he", qf[t], Sc) / den[:, None]
    bank = (start + N) & 1
    S.copy_(Sc)
    n[bank].copy_(nc)
    m[bank].copy_(mc)
    return head_norm_gate(o.view(N, H * E), norm, gate, H, eps)


def mlstm_step(q, k, v, logits, ib, fb, cap, norm, eps, gate, S, n, m, slots, positions, D, E):
    rows = []
    for s in range(q.shape[0]):
        j = slice(s, s + 1)
        slot = int(slots[s])
        rows.append(mlstm_prefill(q[j], k[j], v[j], logits[j], ib, fb, cap, norm, eps, gate[j], S[slot], n[slot], m[slot], D, E, int(positions[s])))
    return torch.cat(rows)


def head_norm_gate(o, w, gate, H, eps):
    R, HE = o.shape
    y = _rms(o.view(R, H, HE // H), eps).reshape(R, HE) * w
    return (y * torch.sigmoid(gate.float())).to(gate.dtype)


# ------------------------------------------------------------------------------------------------ latent attention, experts
_ACT = {"gelu": lambda z: torch.nn.functional.gelu(z, approximate="tanh"), "silu": torch.nn.functional.silu}


def residual_norm(x, eps, *, dtype, norm=None, mult=1.0, y=None, y_norm=None, experts=None, tokens=None, embed=None, rows=None, write=True):
    xs = x if embed is None else embed[tokens.long()].float()
    pick = slice(None) if rows is None else rows.long()
    xs = xs[pick]
    add = None if y is None else y[pick].float()
    if experts is not None:
        z, slots, weight = experts
        e = (z[slots.long()[pick]].float() * weight[pick][..., None]).sum(1)
        add = e if add is None else add + e
    if add is not None:
        xs = xs + mult * (add if y_norm is None else _rms(add, eps, y_norm))
    if write:
        x.copy_(xs)
    return (xs if norm is None else _rms(xs, eps, norm)).to(dtype)


def latent_rope(proj, H, d, r, rot, positions, slots, *, freq, gain=1.0, c_off=-1, rank=0, c_norm=None, eps=1e-6, cache=None, q_out=None,
                lin=None):
    N = proj.shape[0]
    angle = positions.double()[:, None] * freq[None]
    c, s = (torch.cos(angle) * gain).float(), (torch.sin(angle) * gain).float()

    def turn(t, c, s):
        u, v = t[..., 0:rot:2].float(), t[..., 1:rot:2].float()
        y = torch.zeros(t.shape[:-1] + (r,))
        if rot:
            y[..., 0:rot:2], y[..., 1:rot:2] = u * c - v * s, v * c + u * s
        return y.to(proj.dtype)

    q = turn(proj[:, :H * (d + r)].view(N, H, d + r)[..., d:d + rot], c[:, None], s[:, None])
    if q_out is None:
        proj[:, :H * (d + r)].view(N, H, d + r)[..., d:] = q
    else:
        q_out[..., q_out.shape[-1] - r:] = q
    if c_off < 0:
        return
    row = torch.zeros(N, cache.shape[-1], dtype=proj.dtype)
    row[:, :rank] = _rms(proj[:, c_off:c_off + rank].float(), eps, c_norm).to(proj.dtype)
    row[:, cache.shape[-1] - r:] = turn(proj[:, c_off + rank:c_off + rank + rot], c, s)
    bs = cache.shape[2]
    cache[slots.long() // bs, 0, slots.long() % bs] = row
    if lin is not None:
        lin.copy_(row)


def head_linear(x, w, out=None):
    y = torch.einsum("nhk,hmk->nhm", x.float(), w.float()).to(x.dtype).contiguous()
    if out is None:
        return y
    out.copy_(y)
    return out


def shared_rope_fwd(q, k, k_rot, v, *, scale, window=0):
    T, H, d = k.shape
    kk = torch.cat([k, k_rot[:, None].expand(T, H, k_rot.shape[1])], 2)
    return flash_fwd(q[None], kk[None], v[None], causal=True, scale=scale, window=window)[0][0]


def latent_decode(q, cache, tables, ctx, *, rank, window, scale, max_keys):
    return window_attn(q, cache, cache, tables, ctx - 1, D=q.shape[2], E=rank, window=window, scale=scale)


def act_glu(gu, act):
    g, u = gu.float().chunk(2, -1)
    return (_ACT[act](g) * u).to(gu.dtype)


def glu_mlp(x, gu, down, act):
    return linear(act_glu(linear(x, gu), act), down)


def moe_route(logits, correction, top):
    s = torch.sigmoid(logits.float())
    idx = torch.argsort(s + correction, dim=-1, descending=True, stable=True)[:, :top]
    return idx.to(torch.int32), s.gather(1, idx)


def moe_experts(x, router, correction, top, gu, down, act):
    idx, weight = moe_route(rows_dot(x, router), correction, top)
    flat = idx.reshape(-1).long()
    z = torch.empty(flat.numel(), x.shape[1], dtype=x.dtype)
    for e in flat.unique().tolist():
        at = (flat == e).nonzero()[:, 0]
        z[at] = glu_mlp(x[at // top], gu[e], down[e], act)
    return z, torch.arange(flat.numel(), dtype=torch.int32).view(-1, top), weight


def token_gate(g, tokens, table, off, dim):
    e = torch.nn.functional.pad(table[tokens.long(), off:off + dim].float(), (0, g.shape[1] - dim))
    return (_ACT["gelu"](g.float()) * e).to(g.dtype)
