"""The Ravenex step functions: prompt portions and batched decode over a paged cache of latents.

A layer with latents of its own writes one row per token (normed latent, rotated key part) into the pages; a layer that
reads another's has no cache.  Prompts turn the latents that the portion can see into keys and values of every head and run
the FlashAttention kernel on them, the shared key part being read in place; decoding moves the query to the latents' side
instead, so that the pages are read once for all heads.  Both see the same rows, so either can go on from the other.

Every sublayer ends in `residual_norm`: its output (for a mixture of experts, the weighted rows of the chosen experts) is
normed and joins the fp32 residual in the kernel that norms the next sublayer's input.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ..serving import PagedKVCache
from .ravenex import MoeConfig, RavenexEngine
from .serving_base import ServingModel


class RavenexModel(ServingModel):
    def __init__(self, engine: RavenexEngine, num_blocks: int, block_size: int = 16, graphs: bool = True):
        super().__init__(engine, block_size, graphs)
        # the pages of a layer hold a latent and the rotated key part as one key of one head; there are no values beside it
        self.cache = PagedKVCache.per_layer([None if lay.mix.c_norm is None else (1, lay.mix.c + lay.mix.r, 0) for lay in engine.layers],
                                            num_blocks, block_size, engine.device, engine.dtype)
        self.page_copies = block_size in (8, 16) or block_size % 32 == 0          # what the decode kernel on latents copies whole
        self.source = [i if lay.cfg.mixer.kv_from is None else lay.cfg.mixer.kv_from for i, lay in enumerate(engine.layers)]
        # per layer with latents: the windows of the layers that want them unrolled in prompts
        self.windows = {j: [lay.cfg.mixer.window for i, lay in enumerate(engine.layers) if self.source[i] == j and lay.mix.tensor_cores]
                        for j in set(self.source)}

    # ------------------------------------------------------------------ the layers
    def _feed_forward(self, lay, h) -> dict:
        """The output on its way into the residual (arguments of `residual_norm`)."""
        K, f = self.e.K, lay.mlp
        if not isinstance(lay.cfg.mlp, MoeConfig):
            return dict(y=K.glu_mlp(h, f.gu, f.down, "gelu"))
        out = dict(experts=K.moe_experts(h, f.router, f.correction, f.cfg.top, f.gu, f.down, "silu"))
        if f.shared is not None:
            out["y"] = K.glu_mlp(h, f.shared.gu, f.shared.down, "silu")
        return out

    def _layers(self, tok: torch.Tensor, attention):
        """The residual [T, width] after the last layer but its last sublayer, and that sublayer's output on its way in."""
        e, K = self.e, self.e.K
        cfg = e.cfg
        opt = dict(dtype=e.dtype, mult=cfg.residual_mult)
        x = torch.empty(tok.shape[0], cfg.width, dtype=torch.float32, device=e.device)
        pending = dict(tokens=tok, embed=e.embed)
        for i, lay in enumerate(e.layers):
            h = K.residual_norm(x, cfg.eps, norm=lay.norm1, **opt, **pending)
            o = attention(i, lay, K.linear(h, lay.mix.w_in))
            pending = dict(y=K.linear(o, lay.mix.o), y_norm=lay.norm1b)
            if lay.mlp is not None:
                h = K.residual_norm(x, cfg.eps, norm=lay.norm2, **opt, **pending)
                pending = dict(self._feed_forward(lay, h), y_norm=lay.norm2b)
            if cfg.side_dim:
                h = K.residual_norm(x, cfg.eps, **opt, **pending)
                g = K.token_gate(K.linear(h, lay.side_gate), tok, e.side_embed, i * cfg.side_dim, cfg.side_dim)
                pending = dict(y=K.linear(g, lay.side_proj), y_norm=lay.side_norm)
        return x, pending

    def _logits(self, hidden, rows: Optional[List[int]] = None) -> torch.Tensor:
        e, K = self.e, self.e.K
        x, pending = hidden
        if rows is not None:
            rows = torch.tensor(rows, dtype=torch.int32, device=e.device)
        h = K.residual_norm(x, e.cfg.eps, norm=e.final_norm, dtype=e.dtype, mult=e.cfg.residual_mult, rows=rows, write=False, **pending)
        return K.linear(h, e.head, out_dtype=torch.float32)

    def _rope(self, i: int, lay, proj, pos, slots, q_out=None, lin=None):
        """Rotates the queries (in place, or into q_out) and writes the layer's own latents, if it has any, to the pages."""
        a, w = lay.cfg.mixer, lay.mix
        self.e.K.latent_rope(proj, a.heads, w.d, w.r, a.rot_dim, pos, slots, freq=w.freq, gain=w.rot_gain, c_off=w.c_off, rank=a.kv_rank,
                             c_norm=w.c_norm, eps=self.e.cfg.eps, cache=self.cache.k[i], q_out=q_out, lin=lin)

    def _on_latents(self, i: int, lay, proj, pos, slots, attend):
        """Attention on the pages themselves, `attend(query [N, heads, c + r], cache)` -> sums of latents [N, heads, c]."""
        K, a, w = self.e.K, lay.cfg.mixer, lay.mix
        n = proj.shape[0]
        q = torch.empty(n, a.heads, w.c + w.r, dtype=proj.dtype, device=proj.device)
        self._rope(i, lay, proj, pos, slots, q_out=q)
        K.head_linear(proj[:, :a.heads * (w.d + w.r)].unflatten(1, (a.heads, w.d + w.r))[..., :w.d], w.w_qk, out=q[..., :w.c])
        return K.head_linear(attend(q, self.cache.k[self.source[i]]), w.w_v).view(n, -1)

    # ------------------------------------------------------------------ prompt portions
    def _prompt_hidden(self, tokens: Sequence[int], start: int, block_ids: Sequence[int], slot: int):
        e, K = self.e, self.e.K
        n, bs = len(tokens), self.block_size
        nb = (start + n + bs - 1) // bs
        host = torch.empty(3 * n + nb, dtype=torch.int32)
        host[:n] = torch.tensor(list(tokens), dtype=torch.int32)
        host[n:2 * n] = torch.arange(start, start + n, dtype=torch.int32)
        host[2 * n:3 * n] = self._slots(block_ids, start, n)
        host[3 * n:] = torch.tensor(list(block_ids[:nb]), dtype=torch.int32)
        d = host.to(e.device, non_blocking=True)
        tok, pos, slots, table = d[:n], d[n:2 * n], d[2 * n:3 * n], d[3 * n:]
        unrolled = {}                                    # layer with latents -> what its readers see of them, one after another

        def before(window):                              # how many earlier tokens the portion's first token sees
            return min(start, window - 1) if window > 0 else start

        def attention(i, lay, proj):
            a, w, j = lay.cfg.mixer, lay.mix, self.source[i]
            lin = None
            if j == i and self.windows[i]:
                prev = max(before(x) for x in self.windows[i])
                rows = unrolled[i] = torch.empty(prev + n, w.c + w.r, dtype=e.dtype, device=e.device)
                if prev:
                    K.kv_gather(self.cache.k[i], None, table, start - prev, prev, rows[:prev], None)
                lin = rows[prev:]
            if not w.tensor_cores:
                if lin is not None:                      # only others unroll them: they are written beside the cache here
                    self._rope(i, lay, proj.clone(), pos, slots, lin=lin)
                return self._on_latents(i, lay, proj, pos, slots,
                                        lambda q, kc: K.window_attn(q, kc, kc, table, pos, D=w.c + w.r, E=w.c, window=a.window, scale=a.scale))
            self._rope(i, lay, proj, pos, slots, lin=lin)
            seen = unrolled[j][unrolled[j].shape[0] - before(a.window) - n:]
            kv = K.linear(seen[:, :w.c], w.w_kv)
            k, v = kv[:, :a.heads * w.d].unflatten(1, (a.heads, w.d)), kv[:, a.heads * w.d:].unflatten(1, (a.heads, w.v))
            q = proj[:, :a.heads * (w.d + w.r)].unflatten(1, (a.heads, w.d + w.r))
            return K.shared_rope_fwd(q, k, seen[:, w.c:], v, scale=a.scale, window=a.window).view(n, -1)

        return self._layers(tok, attention)

    # ------------------------------------------------------------------ one token of every sequence
    def _decode_hidden(self, d: torch.Tensor, S: int, width: int):
        K = self.e.K
        d = d.to(torch.int32)
        tok, pos, slots, ctx = d[0], d[1], d[2], d[3]
        tables = d[5:].t().contiguous()

        def attention(i, lay, proj):
            a, w = lay.cfg.mixer, lay.mix

            def attend(q, kc):
                if w.tensor_cores and self.page_copies:
                    keys = min(a.window, width * self.block_size) if a.window > 0 else width * self.block_size
                    return K.latent_decode(q, kc, tables, ctx, rank=w.c, window=a.window, scale=a.scale, max_keys=keys)
                return K.window_attn(q, kc, kc, tables, pos, D=w.c + w.r, E=w.c, window=a.window, scale=a.scale)
            return self._on_latents(i, lay, proj, pos, slots, attend)

        return self._layers(tok, attention)
