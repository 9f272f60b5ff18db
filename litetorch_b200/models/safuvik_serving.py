"""The Safuvik step functions: prompt portions and batched decode over the paged cache (windowed attention) and the
recurrent state pool (linear recurrence, convolution tail, matrix memory).

Every sublayer is: one kernel that folds the finished sublayer into the residual streams and norms the next input
(`hyper_norm`), one product for all projections that read it, the mixer, the output product.  The mixers' prompt and
decode forms differ only in the kernels they call; both leave keys, values and states so that the other can go on.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ..serving import PagedKVCache, RecurrentStatePool
from .safuvik import ParallelConfig, SafuvikEngine
from .serving_base import ServingModel


class SafuvikModel(ServingModel):
    def __init__(self, engine: SafuvikEngine, num_blocks: int, block_size: int = 16, max_num_seqs: int = 64, graphs: bool = True):
        super().__init__(engine, block_size, graphs)
        self.state_slots = max_num_seqs
        self.tensor_cores = engine.device.type == "cuda" and engine.dtype == torch.bfloat16
        shapes = []
        self.state = RecurrentStatePool(max_num_seqs, engine.device)
        for i, lay in enumerate(engine.layers):
            x = lay.cfg.mixer
            if isinstance(x, ParallelConfig):
                shapes.append((x.left.kv_heads,) + self._head_sizes(x.left.dim, x.left.vdim))
                self.state.add(i, "S", x.right.width)
                self.state.add(i, "ring", x.right.conv, x.right.width)
            else:
                shapes.append(None)
                self.state.add(i, "S", x.heads, x.dim, x.vdim)
                self.state.add(i, "n", 2, x.heads, x.dim)
                self.state.add(i, "m", 2, x.heads)
        self.cache = PagedKVCache.per_layer(shapes, num_blocks, block_size, engine.device, engine.dtype)

    def _head_sizes(self, dim: int, vdim: int):
        """Key and value sizes as stored: the tensor-core kernels take 64 or 128 for both."""
        m = max(dim, vdim)
        if self.tensor_cores and m <= 128:
            return (64, 64) if m <= 64 else (128, 128)
        return (dim + 7) // 8 * 8, (vdim + 7) // 8 * 8

    # ------------------------------------------------------------------ the layers
    def _layers(self, tok: torch.Tensor, parallel, mlstm):
        """Residual streams [T, streams, width] after the last layer but its last sublayer, and that sublayer's output on
        its way into them (arguments of `hyper_norm`)."""
        e, K = self.e, self.e.K
        cfg = e.cfg
        x = torch.empty(tok.shape[0], cfg.streams, cfg.width, dtype=torch.float32, device=e.device)
        pending = dict(tokens=tok, embed=e.embed)
        for i, lay in enumerate(e.layers):
            h = K.hyper_norm(x, lay.norm1, cfg.eps, dtype=e.dtype, inn=lay.hc1.inn, **pending)
            if isinstance(lay.cfg.mixer, ParallelConfig):
                left, right = parallel(i, lay, K.linear(h, lay.w_in))
                pending = dict(y=K.linear(left, lay.left_o), y_norm=lay.left_out, y2=K.linear(right, lay.right_o), y2_norm=lay.right_out)
            else:
                pending = dict(y=K.linear(mlstm(i, lay, K.linear(h, lay.w_in), K.rows_dot(h, lay.w_if)), lay.o))
            pending.update(mix=lay.hc1.mix, out=lay.hc1.out)
            if lay.cfg.mlp is not None:
                h = K.hyper_norm(x, lay.norm2, cfg.eps, dtype=e.dtype, inn=lay.hc2.inn, **pending)
                y = K.linear(K.clamped_glu(K.linear(h, lay.w_gu), lay.cfg.mlp.limit), lay.w_down)
                pending = dict(y=y, mix=lay.hc2.mix, out=lay.hc2.out)
        return x, pending

    def _logits(self, hidden, rows: Optional[List[int]] = None) -> torch.Tensor:
        e, K = self.e, self.e.K
        x, pending = hidden
        if rows is not None:
            rows = torch.tensor(rows, dtype=torch.int32, device=e.device)
        h = K.hyper_norm(x, e.final_norm, e.cfg.eps, dtype=e.dtype, rows=rows, write=False, **pending)
        return K.linear(h, e.head, out_dtype=torch.float32, alpha=e.cfg.logit_scale)

    def _qkv(self, i: int, lay, proj, pos, slots, lin=None):
        a = lay.cfg.mixer.left
        q_off, k_off, v_off = lay.offs[:3]
        return self.e.K.qkv_rope(proj, q_off, k_off, v_off, a.heads, a.kv_heads, a.dim, a.vdim, pos, slots, self.cache.k[i], self.cache.v[i],
                                 freq=lay.freq, rot_dims=a.rot.dims, gain=lay.rot_gain, q_norm=lay.q_norm, k_norm=lay.k_norm,
                                 eps=self.e.cfg.eps, lin=lin)

    @staticmethod
    def _cut(lay, proj):
        """Columns of the fused projection of a parallel layer: head gates, GELU branch, convolution input."""
        x = lay.cfg.mixer
        g, y, c = lay.offs[3:]
        return proj[:, g:g + x.left.heads], proj[:, y:y + x.right.width], proj[:, c:c + x.right.width]

    @staticmethod
    def _cut_mlstm(lay, proj):
        x = lay.cfg.mixer
        q, k, v, g = lay.offs
        hd, he = x.heads * x.dim, x.heads * x.vdim
        return proj[:, q:q + hd], proj[:, k:k + hd], proj[:, v:v + he], proj[:, g:g + he]

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

        def attention(i, lay, proj, gate):
            a = lay.cfg.mixer.left
            kc, vc = self.cache.k[i], self.cache.v[i]
            if not (self.tensor_cores and kc.shape[3] == vc.shape[3] and kc.shape[3] in (64, 128)):
                q = self._qkv(i, lay, proj, pos, slots)
                return K.window_attn(q, kc, vc, table, pos, D=a.dim, E=a.vdim, window=a.window, scale=a.scale, gate=gate)
            # the keys that the portion's first token still sees, then the portion's own, one after another
            prev = min(start, a.window - 1)
            lin = torch.empty(2, prev + n, a.kv_heads, kc.shape[3], dtype=e.dtype, device=e.device)
            q = self._qkv(i, lay, proj, pos, slots, lin=(lin[0, prev:], lin[1, prev:]))
            if prev:
                K.kv_gather(kc, vc, table, start - prev, prev, lin[0], lin[1])
            o, _ = K.flash_fwd(q[None], lin[0][None], lin[1][None], causal=True, scale=a.scale, window=a.window)
            return K.head_gate(o[0], gate, a.vdim)

        def parallel(i, lay, proj):
            gate, y, xin = self._cut(lay, proj)
            left = attention(i, lay, proj, gate).view(n, -1)
            S, ring = self.state[i, "S"][slot], self.state[i, "ring"][slot]
            u = K.conv_causal(xin, lay.x_b, lay.conv, lay.conv_b, ring, start)
            right = K.rglru_scan(u, K.block_diag(u, lay.gates), lay.r_b, lay.i_b, lay.decay, y, lay.y_b, xin, lay.x_b, S, ring,
                                 lay.cfg.mixer.right.conv, start)
            return left, right

        def mlstm(i, lay, proj, logits):
            x = lay.cfg.mixer
            q, k, v, gate = self._cut_mlstm(lay, proj)
            return K.mlstm_prefill(q, k, v, logits, lay.i_b, lay.f_b, x.gate_cap, lay.head_norm, e.cfg.eps, gate, self.state[i, "S"][slot],
                                   self.state[i, "n"][slot], self.state[i, "m"][slot], x.dim, x.vdim, start)

        return self._layers(tok, parallel, mlstm)

    # ------------------------------------------------------------------ one token of every sequence
    def _warm_input(self, host: torch.Tensor) -> torch.Tensor:
        warm = host.clone()
        warm[4] = self.state.scratch                     # a state must advance once per token, not once per pass
        return warm

    def _decode_hidden(self, d: torch.Tensor, S: int, width: int):
        e, K = self.e, self.e.K
        d = d.to(torch.int32)
        tok, pos, slots, ctx, rows = d[0], d[1], d[2], d[3], d[4]
        tables = d[5:].t().contiguous()

        def parallel(i, lay, proj):
            a = lay.cfg.mixer.left
            gate, y, xin = self._cut(lay, proj)
            kc, vc = self.cache.k[i], self.cache.v[i]
            q = self._qkv(i, lay, proj, pos, slots)
            if self.tensor_cores and kc.shape[3] == vc.shape[3] and kc.shape[3] in (64, 128):
                splits = self._splits_for(S * a.kv_heads, min(a.window, width * self.block_size))
                left = K.paged_decode(q, kc, vc, tables, ctx, self.block_size, splits, a.scale, window=a.window, gate=gate, vdim=a.vdim)
            else:
                left = K.window_attn(q, kc, vc, tables, pos, D=a.dim, E=a.vdim, window=a.window, scale=a.scale, gate=gate)
            right = K.rglru_step(xin, lay.x_b, lay.conv, lay.conv_b, lay.gates, lay.r_b, lay.i_b, lay.decay, y, lay.y_b,
                                 self.state[i, "S"], self.state[i, "ring"], rows, pos)
            return left.view(S, -1), right

        def mlstm(i, lay, proj, logits):
            x = lay.cfg.mixer
            q, k, v, gate = self._cut_mlstm(lay, proj)
            return K.mlstm_step(q, k, v, logits, lay.i_b, lay.f_b, x.gate_cap, lay.head_norm, e.cfg.eps, gate, self.state[i, "S"],
                                self.state[i, "n"], self.state[i, "m"], rows, pos, x.dim, x.vdim)

        return self._layers(tok, parallel, mlstm)
