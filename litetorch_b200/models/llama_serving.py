"""KV-cache serving on the Llama engine's weights: chunked prefill into a paged cache, batched one-token decode on
the split-K paged attention kernel, greedy sampling on the device.

`LlamaKVModel` is the model side of `serving.ServingScheduler.step`: the native scheduler (admission, block tables,
chunked prefill within a token budget, completion) hands it prompt chunks and the running sequences' newest tokens
together with their block tables, and gets next tokens back.  Nothing is recomputed: every token's K and V are
written once (`lt_kv_append`) and read by the attention of later tokens (`lt_paged_decode`, `lt_flash_fwd` for a
prompt chunk).  The reference's counterparts: ContinuousBatchingScheduler::step and its block tables
(src/llm/continuous_batching.cpp:20-197), paged attention (src/ops/attention.cpp:351-477) and flash-decoding
(src/ops/flash_decoding.cpp:13-115); its cache is never filled, here `PagedKVCache.append` is the write path.
"""
from __future__ import annotations

from collections import OrderedDict
from typing import List, Sequence

import torch

from ..serving import PagedKVCache
from .llama import LlamaEngine
from .serving_base import Sampler, ServingModel, generate          # noqa: F401  (their names live here as well)


class LlamaKVModel(ServingModel):
    def __init__(self, engine: LlamaEngine, num_blocks: int, block_size: int = 16, kv_dtype=torch.bfloat16, num_splits: int = 0,
                 graphs: bool = True, prefix_cache_bytes: int = 0):
        assert engine.w.tp == 1 and hasattr(engine.w, "flat_p"), "serving runs on whole (unsharded) weights"
        super().__init__(engine, block_size, graphs)
        cfg = engine.cfg
        self.num_splits = num_splits
        self.cache = PagedKVCache(cfg.n_layers, num_blocks, block_size, cfg.n_kv_heads, cfg.head_dim, device=engine.device,
                                  dtype=kv_dtype)
        self.kv_bytes_per_token = 2 * cfg.n_layers * cfg.n_kv_heads * cfg.head_dim * self.cache.k[0].element_size()
        # ---- prefix reuse: K / V of finished prompts' whole blocks are kept as snapshots (up to `prefix_cache_bytes`,
        # least recently used first out); a later prompt that starts with the same tokens gets those blocks by a copy
        # and only its remaining tokens are computed.  The reference has the prefix map (src/llm/prefix_cache.cpp) but
        # never consults it while serving.
        self.prefix_cache_bytes = int(prefix_cache_bytes)
        self._snap = OrderedDict()           # handle -> (k [layers, nb, Hkv, bs, hd], v, bytes)
        self._snap_bytes = 0
        self._next_handle = 1
        self._seq_tokens = {}                # first block of a sequence in prefill -> its prompt tokens so far
        if self.prefix_cache_bytes > 0:
            from ..serving import PrefixCache
            self._index = PrefixCache()

    # ------------------------------------------------------------------ shared layer body
    def _layers(self, x, positions, attend):
        e, cfg, w, K = self.e, self.e.cfg, self.e.w, self.e.K
        Hq, Hkv, hd = cfg.n_heads, cfg.n_kv_heads, cfg.head_dim
        n = x.shape[0]
        for i in range(cfg.n_layers):
            p = "layers.%d." % i
            h, _, _, _ = K.norm_fwd(x, w.p(p + "attn_norm"), eps=cfg.rms_eps)
            qkv = K.gemm(h, w.p(p + "wqkv"))
            K.rope_(qkv, e.cos, e.sin, 1, Hq, hd, col_offset=0, positions=positions)
            K.rope_(qkv, e.cos, e.sin, 1, Hkv, hd, col_offset=Hq * hd, positions=positions)
            q = qkv[:, :Hq * hd].view(n, Hq, hd)
            k = qkv[:, Hq * hd:(Hq + Hkv) * hd].view(n, Hkv, hd)
            v = qkv[:, (Hq + Hkv) * hd:].view(n, Hkv, hd)
            o = attend(i, q, k, v)
            x1 = K.gemm(o.reshape(n, Hq * hd), w.p(p + "wo"), residual=x)
            h2, _, _, _ = K.norm_fwd(x1, w.p(p + "mlp_norm"), eps=cfg.rms_eps)
            hm = K.swiglu_fwd(K.gemm(h2, w.p(p + "w_gu")))
            x = K.gemm(hm, w.p(p + "w_down"), residual=x1)
        return x

    def _logits(self, hidden, rows=None):
        e, K = self.e, self.e.K
        hf, _, _, _ = K.norm_fwd(hidden if rows is None else hidden[rows], e.w.p("final_norm"), eps=e.cfg.rms_eps)
        return K.gemm(hf, e.w.p("lm_head"))

    # ------------------------------------------------------------------ prompt chunks
    @torch.no_grad()
    def prefill_chunk(self, tokens: Sequence[int], start: int, block_ids: Sequence[int], want_token: bool, slot: int = 0) -> int:
        """Run prompt positions [start, start + len(tokens)) of one sequence: their K / V go into the sequence's blocks,
        their queries attend to everything cached so far.  Returns the next token when `want_token` (the chunk completes
        the prompt), else -1."""
        if self.prefix_cache_bytes > 0:
            return self._prefill_with_reuse(list(tokens), start, block_ids, want_token)
        return super().prefill_chunk(tokens, start, block_ids, want_token)

    # ---- prefix reuse around the computation
    def _prefill_with_reuse(self, tokens: List[int], start: int, block_ids: Sequence[int], want_token: bool) -> int:
        bs = self.block_size
        key = block_ids[0]
        sofar = (self._seq_tokens.get(key, []) if start > 0 else []) + tokens
        end = start + len(tokens)
        matched, handles = self._index.longest_prefix(sofar, bs)
        snap = self._snap.get(handles[0]) if handles else None
        covered = start
        if snap is not None and matched > start:
            self._snap.move_to_end(handles[0])
            m = min(matched, snap[0].shape[1] * bs)
            if m >= end and want_token:                           # the last token's logits are needed: compute it
                m = (end - 1) // bs * bs
            if m > start:
                b0, b1 = start // bs, m // bs
                dst = torch.tensor(list(block_ids[b0:b1]), dtype=torch.int64, device=self.e.device)
                for i in range(self.e.cfg.n_layers):
                    self.cache.k[i][dst] = snap[0][i, b0:b1]
                    self.cache.v[i][dst] = snap[1][i, b0:b1]
                self.prefill_tokens_reused += m - start
                covered = m
        out = super().prefill_chunk(sofar[covered:end], covered, block_ids, want_token) if covered < end else -1
        if want_token:
            self._seq_tokens.pop(key, None)
            self._remember(sofar, block_ids)
        else:
            self._seq_tokens[key] = sofar
        return out

    def _remember(self, prompt: List[int], block_ids: Sequence[int]) -> None:
        bs = self.block_size
        nb = len(prompt) // bs
        if nb == 0:
            return
        L = nb * bs
        got, handles = self._index.longest_prefix(prompt[:L], bs)
        if got == L and handles and handles[0] in self._snap:
            return                                                # this prefix is cached already
        blocks = torch.tensor(list(block_ids[:nb]), dtype=torch.int64, device=self.e.device)
        k = torch.stack([self.cache.k[i][blocks] for i in range(self.e.cfg.n_layers)])
        v = torch.stack([self.cache.v[i][blocks] for i in range(self.e.cfg.n_layers)])
        nbytes = 2 * k.numel() * k.element_size()
        if nbytes > self.prefix_cache_bytes:
            return
        while self._snap and self._snap_bytes + nbytes > self.prefix_cache_bytes:
            _, (_, _, old) = self._snap.popitem(last=False)
            self._snap_bytes -= old
        h = self._next_handle
        self._next_handle += 1
        self._snap[h] = (k, v, nbytes)
        self._snap_bytes += nbytes
        # findable by prompts that share the whole thing or a power-of-two number of its blocks: a later prompt reuses at
        # least half of the whole blocks it shares, for a logarithmic number of index entries per prompt
        lengths, j = {L}, 1
        while j * bs < L:
            lengths.add(j * bs)
            j *= 2
        from ..serving import _i32
        for n in sorted(lengths):                                 # the native index alone (it evicts by itself)
            self._index._lib.lt_prefix_insert(self._index._c, _i32(prompt[:n]), n, _i32([h]), 1)

    def _prompt_hidden(self, tokens: Sequence[int], start: int, block_ids: Sequence[int], slot: int = 0):
        e, K = self.e, self.e.K
        dev = e.device
        n = len(tokens)
        host = torch.empty(3, n, dtype=torch.int64)
        host[0] = torch.tensor(tokens, dtype=torch.int64)
        host[1] = torch.arange(start, start + n)
        host[2] = self._slots(block_ids, start, n)
        d = host.to(dev, non_blocking=True)
        tok, pos, slots = d[0], d[1].to(torch.int32), d[2].to(torch.int32)
        bs = self.block_size
        nb = (start + n + bs - 1) // bs
        blocks = torch.tensor(list(block_ids[:nb]), dtype=torch.int64, device=dev) if start > 0 else None

        def attend(i, q, k, v):
            self.cache.append(i, k.contiguous(), v.contiguous(), slots)
            if start == 0:
                o, _ = K.flash_fwd(q.unsqueeze(0), k.unsqueeze(0), v.unsqueeze(0), causal=True)
                return o[0]
            # later chunk: keys and values of the whole context so far, read back from the sequence's blocks
            Hkv, hd = k.shape[1], k.shape[2]
            kc = self.cache.k[i][blocks].permute(0, 2, 1, 3).reshape(nb * bs, Hkv, hd)[:start + n]
            vc = self.cache.v[i][blocks].permute(0, 2, 1, 3).reshape(nb * bs, Hkv, hd)[:start + n]
            if self.cache.fp8:
                kc = (kc.float() * self.cache.k_scale).to(q.dtype)
                vc = (vc.float() * self.cache.v_scale).to(q.dtype)
            o, _ = K.flash_fwd(q.unsqueeze(0), kc.contiguous().unsqueeze(0), vc.contiguous().unsqueeze(0), causal=True)
            return o[0]

        return self._layers(K.embedding_fwd(tok, e.w.p("embed")), pos, attend)

    # ------------------------------------------------------------------ one token for every running sequence
    def _decode_hidden(self, d: torch.Tensor, S: int, width: int) -> torch.Tensor:
        from ..serving import paged_attention
        e, K = self.e, self.e.K
        bs = self.block_size
        tok = d[0]
        pos, slots, ctx = d[1].to(torch.int32), d[2].to(torch.int32), d[3].to(torch.int32)
        bt = d[5:].t().contiguous().to(torch.int32)
        splits = self.num_splits or self._splits_for(S * e.cfg.n_kv_heads, width * bs)

        def attend(i, q, k, v):
            self.cache.append(i, k.contiguous(), v.contiguous(), slots)
            return paged_attention(q.contiguous(), self.cache.k[i], self.cache.v[i], bt, ctx, bs, num_splits=splits,
                                   k_scale=self.cache.k_scale, v_scale=self.cache.v_scale)

        return self._layers(K.embedding_fwd(tok, e.w.p("embed")), pos, attend)
