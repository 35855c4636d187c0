"""What every paged engine shares: the page pool, batch assembly, the step function, graph-replayed decode and generation.

``PagedEngine`` owns no weights and no kernels of a model.  A subclass loads its weights, allocates its caches and
activations, and provides ``_embed``, ``_run_layers`` and ``_head``; batching, page bookkeeping, recurrent-state slots, CUDA
graphs and the public operations (``begin`` / ``forward_tokens`` / ``decode`` / ``decode_steps`` / ``truncate`` / ``end``) live here, so
that every model family is scheduled and served the same way.
"""
from __future__ import annotations

import contextlib
import ctypes
import os

import torch

from .. import _native
from ..ops import cuda_ops as ops
from ..utils.nvtx import nvtx_method

PAGE = 16


class KVPool:
    """Host-side page bookkeeping (C++), shared by every layer's device cache."""

    def __init__(self, n_pages: int, page_size: int = PAGE, state_slots: int = 0):
        """``state_slots``: recurrent-state slots (0: the model has no recurrent layers).  A sequence of such a pool holds one from
        ``begin`` to ``end``, and no pages are shared between sequences."""
        L = _native.host()
        if not getattr(L, "_b200_kv_ready", False):
            vp, i64, i32, u64 = ctypes.c_void_p, ctypes.c_int64, ctypes.c_int32, ctypes.c_uint64
            P32 = ctypes.POINTER(ctypes.c_int32)
            sig = {"b200_kv_create": ([i32, i32], vp), "b200_kv_destroy": ([vp], None),
                   "b200_kv_free_pages": ([vp], i32), "b200_kv_total_pages": ([vp], i32), "b200_kv_retained_pages": ([vp], i32), "b200_kv_set_retention": ([vp, i32], None),
                   "b200_kv_prefix_hits": ([vp], u64), "b200_kv_prefix_lookups": ([vp], u64),
                   "b200_kv_seq_begin": ([vp, i64, P32, i64], i64), "b200_kv_seq_extend": ([vp, i64, i64], i32),
                   "b200_kv_seq_publish": ([vp, i64, P32, i64], None), "b200_kv_seq_len": ([vp, i64], i64),
                   "b200_kv_seq_n_pages": ([vp, i64], i32), "b200_kv_seq_pages": ([vp, i64, P32, i32], i32),
                   "b200_kv_seq_truncate": ([vp, i64, i64, P32, P32], i32), "b200_kv_seq_end": ([vp, i64], None),
                   "b200_kv_stage_decode": ([vp, vp, i32, i32, i32, vp, vp, vp, vp, vp], i32),
                   "b200_kv_set_slots": ([vp, i32], i32), "b200_kv_free_slots": ([vp], i32), "b200_kv_seq_slots": ([vp, vp, i32, vp], i32)}
            for n, (a, r) in sig.items():
                f = getattr(L, n)
                f.argtypes, f.restype = a, r
            L._b200_kv_ready = True
        self.L = L
        self.h = L.b200_kv_create(n_pages, page_size)
        self.page_size = page_size
        self.n_pages = n_pages
        self.state_slots = state_slots
        if state_slots and L.b200_kv_set_slots(self.h, state_slots) != 0:
            raise ValueError("bad number of state slots")
        # B200_KV_RETAIN=0: published pages leave the prefix index with their last holder, so that a repeated prompt takes the
        # very same compute path as the first time (bit-exact repeats); the default keeps them until the memory is needed
        if os.environ.get("B200_KV_RETAIN", "1") == "0":
            self.set_retention(False)

    def set_retention(self, on: bool):
        self.L.b200_kv_set_retention(self.h, int(bool(on)))

    @staticmethod
    def _arr(tokens):
        if tokens is None:
            return None, 0
        a = (ctypes.c_int32 * len(tokens))(*tokens)
        return a, len(tokens)

    def begin(self, seq_id: int, tokens=None) -> int:
        a, n = self._arr(tokens)
        r = self.L.b200_kv_seq_begin(self.h, seq_id, a, n)
        if r == -2:
            raise MemoryError("no free sequence state slot")
        if r < 0:
            raise KeyError(f"sequence {seq_id} already exists")
        return r

    @property
    def free_slots(self) -> int:
        return self.L.b200_kv_free_slots(self.h)

    def slots(self, seq_ids) -> list[int]:
        """Recurrent-state slots of the sequences (-1 in a pool without slots)."""
        n = len(seq_ids)
        ids, out = (ctypes.c_int64 * n)(*seq_ids), (ctypes.c_int32 * n)()
        if self.L.b200_kv_seq_slots(self.h, ids, n, out) != 0:
            raise KeyError("unknown sequence")
        return list(out)

    def extend(self, seq_id: int, n_new: int):
        r = self.L.b200_kv_seq_extend(self.h, seq_id, n_new)
        if r == -1:
            raise KeyError(f"unknown sequence {seq_id}")
        if r == -2:
            raise MemoryError("KV cache is out of pages")

    def publish(self, seq_id: int, tokens):
        a, n = self._arr(tokens)
        self.L.b200_kv_seq_publish(self.h, seq_id, a, n)

    def length(self, seq_id: int) -> int:
        return self.L.b200_kv_seq_len(self.h, seq_id)

    def n_pages_of(self, seq_id: int) -> int:
        return self.L.b200_kv_seq_n_pages(self.h, seq_id)

    def pages(self, seq_id: int) -> list[int]:
        n = self.L.b200_kv_seq_n_pages(self.h, seq_id)
        if n < 0:
            raise KeyError(f"unknown sequence {seq_id}")
        buf = (ctypes.c_int32 * max(n, 1))()
        self.L.b200_kv_seq_pages(self.h, seq_id, buf, n)
        return list(buf[:n])

    def stage_decode(self, seq_ids_ptr: int, B: int, max_pages: int, full_table: bool, pos_ptr: int, slot_ptr: int, ctx_ptr: int,
                     table_ptr: int) -> bool:
        """Grow ``B`` sequences by one token and fill the staging arrays (raw host pointers); returns
        whether any page-table row was rewritten."""
        dirty = ctypes.c_int32(0)
        r = self.L.b200_kv_stage_decode(self.h, seq_ids_ptr, B, max_pages, int(full_table), pos_ptr, slot_ptr, ctx_ptr, table_ptr,
                                        ctypes.addressof(dirty))
        if r == -1:
            raise KeyError("unknown sequence in the decode batch")
        if r == -2:
            raise MemoryError("KV cache is out of pages")
        if r == -3:
            raise ValueError("sequence exceeds the engine's max context")
        return bool(dirty.value)

    def truncate(self, seq_id: int, new_len: int):
        """Drop the tokens from ``new_len`` on.  Returns ``None``, or ``(src_page, dst_page)`` when the partly kept page
        was shared with another sequence and this one was given a page of its own: the caller must copy that page's
        K/V before writing to it."""
        src, dst = ctypes.c_int32(-1), ctypes.c_int32(-1)
        r = self.L.b200_kv_seq_truncate(self.h, seq_id, new_len, ctypes.byref(src), ctypes.byref(dst))
        if r == -2:
            raise MemoryError("KV cache is out of pages")
        if r < 0:
            raise ValueError("bad truncate")
        return (src.value, dst.value) if r == 1 else None

    def end(self, seq_id: int):
        self.L.b200_kv_seq_end(self.h, seq_id)

    @property
    def free_pages(self) -> int:
        return self.L.b200_kv_free_pages(self.h)

    @property
    def retained_pages(self) -> int:
        """Published pages no sequence holds any more: still in the prefix index, reclaimed (oldest first) when pages run short.
        They are counted in ``free_pages``."""
        return self.L.b200_kv_retained_pages(self.h)

    @property
    def prefix_stats(self) -> tuple[int, int]:
        return self.L.b200_kv_prefix_hits(self.h), self.L.b200_kv_prefix_lookups(self.h)

    def __del__(self):
        try:
            self.L.b200_kv_destroy(self.h)
        except Exception:
            pass

class PagedEngine:
    """Subclass contract: ``__init__`` calls ``_init_paged`` first, allocates with ``_ws`` / ``_alloc_batch`` and ends with the hooks
    ``_embed(T)``, ``_run_layers(T, decode, n_seqs, max_q, pages) -> launches`` and ``_head(rows, nb, greedy) -> launches`` ready.
    ``rows`` of ``_head`` is ``self.x[:nb]`` itself when every row of the step is wanted."""

    def _init_paged(self, device, max_batch: int, max_ctx: int, n_pages: int | None, max_tokens: int, canaries: bool | None,
                    state_slots: int = 0):
        self.device = torch.device(device)
        self.canaries = (os.environ.get("B200_CANARY", "0") == "1") if canaries is None else bool(canaries)
        self._guards: dict[str, tuple[torch.Tensor, int]] = {}
        self.max_batch, self.max_tokens = max_batch, max_tokens
        self.max_pages = (max_ctx + PAGE - 1) // PAGE
        self.n_pages = n_pages if n_pages is not None else max_batch * self.max_pages + 1
        self.pool = KVPool(self.n_pages, state_slots=state_slots)
        self.state_slots = state_slots
        self.status = torch.zeros(1, dtype=torch.int32, device=self.device)
        self._graphs: dict[int, tuple] = {}
        self.launches_per_decode = 0
        self.max_splits = 64
        self.attn_target_ctas = int(os.environ.get("B200_ATTN_CTAS", 0))   # split-K decode attention: CTAs to aim for (0: built-in rule)
        self.h2d_bytes = 0                              # host-to-device bytes copied by decode() so far

    def _alloc_batch(self):
        """Per-step metadata on the device."""
        T, i32 = self.max_tokens, torch.int32
        ws = self._ws
        self.ids = ws("ids", (T,), i32, zero=True)
        self.pos = ws("pos", (T,), i32, zero=True)
        self.slot = ws("slot", (T,), i32, zero=True)
        self.page_table = ws("page_table", (self.max_batch, self.max_pages), i32, zero=True)
        self.seq_lens = ws("seq_lens", (self.max_batch,), i32, zero=True)
        self.q_start = ws("q_start", (self.max_batch,), i32, zero=True)
        self.q_len = ws("q_len", (self.max_batch,), i32, zero=True)
        self.out_ids = ws("out_ids", (self.max_batch,), i32, zero=True)
        self.out_val = ws("out_val", (self.max_batch,), torch.float32, zero=True)
        if self.state_slots:
            self.state_slot = ws("state_slot", (self.max_batch,), i32, zero=True)

    # ------------------------------------------------------------------ workspaces
    _GUARD_BYTES, _GUARD_FILL = 256, 0xA5

    def _ws(self, name: str, shape, dtype, zero: bool = False) -> torch.Tensor:
        """One workspace tensor.  With canaries on (``B200_CANARY=1`` or ``canaries=True``) it sits between two 256-byte
        guard zones of a known byte, and ``check_canaries`` tells which guards a kernel has written into: the
        substitute for a memory checker on the engine's own buffers."""
        n = 1
        for v in shape:
            n *= int(v)
        if not self.canaries:
            return (torch.zeros if zero else torch.empty)(tuple(shape), dtype=dtype, device=self.device)
        G = self._GUARD_BYTES
        nbytes = n * torch.empty((), dtype=dtype).element_size()
        body_bytes = (nbytes + G - 1) // G * G
        raw = torch.full((G + body_bytes + G,), self._GUARD_FILL, dtype=torch.uint8, device=self.device)
        body = raw[G: G + nbytes].view(dtype).view(*shape)
        if zero:
            body.zero_()
        self._guards[name] = (raw, nbytes)
        return body

    def check_canaries(self) -> list[str]:
        """Names of the workspaces whose guard zones no longer hold the fill byte (empty list: all intact, or canaries
        off).  ``name:before`` / ``name:after`` says on which side the stray write landed."""
        bad = []
        G = self._GUARD_BYTES
        torch.cuda.synchronize(self.device) if self.device.type == "cuda" else None
        for name, (raw, nbytes) in self._guards.items():
            if not bool((raw[:G] == self._GUARD_FILL).all()):
                bad.append(name + ":before")
            if not bool((raw[G + nbytes:] == self._GUARD_FILL).all()):
                bad.append(name + ":after")
        return bad

    def _attn_splits(self, B: int, kv_heads: int, ctx_pages: int) -> int:
        """Split-K factor of decode attention.  Measured on the 8B shape: a CTA should keep at least ~24
        pages (the merge of the partial results and each CTA's set-up are a fixed cost), small batches
        want just enough CTAs to cover the SMs once, and large batches run best at ~2000 CTAs (several
        waves even out the tail)."""
        if self.attn_target_ctas:                      # explicit override (benchmark sweeps)
            want = max(1, (self.attn_target_ctas + B * kv_heads - 1) // (B * kv_heads))
        else:
            rows = B * kv_heads
            fill = (148 + rows - 1) // rows
            big = (2048 + rows - 1) // rows if rows >= 148 else 0
            want = min(max(1, ctx_pages // 24), max(fill, big))
        return max(1, min(self.max_splits, want, ctx_pages))

    # ------------------------------------------------------------------ host-side batch assembly
    def _stage_batch(self, seq_ids, new_tokens: list[list[int]]):
        """Extend the sequences' page lists and build ids/pos/slot/page-table for the new tokens."""
        ids, pos, slot, q_start, q_len, ctx = [], [], [], [], [], []
        table = torch.zeros((len(seq_ids), self.max_pages), dtype=torch.int32)
        # Check the whole batch before any sequence grows: a refused batch must leave the page lists as they were.
        if len(seq_ids) > self.max_batch or sum(len(t) for t in new_tokens) > self.max_tokens:
            raise ValueError("batch exceeds the engine's workspace")
        need = 0
        for sid, toks in zip(seq_ids, new_tokens):
            p0 = self.pool.length(sid)
            if p0 < 0:
                raise KeyError(f"unknown sequence {sid}")
            after = (p0 + len(toks) + PAGE - 1) // PAGE
            if after > self.max_pages:
                raise ValueError("sequence exceeds the engine's max context")
            need += max(0, after - self.pool.n_pages_of(sid))
        if need > self.pool.free_pages:
            raise MemoryError("KV cache is out of pages")
        for b, (sid, toks) in enumerate(zip(seq_ids, new_tokens)):
            p0 = self.pool.length(sid)
            self.pool.extend(sid, len(toks))
            pages = self.pool.pages(sid)
            table[b, : len(pages)] = torch.tensor(pages, dtype=torch.int32)
            q_start.append(len(ids))
            q_len.append(len(toks))
            ctx.append(p0 + len(toks))
            for i, t in enumerate(toks):
                p = p0 + i
                ids.append(t)
                pos.append(p)
                slot.append(pages[p // PAGE] * PAGE + p % PAGE)
        return ids, pos, slot, q_start, q_len, ctx, table

    def _upload(self, ids, pos, slot, q_start, q_len, ctx, table):
        T, B = len(ids), len(ctx)
        if getattr(self, "_stg", None) is not None:
            self._stg["last_batch"] = None        # the decode fast path must resend its page-table rows
        pin = lambda v: torch.tensor(v, dtype=torch.int32).pin_memory()
        self.ids[:T].copy_(pin(ids), non_blocking=True)
        self.pos[:T].copy_(pin(pos), non_blocking=True)
        self.slot[:T].copy_(pin(slot), non_blocking=True)
        self.q_start[:B].copy_(pin(q_start), non_blocking=True)
        self.q_len[:B].copy_(pin(q_len), non_blocking=True)
        self.seq_lens[:B].copy_(pin(ctx), non_blocking=True)
        self.page_table[:B].copy_(table.pin_memory(), non_blocking=True)

    def _upload_slots(self, seq_ids):
        if self.state_slots:
            self.state_slot[: len(seq_ids)].copy_(torch.tensor(self.pool.slots(seq_ids), dtype=torch.int32).pin_memory(), non_blocking=True)

    @contextlib.contextmanager
    def _state_held(self):
        """A step run inside leaves every sequence's recurrent state alone (slot -1: start from zero, keep nothing): the warm-up run
        ahead of a graph capture."""
        if not self.state_slots:
            yield
            return
        saved = self.state_slot.clone()
        self.state_slot.fill_(-1)
        torch.cuda.synchronize()
        try:
            yield
        finally:
            torch.cuda.synchronize()
            self.state_slot.copy_(saved)

    def _batch_order(self, q_len: list[int]) -> list[int] | None:
        """The order a step's entries are laid out in (None: as given), for models whose kernels want some of them next to one another."""
        return None

    def _plan_batch(self, q_len: list[int], ctx: list[int]):
        """Called ahead of every step that is not a decode step, with the new tokens and the context of each entry as laid out."""

    # ------------------------------------------------------------------ public operations
    def _caches(self):
        """Every per-page tensor of the model (first axis: page)."""
        return [*self.kc, *self.vc]

    def begin(self, seq_id: int, prompt=None) -> int:
        """Open a sequence; returns how many prompt tokens are already cached (prefix reuse)."""
        return self.pool.begin(seq_id, list(prompt) if prompt is not None else None)

    def end(self, seq_id: int):
        self.pool.end(seq_id)

    def truncate(self, seq_id: int, new_len: int):
        """Drop the sequence's tokens from position ``new_len`` on (a cancelled turn, a rejected speculative tail).
        If the page that stays partly filled was shared through the prefix cache, the sequence gets a private copy of
        it, so writing the next tokens cannot touch another sequence's K/V.  A recurrent state cannot be rolled back: a model
        that has one only takes its current length, or 0 (start over)."""
        if self.state_slots and new_len not in (0, self.pool.length(seq_id)):
            raise ValueError("a sequence with recurrent state cannot be cut at an earlier token")
        cow = self.pool.truncate(seq_id, new_len)
        if cow is not None:
            src, dst = cow
            for c in self._caches():
                c[dst].copy_(c[src])
        if getattr(self, "_stg", None) is not None:
            self._stg["last_batch"] = None        # page lists changed: the decode fast path must resend its rows

    @torch.no_grad()
    @nvtx_method("engine.prefill")
    def forward_tokens(self, seq_ids: list[int], new_tokens: list[list[int]], greedy: bool = True, all_positions: bool = False,
                       positions: list[list[int]] | None = None):
        """Append ``new_tokens[b]`` to sequence ``seq_ids[b]`` and return the logits of each
        sequence's last new token ([B, V] view, valid until the next call) and their arg-max.  ``all_positions``: the
        logits and arg-max of EVERY new token instead ([T, V], in feeding order): what verifying a speculated
        continuation needs; T is then limited by the logits workspace (``max_batch`` rows).  ``positions[b]``: the places among
        sequence b's new tokens whose logits are wanted, in any number (the result is then a tensor of its own, in that order)."""
        B = len(seq_ids)
        order = self._batch_order([len(t) for t in new_tokens])
        if order is not None:
            seq_ids, new_tokens = [seq_ids[i] for i in order], [new_tokens[i] for i in order]
        staged = self._stage_batch(seq_ids, new_tokens)
        ids, pos, slot, q_start, q_len, ctx, table = staged
        T = len(ids)
        if T > self.max_tokens or B > self.max_batch or (all_positions and T > self.max_batch):
            raise ValueError("batch exceeds the engine's workspace")
        self._upload(*staged)
        self._upload_slots(seq_ids)
        self._embed(T)
        decode = all(n == 1 for n in q_len)
        pages = max((c + PAGE - 1) // PAGE for c in ctx)
        if not decode or positions is not None:
            self._plan_batch(q_len, ctx)
        self._run_layers(T, decode and positions is None, B, max(q_len), pages)
        if order is not None:                         # from here on in the caller's order again
            back = sorted(range(B), key=order.__getitem__)
            q_start, q_len = [q_start[i] for i in back], [q_len[i] for i in back]
            if all_positions:
                positions = [range(n) for n in q_len]
        if positions is not None:
            at = [s + i for s, want in zip(q_start, positions) for i in want]
            parts = []
            for lo in range(0, len(at), self.max_batch):
                rows = self.x[:T].index_select(0, torch.tensor(at[lo: lo + self.max_batch], device=self.device)).contiguous()
                self._head(rows, rows.shape[0], greedy)
                parts.append((self.logits[: rows.shape[0]].clone(), self.out_ids[: rows.shape[0]].clone()))
            if not parts:
                return self.logits[:0], self.out_ids[:0]
            return torch.cat([p[0] for p in parts]), torch.cat([p[1] for p in parts])
        if all_positions:
            self._head(self.x[:T], T, greedy)
            return self.logits[:T], self.out_ids[:T]
        if decode:
            rows = self.x[:B]
        else:
            last = torch.tensor([s + n - 1 for s, n in zip(q_start, q_len)], device=self.device)
            rows = self.x[:T].index_select(0, last).contiguous()
        self._head(rows, B, greedy)
        return self.logits[:B], self.out_ids[:B]

    # ---- graph-replayed decode
    def _capture(self, B: int, pages: int, advance: bool = False):
        g = torch.cuda.CUDAGraph()
        s = torch.cuda.Stream(device=self.device)
        s.wait_stream(torch.cuda.current_stream())

        def body():
            self._embed(B)
            n = 1 + self._run_layers(B, True, B, 1, pages)
            n += self._head(self.x[:B], B, True)
            if advance:
                ops.decode_advance(self.ids, self.out_ids, self.pos, self.slot, self.seq_lens, self.page_table, PAGE, B,
                                   self._hist, self._step, self._hist.numel() // B)
                n += 1
            return n

        if advance:   # the warm-up run must not move the real state: save and restore it
            saved = [t.clone() for t in (self.ids, self.pos, self.slot, self.seq_lens, self._step)]
        with self._state_held(), torch.cuda.stream(s):
            body()  # warm-up outside capture: sets kernel attributes, allocates the scratch
        if advance:
            torch.cuda.synchronize()
            for t, v in zip((self.ids, self.pos, self.slot, self.seq_lens, self._step), saved):
                t.copy_(v)
        torch.cuda.current_stream().wait_stream(s)
        torch.cuda.synchronize()
        with torch.cuda.graph(g, stream=s):
            n = body()
        return g, n

    def _decode_staging(self):
        """Pinned host staging for decode steps, allocated once: per-step metadata goes from the page
        allocator (one native call for the whole batch) into these arrays and from there to the device
        in four small asynchronous copies; the page table moves only when a sequence took a new page
        or the batch changed."""
        if getattr(self, "_stg", None) is None:
            B, P = self.max_batch, self.max_pages
            pin = lambda *shape, dt=torch.int32: torch.zeros(shape, dtype=dt).pin_memory() if torch.cuda.is_available() else torch.zeros(shape, dtype=dt)
            self._stg = {"seq": pin(B, dt=torch.int64), "ids": pin(B), "pos": pin(B), "slot": pin(B), "ctx": pin(B), "table": pin(B, P),
                         "out": pin(B), "last_batch": None, "copied": torch.cuda.Event() if torch.cuda.is_available() else None}
        return self._stg

    @torch.no_grad()
    @nvtx_method("engine.decode_step")
    def decode(self, seq_ids: list[int], tokens: list[int], use_graph: bool = True):
        """One decode step: append one token per sequence, return (logits view, arg-max ids)."""
        if not use_graph:
            return self.forward_tokens(seq_ids, [[t] for t in tokens])
        B = len(seq_ids)
        if B > self.max_batch:
            raise ValueError("batch exceeds the engine's workspace")
        st = self._decode_staging()
        if st["copied"] is not None:              # the arrays are rewritten only once the previous step's copies have left them
            st["copied"].synchronize()
        batch = tuple(seq_ids)
        same = st["last_batch"] == batch
        if not same:
            st["seq"][:B] = torch.tensor(seq_ids, dtype=torch.int64)
        st["ids"][:B] = torch.tensor(tokens, dtype=torch.int32)
        dirty = self.pool.stage_decode(st["seq"].data_ptr(), B, self.max_pages, not same, st["pos"].data_ptr(), st["slot"].data_ptr(),
                                       st["ctx"].data_ptr(), st["table"].data_ptr())
        st["last_batch"] = batch
        pages = (int(st["ctx"][:B].max()) + PAGE - 1) // PAGE
        # Split count is baked into the captured launch; bucket the context length so a graph is
        # reused while the sequence grows.
        bucket = 1 << max(0, (pages - 1)).bit_length()
        key = (B, bucket)

        def upload():
            self.ids[:B].copy_(st["ids"][:B], non_blocking=True)
            self.pos[:B].copy_(st["pos"][:B], non_blocking=True)
            self.slot[:B].copy_(st["slot"][:B], non_blocking=True)
            self.seq_lens[:B].copy_(st["ctx"][:B], non_blocking=True)
            self.h2d_bytes += 16 * B
            if not same:
                self._upload_slots(seq_ids)
            if dirty or not same:     # otherwise the device rows are still those of the previous step
                self.page_table[:B].copy_(st["table"][:B], non_blocking=True)
                self.h2d_bytes += 4 * B * self.max_pages

        if key not in self._graphs:
            upload()
            self._graphs[key] = self._capture(B, bucket)
        upload()
        if st["copied"] is not None:
            st["copied"].record()
        g, n = self._graphs[key]
        g.replay()
        self.launches_per_decode = n
        return self.logits[:B], self.out_ids[:B]

    @torch.no_grad()
    @nvtx_method("engine.decode_steps")
    def decode_steps(self, seq_ids: list[int], tokens: list[int], n_steps: int, on_replay=None):
        """``n_steps`` greedy decode steps with the autoregression kept on the device: one upload,
        ``n_steps`` graph replays (each ends by turning its arg-max into the next step's input),
        one read-back.  Returns the generated ids as an int32 tensor [n_steps, B] (on the device).
        ``on_replay(i)`` is called before replay ``i`` (benchmarks place their events there)."""
        B = len(seq_ids)
        staged = self._stage_batch(seq_ids, [[t] for t in tokens])
        ctx = staged[5]
        table = staged[6]
        for b, sid in enumerate(seq_ids):        # pages for every later step up front
            if (self.pool.length(sid) + n_steps - 1 + PAGE - 1) // PAGE > self.max_pages:
                raise ValueError("sequence exceeds the engine's max context")
            self.pool.extend(sid, n_steps - 1)
            pages = self.pool.pages(sid)
            if len(pages) > self.max_pages:
                raise ValueError("sequence exceeds the engine's max context")
            table[b, : len(pages)] = torch.tensor(pages, dtype=torch.int32)
        pages = max((c + n_steps + PAGE - 1) // PAGE for c in ctx)
        bucket = 1 << max(0, (pages - 1)).bit_length()
        key = ("loop", B, bucket)
        if getattr(self, "_hist", None) is None or self._hist.numel() < n_steps * B:
            self._hist = torch.zeros(max(n_steps * B, 4096), dtype=torch.int32, device=self.device)
            self._step = torch.zeros(1, dtype=torch.int32, device=self.device)
            self._graphs = {k: v for k, v in self._graphs.items() if not (isinstance(k, tuple) and k[0] == "loop")}
        self._upload_slots(seq_ids)
        if key not in self._graphs:
            self._upload(*staged)
            self._graphs[key] = self._capture(B, bucket, advance=True)
        self._upload(*staged)
        self._step.zero_()
        g, n = self._graphs[key]
        for i in range(n_steps):
            if on_replay is not None:
                on_replay(i)
            g.replay()
        self.launches_per_decode = n
        return self._hist[: n_steps * B].view(n_steps, B)

    def check_status(self):
        s = int(self.status.item())
        if s:
            raise RuntimeError(f"a kernel wait timed out (status {s})")

    @torch.no_grad()
    def generate(self, prompt: list[int], n_new: int, seq_id: int = 0, use_graph: bool = True):
        """Greedy generation for one sequence.  Returns (ids, per-step logits [n_new, V] on CPU)."""
        cached = self.begin(seq_id, prompt)
        logits, nxt = self.forward_tokens([seq_id], [list(prompt[cached:])])
        out, all_logits = [], []
        for _ in range(n_new):
            all_logits.append(logits[0].float().cpu().clone())
            tok = int(nxt[0].item())
            out.append(tok)
            logits, nxt = self.decode([seq_id], [tok], use_graph=use_graph)
        self.pool.publish(seq_id, list(prompt) + out)
        return out, torch.stack(all_logits)
