"""Chunk path of layer-stack models: R prompt rows go through every layer in one pass over the step's own caches.

    rows (stream update + norms)
    token mixer        one class per mechanism in ``prefill/stack_mixers.py``
    feed-forward       two-product GLU -> down, or squared ReLU -> down; routed experts: scores -> choice -> rows sorted by
                       expert -> grouped products -> weighted sum inside the next row kernel

A chunk may start and end anywhere and has any length up to ``chunk`` rows; the caches and states it leaves are those
the step continues from.
"""
from __future__ import annotations

from contextlib import contextmanager
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from ..ops import kernels as K
from ..ops import stack_kernels as S
from ..runtime.packing import Packed, pad
from ..runtime.stack import StackRuntime
from .stack_mixers import MIXERS

SMS = 148


class StackPrefill:
    quantum = 1

    def __init__(self, runtime: StackRuntime, chunk: int = 2048, kv_block: int = 16384):
        self.t, self.spec, self.C, self.dev = runtime, runtime.spec, chunk, runtime.dev
        self.f32, self.act = runtime.f32, runtime.act
        self.kv_block = pad(min(kv_block, runtime.capacity), 64)
        s, dev, C = self.spec, self.dev, chunk
        f32, i32 = torch.float32, torch.int32
        L = runtime.layers
        ffs = [d["spec"].mlp for d in L if d["spec"].mlp is not None]
        moe = [f for f in ffs if f.kind == "moe"]
        self.h_ld = pad(s.hidden, 8)

        def z(n: int, t=f32) -> torch.Tensor:
            return torch.zeros(max(8, n), dtype=t, device=dev)

        def most(it) -> int:
            return max(list(it), default=0)

        self.pos = torch.zeros(1, dtype=i32, device=dev)
        self.tokens = torch.zeros(C, dtype=i32, device=dev)
        self.x = torch.zeros(C, s.hidden, dtype=f32, device=dev)
        self.h = torch.zeros(C, self.h_ld, dtype=self.act, device=dev)
        self.y = torch.zeros(C, s.hidden, dtype=f32, device=dev)
        self.y2 = torch.zeros(C, s.hidden, dtype=f32, device=dev) if any(d["kind"] == "parallel" for d in L) else None
        # buffers of the mixers, one per role, shared by the layers (sizes differ from layer to layer)
        sizes: Dict[tuple, int] = {}
        for d in L:
            for name, (n, t) in MIXERS[d["kind"]].scratch(self, d["spec"].mixer, d).items():
                sizes[name, t] = max(n, sizes.get((name, t), 0))
        self.buf = {name: z(n, t) for (name, t), n in sizes.items()}
        self.ff = z(C * most(pad(f.ff, 8) for f in ffs if f.kind != "moe"), self.act)
        if moe:
            E, T = most(f.routing.expert_count for f in moe), most(f.routing.top_k for f in moe)
            self.scores, self.ids, self.probs = z(C * E), z(C * T, i32), z(C * T)
            self.slot_of, self.n_items, self.seg_rows = z(C * T, i32), z(1, i32), z(E, i32)
            self.max_items = -(-C * T // 64) + E
            self.item_z, self.item_row = z(self.max_items, i32), z(self.max_items, i32)
            self.cap = most(self._segment_rows(C, f.routing) for f in moe)
            self.sorted = z(self.cap * self.h_ld, self.act)
            self.ea = z(self.cap * most(pad(f.ff, 8) for f in moe), self.act)
            self.ey = z(self.cap * s.hidden)
        self.head_rows = 256
        self.hw = torch.zeros(self.head_rows, self.h_ld, dtype=self.act, device=dev)
        self.tensor_cores = not self.f32              # attention of chunk rows on tcgen05 (else the plain kernel)
        self.maps: Dict[tuple, object] = {}
        self.phases: dict = {}
        self.profile = False                          # per-stage CUDA-event timing (adds an event pair per stage)
        self._timed: Dict[str, list] = {}

    @contextmanager
    def stage(self, name: str):
        if not self.profile:
            yield
            return
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        yield
        b.record()
        self._timed.setdefault(name, []).append((a, b))

    def stage_ms(self) -> Dict[str, Tuple[float, int]]:
        """(device milliseconds, calls) per stage since the last call (``profile`` must be on); waits for the stream."""
        torch.cuda.current_stream().synchronize()
        out = {k: (sum(a.elapsed_time(b) for a, b in v), len(v)) for k, v in self._timed.items()}
        self._timed = {}
        return out

    @staticmethod
    def _item_rows(rows: int, routing, f32: bool = False) -> int:
        """Rows of a segment of the expert list: 128 where the experts are well filled."""
        return 128 if not f32 and rows * routing.top_k >= 96 * routing.expert_count else 64

    def _items(self, rows: int, routing, item_rows: int) -> int:
        """Most segments the choices of ``rows`` tokens can need."""
        pairs = rows * routing.top_k
        return pairs // item_rows + min(pairs, routing.expert_count)

    def _segment_rows(self, rows: int, routing) -> int:
        """Rows the sorted buffers need for chunks of at most ``rows`` tokens."""
        return max(self._items(rows, routing, i) * i for i in (64, 128))

    # ------------------------------------------------------------------ products
    def _wmap(self, p: Packed) -> K.TensorMap:
        key = ("w", p.w.data_ptr(), p.z, p.n)
        if key not in self.maps:
            self.maps[key] = S.weight_map(p.w, p.k)
        return self.maps[key]

    def _xmap(self, t: torch.Tensor, k: int, zcount: int, zstride: int, rows: int, ld: int, box: int, offset: int) -> K.TensorMap:
        key = ("x", t.data_ptr(), k, zcount, zstride, rows, ld, box, offset)
        if key not in self.maps:
            self.maps[key] = S.token_map(t, k, zcount, zstride, rows, ld, box, offset)
        return self.maps[key]

    def gemm(self, epi: int, w: Packed, x: torch.Tensor, x_ld: int, rows: int, out: torch.Tensor, out_ld: int, *, w2: Optional[Packed] = None,
              z: int = 1, x_z: int = 0, out_z: int = 0, x_off: int = 0, x_rows: Optional[int] = None, items: Optional[tuple] = None,
              bias: Optional[torch.Tensor] = None, rate: Optional[torch.Tensor] = None, act_cols: int = 0, scale: float = 1.0, limit: float = 0.0, alpha: float = 0.0) -> None:
        """out[row, z, :] = epilogue(W_z x[row, z, :]) for every token row; ``items`` = (segment rows, most segments)."""
        a = S.StackGemmArgs()
        a.n, a.k, a.rows, a.zcount = w.n, w.k, rows, z
        a.out, a.out_ld, a.out_zstride, a.out_f32 = out.data_ptr(), out_ld, out_z, int(out.dtype == torch.float32)
        a.bias = None if bias is None else bias.data_ptr()
        a.rate = None if rate is None else rate.data_ptr()
        a.act_cols, a.scale, a.limit, a.alpha, a.status = act_cols, scale, limit, alpha, self.t.fab.status.data_ptr()
        if items is not None:
            a.n_items, a.item_z, a.item_row = self.n_items.data_ptr(), self.item_z.data_ptr(), self.item_row.data_ptr()
            a.item_rows, a.max_items = items
        if self.f32:
            a.act, a.act_ld, a.act_zstride = x.data_ptr() + 4 * x_off, x_ld, x_z
            a.w, a.w2 = w.w.data_ptr(), None if w2 is None else w2.w.data_ptr()
            a.w_ld, a.w_zstride = w.ld, w.n * w.ld
            S.gemm_f32(epi, a)
            return
        dual = w2 is not None
        if items is not None:
            ntok = items[0]
        else:
            tiles = -(-w.n // 128) * z
            sizes = (128, 64) if dual else (256, 128, 64) if epi in (S.EPI_STORE, S.EPI_RELU2) else (256, 64)
            ntok = next((t for t in sizes if tiles * -(-rows // t) >= SMS - 20), 64)
        live = x_rows if x_rows is not None else x.numel() // x_ld
        xm = self._xmap(x, w.k, z, x_z, live, x_ld, ntok, x_off)
        wbytes = w.nbytes * (2 if dual else 1)
        S.gemm(epi, ntok, self._wmap(w), self._wmap(w2) if dual else None, xm, a, items is None and wbytes > (96 << 20))

    # ------------------------------------------------------------------ one chunk
    def _rows(self, R: int, *, embed: bool = False, y: Optional[torch.Tensor] = None, post=None, y2: Optional[torch.Tensor] = None, join=None,
              moe=None, add=None, pre=None, copy: bool = False) -> None:
        """Stream update; then the input rows ``h`` of the next sublayer: normed by ``pre``, or the stream itself (``copy``)."""
        s, a = self.spec, S.StackRowArgs()
        if embed:
            a.tokens, a.table, a.vocab, a.embed_scale = self.tokens.data_ptr(), self.t.embed.data_ptr(), s.vocab, s.embed_scale
        if y is not None:
            a.y, a.y_ld, a.post_w = y.data_ptr(), s.hidden, post.data_ptr()
            if join is not None:
                a.y2, a.join_w, a.join_w2 = y2.data_ptr(), join[0].data_ptr(), join[1].data_ptr()
            if moe is not None:
                a.slot_of, a.probs, a.top_k = self.slot_of.data_ptr(), self.probs.data_ptr(), moe.top_k
        a.add = None if add is None else add.data_ptr()
        a.x, a.width, a.rows, a.eps = self.x.data_ptr(), s.hidden, R, s.norm_eps
        a.pre_w = None if pre is None else pre.data_ptr()
        a.norm, a.copy_h = S.NORM[s.norm], int(copy)
        a.h, a.h_f32, a.h_ld = self.h.data_ptr(), int(self.f32), self.h_ld
        with self.stage("rows"):
            S.rows(a)

    def _feed_forward(self, d: dict, R: int) -> torch.Tensor:
        """Returns the buffer that holds the result rows (sorted by expert for routed layers)."""
        f, W = d["spec"].mlp, self.spec.hidden
        fp = pad(f.ff, 8)
        if f.kind == "relu2":
            with self.stage("ff_up"):
                self.gemm(S.EPI_RELU2, d["up"], self.h, self.h_ld, R, self.ff, fp)
            with self.stage("ff_down"):
                self.gemm(S.EPI_STORE, d["down"], self.ff, fp, R, self.y, W)
            return self.y
        if f.kind == "dense":
            with self.stage("dense_gate_up"):
                self.gemm(S.EPI_CLAMPED_GLU, d["gate"], self.h, self.h_ld, R, self.ff, fp, w2=d["up"], limit=f.limit, alpha=f.alpha)
            with self.stage("dense_down"):
                self.gemm(S.EPI_STORE, d["down"], self.ff, fp, R, self.y, W)
            return self.y
        rt = f.routing
        with self.stage("router"):
            self.gemm(S.EPI_STORE, d["router"], self.h, self.h_ld, R, self.scores, rt.expert_count)
        q = K.RouterArgs()
        q.bias, q.hidden, q.experts, q.rows, q.top_k = d["correction"].data_ptr(), W, rt.expert_count, R, rt.top_k
        q.sigmoid, q.normalize, q.route_scale = 1, int(rt.normalize_top_k), rt.route_scale
        q.scores, q.topk_ids, q.topk_p = self.scores.data_ptr(), self.ids.data_ptr(), self.probs.data_ptr()
        with self.stage("choice"):
            S.route(q, rt.group_count, rt.limited_group_count)
        ir = self._item_rows(R, rt, self.f32)
        items = self._items(R, rt, ir)
        e = K.EpArgs()
        e.topk_ids, e.topk_p, e.tokens, e.top_k = self.ids.data_ptr(), self.probs.data_ptr(), R, rt.top_k
        e.experts = e.experts_local = rt.expert_count
        e.slot_of, e.n_items, e.item_expert, e.item_row = (self.slot_of.data_ptr(), self.n_items.data_ptr(), self.item_z.data_ptr(),
                                                           self.item_row.data_ptr())
        e.seg_rows, e.max_items, e.item_rows, e.x_args = self.seg_rows.data_ptr(), items, ir, self.t.fab.xchg_args()
        with self.stage("expert_count"):
            S.moe_count(e)
        g = S.MoeGatherArgs()
        eb = self.h.element_size()
        g.h, g.h_ld, g.sorted, g.slot_of = self.h.data_ptr(), self.h_ld * eb, self.sorted.data_ptr(), self.slot_of.data_ptr()
        g.rows, g.top_k, g.row_bytes, g.cap = R, rt.top_k, self.h_ld * eb, self.cap
        with self.stage("expert_gather"):
            S.moe_gather(g)
        seg = dict(items=(ir, items))
        with self.stage("expert_gate_up"):
            self.gemm(S.EPI_SILU_GLU, d["gate"], self.sorted, self.h_ld, ir, self.ea, fp, w2=d["up"], x_rows=self.cap, **seg)
        with self.stage("expert_down"):
            self.gemm(S.EPI_STORE, d["down"], self.ea, fp, ir, self.ey, W, x_rows=self.cap, **seg)
        return self.ey

    def _chunk(self, pos0: int, R: int, want: Sequence[int] = (), trace: Optional[list] = None) -> Optional[torch.Tensor]:
        """Rows [0, R) of ``tokens`` at positions pos0 ..: fills caches and states; logits of the rows in ``want``.
        ``trace`` collects the stream after every layer run."""
        t, s = self.t, self.spec
        self.pos.fill_(pos0)
        wait = dict(embed=True)                         # what the next row kernel adds to the stream first
        for r in t.runs:
            d, run = r["layer"], r["run"]
            add = None if run.pass_start is None else t.loop_step[run.pass_start]
            self._rows(R, add=add, pre=d["norm1"], copy=d["norm1"] is None and d["kind"] != "wkv", **wait)
            MIXERS[d["kind"]].run(self, r, R, pos0)
            wait = dict(y=self.y, post=d["norm1b"])
            if d["kind"] == "parallel":
                wait.update(y2=self.y2, join=(d["out"], d["out2"]))
            f = d["spec"].mlp
            if f is not None:
                self._rows(R, pre=d["norm2"], copy=d["norm2"] is None, **wait)
                wait = dict(y=self._feed_forward(d, R), post=d["norm2b"], moe=f.routing if f.kind == "moe" else None)
            if trace is not None:
                self._rows(R, **wait)
                wait = {}
                trace.append(self.x[:R].clone())
        if not len(want):
            return None
        self._rows(R, pre=t.g_final, **wait)
        idx = torch.as_tensor(list(want), dtype=torch.long, device=self.dev)
        out = torch.empty(len(idx), s.vocab, dtype=torch.float32, device=self.dev)
        for i in range(0, len(idx), self.head_rows):
            n = min(self.head_rows, len(idx) - i)
            self.hw[:n].copy_(self.h.index_select(0, idx[i:i + n]))
            self.gemm(S.EPI_STORE, t.head, self.hw, self.h_ld, n, out[i:i + n], s.vocab, scale=s.logit_scale)
        return out

    # ------------------------------------------------------------------ public API (that of ``NativePrefill``)
    def extend(self, tokens: torch.Tensor, pos0: int, want: Sequence[int] = (), trace: Optional[list] = None) -> torch.Tensor:
        """Feed ``tokens`` (host or device) at positions pos0 .. in chunks; logits [len(want), vocab] of the rows in ``want``."""
        n = int(tokens.numel())
        if not 0 <= pos0 <= pos0 + n <= self.t.capacity:
            raise ValueError(f"rows [{pos0}, {pos0 + n}) outside the cache capacity {self.t.capacity}")
        out: List[torch.Tensor] = []
        order = [w for w in want]
        if order != sorted(order):
            raise ValueError("wanted rows must ascend")
        for c0 in range(0, n, self.C):
            R = min(self.C, n - c0)
            self.tokens[:R].copy_(tokens[c0:c0 + R].to(torch.int32), non_blocking=True)
            got = self._chunk(pos0 + c0, R, [w - c0 for w in order if c0 <= w < c0 + R], trace)
            if got is not None:
                out.append(got)
        return torch.cat(out) if out else torch.empty(0, self.spec.vocab, dtype=torch.float32, device=self.dev)

    def run(self, prompt: torch.Tensor, start: int = 0, end: Optional[int] = None) -> int:
        n = int(prompt.numel())
        end = n if end is None else end
        if not 0 <= start <= end <= n or end > self.t.capacity:
            raise ValueError(f"prefill range [{start}, {end}) outside the prompt / cache capacity")
        ev = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        ev[0].record()
        self.extend(prompt[start:end], start)
        ev[1].record()
        self.phases = {"chunks": -(-(end - start) // self.C), "rows": end - start, "events": ev}
        return end

    def executor_ms(self) -> float:
        a, b = self.phases["events"]
        b.synchronize()
        return a.elapsed_time(b)

    def warm_chunks(self, sizes=None) -> None:
        """Run chunk sizes once at position 0 (module loading, kernel attributes); the next request overwrites the rows."""
        for r in sorted(set(sizes or [1, self.C])):
            self.tokens.zero_()
            self._chunk(0, min(r, self.C, self.t.capacity))
        torch.cuda.current_stream().synchronize()
        self.check()

    def check(self) -> None:
        self.t.fab.check()

    def close(self) -> None:
        self.maps.clear()
