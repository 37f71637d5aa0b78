"""Inference-side model execution for the decoder families: prefill of a prompt, steps that mix prompt portions with
decoded tokens, and batched single-token decode, all against a paged KV cache.  The runner assembles the rows of a step
(positions, cache slots, block tables), runs the model's layer body (serve.decoder_body, chosen by the configuration's
architecture) over them and replays decode steps from CUDA graphs.  Every matmul is the tcgen05 GEMM, prompt attention is
the flash kernel, decode attention the paged kernel; K and V of new tokens go straight from the packed projection into
their cache slots.  Layers with recurrent state find each sequence's rows and state slot in the step's segment table.

This is the model forward the reference's ServingEngine lacks (it fabricates token 1, crates/nn/src/continuous_batching.rs:516-526)
and the cached decode its TransformerDecoder::generate_token does not have (full re-forward per token, crates/nn/src/transformer.rs:837-862).
"""
from __future__ import annotations

import gc

import torch

from .. import ops
from ..models.registry import architecture, build_weights
from ..ops import attention as attn_ops
from ..ops import latent as latent_ops
from ..ops import paged as paged_ops
from ..ops import rotary as rope_ops
from ..ops.matmul import gemm
from ..ops.recurrent import Segments
from ..runtime.fused_gpt import FlatParams
from . import decoder_body
from .kv_cache import PagedCache


class StepBatch:
    """The rows of one model pass: prompt portions first (`spans`), then one row per decoded sequence (from row `rd`).
    `segments`: the same sequences for layers with recurrent state (None: the model has none)."""

    def __init__(self, ids, pos, slots, spans, rd, tables, bt, ctx, block_size, segments=None):
        self.ids, self.pos, self.slots = ids, pos, slots          # int64 device tensors, one entry per row
        self.spans = spans                                        # (first row, end row, first position) per portion
        self.rd, self.rows = rd, ids.shape[0]
        self.tables = tables                                      # block table (list) of every portion's sequence
        self.bt, self.ctx = bt, ctx                               # decode rows: block tables, context lengths (int32)
        self.block_size = block_size
        self.segments = segments
        self._keys, self._row_tables, self._rotations, self._all_keys = {}, None, {}, None

    def rotation(self, rot, freqs: torch.Tensor) -> torch.Tensor:
        """Cosines and sines of the rows' positions for the rotary positions `rot` (models.layered.RotarySpec), one table for all
        layers that share them."""
        if rot not in self._rotations:
            self._rotations[rot] = rope_ops.rotary_table(self.pos, freqs, rot.magnitude)
        return self._rotations[rot]

    def all_keys(self):
        """(cache slots of every position up to the end of each portion, one portion after the other; first entry of each portion and
        the end).  Slots are None where the portions are whole prompts: the keys are the step's own rows."""
        if self._all_keys is None:
            ends = [0]
            for r0, r1, start in self.spans:
                ends.append(ends[-1] + start + r1 - r0)
            whole = all(start == 0 for _, _, start in self.spans)
            slots = None if whole else torch.cat([self.key_slots(i, 0) for i in range(len(self.spans))])
            self._all_keys = (slots, ends)
        return self._all_keys

    def key_slots(self, i: int, first: int, kept: int = 0) -> torch.Tensor:
        """Cache slots of positions 0 .. `kept` and `first` .. end of portion i (earlier portions and this one)."""
        key = (i, first, kept)
        if key not in self._keys:
            r0, r1, start = self.spans[i]
            bs = self.block_size
            pos = torch.cat([torch.arange(kept), torch.arange(first, start + r1 - r0)])
            self._keys[key] = (torch.tensor(self.tables[i], dtype=torch.int64)[pos // bs] * bs + pos % bs).to(self.ids.device)
        return self._keys[key]

    def row_tables(self):
        """(block tables int32 [sequences, width], sequence index int32 per row) over all rows of the step."""
        if self._row_tables is None:
            if not self.spans:
                self._row_tables = (self.bt, torch.arange(self.rows, dtype=torch.int32, device=self.ids.device))
            else:
                seq = [i for i, (r0, r1, _) in enumerate(self.spans) for _ in range(r1 - r0)]
                seq += [len(self.spans) + i for i in range(self.rows - self.rd)]
                width = max([len(t) for t in self.tables] + ([self.bt.shape[1]] if self.bt is not None else []))
                bt = torch.tensor([t + [0] * (width - len(t)) for t in self.tables], dtype=torch.int32)
                bt = bt.to(self.ids.device)
                if self.bt is not None:
                    bt = torch.cat([bt, torch.nn.functional.pad(self.bt, (0, width - self.bt.shape[1]))], 0)
                self._row_tables = (bt, torch.tensor(seq, dtype=torch.int32, device=self.ids.device))
        return self._row_tables


class ModelRunner:
    """`tp` (a parallel.tp_inference.TPInferenceComm) makes this rank one shard of a tensor-parallel model: `params`
    then holds this rank's shard (serve.weights.InferenceWeights), the cache holds this rank's KV heads, and the
    attention-output, down-projection and LM-head results are exchanged with one-shot peer-memory collectives.  All
    ranks run the same calls in the same order and obtain bit-identical logits.

    `dtype` (bf16 or fp32, where the architecture runs in both) applies when `params` is not given.  `num_slots`: sequences
    that can hold recurrent state at a time (models without such layers have no limit of that kind)."""

    def __init__(self, cfg, params=None, device=None, num_blocks: int = 1024, block_size: int = 16, seed: int = 0, tp=None,
                 dtype=None, num_slots: int = 64):
        if device is None:
            device = "cuda" if torch.cuda.is_available() else "cpu"
        self.cfg = cfg
        self.device = torch.device(device)
        self.tp = tp
        self.tp_world = tp.world if tp is not None else 1
        gpt = cfg.arch in ("gpt2", "llama")
        if tp is not None:
            if cfg.arch != "llama" or cfg.n_head % tp.world or cfg.n_kv_head % tp.world or cfg.ffn_dim % tp.world or \
                    cfg.vocab_padded % (8 * tp.world):
                raise ValueError("tensor-parallel serving: llama-style model whose heads, FFN and vocabulary divide evenly")
            if params is None:
                from .weights import InferenceWeights
                params = InferenceWeights.random_llama(cfg, self.device, tp.rank, tp.world, seed)
        if params is None:
            params = FlatParams(cfg, self.device, seed) if gpt else build_weights(cfg, self.device, dtype, None, seed)
        self.params = params
        self.dtype = self.params.lowp.dtype
        if gpt:
            self.n_head, self.n_kv_head = cfg.n_head // self.tp_world, cfg.n_kv_head // self.tp_world
        self.body = getattr(decoder_body, architecture(cfg.arch).body)(self)
        layers = self.body.cache_layers()
        if layers is None:
            self.cache = PagedCache(num_blocks, block_size, cfg.n_layer, self.n_kv_head, cfg.head_dim, self.dtype, self.device)
        else:
            self.cache = PagedCache(num_blocks, block_size, dtype=self.dtype, device=self.device, layers=layers, num_slots=num_slots)
        self.recurrent = self.cache.num_slots > 0
        self.block_size = block_size
        self.use_graphs = True          # CUDA-graph replay of decode steps
        self._graphs: dict = {}

    # ---- attention over the rows of a step -------------------------------------------------------------------------
    def attend(self, l: int, q, k2, v2, sb: StepBatch, scale: float, rule=None, gate=None, head_gate=None, out=None) -> torch.Tensor:
        """Attention of layer `l` for every row of `sb`; the rows' keys and values (`k2`, `v2`) are already in the cache.
        Prompt portions go through the flash kernel (keys: the cached positions the portion can still see, gathered from the
        pages, plus the portion itself), decoded rows through the paged kernel; operands that those do not take (fp32,
        unusual head sizes) go through the paged row kernel.  `rule`: ops.ScoreRule; `gate` (one number per value
        column) or `head_gate` (fp32, one per head): output times sigmoid(gate); `out` (a row-strided view) receives it."""
        kc, vc = self.cache.k[l], self.cache.v[l]
        nb, bs, G, dk = kc.shape
        dv = vc.shape[3]
        H = q.shape[1] // dk
        T = sb.rows
        flash = attn_ops.prompt_supported(q, k2, v2, dk, dv, rule, gate)
        paged = paged_ops.decode_supported(q, dk, dv, rule, gate)
        if (sb.spans and not flash) or (sb.rd < T and not paged):
            bt, seq = sb.row_tables()
            return paged_ops.paged_attention_rows(q, kc, vc, bt, seq, sb.pos, scale, rule, gate, out, head_gate)
        a = out if out is not None else torch.empty((T, H * dv), dtype=q.dtype, device=self.device)
        for i, (r0, r1, start) in enumerate(sb.spans):
            L = r1 - r0
            kept, first = rule.key_ranges(start) if rule is not None else (0, 0)
            if first == start and kept == 0:
                kk, vv = k2[r0:r1].view(1, L, G, dk), v2[r0:r1].view(1, L, G, dv)
            else:
                cs = sb.key_slots(i, first, kept)
                kk = ops.gather_rows(kc.view(nb * bs, G * dk), cs).view(1, -1, G, dk)
                vv = ops.gather_rows(vc.view(nb * bs, G * dv), cs).view(1, -1, G, dv)
            attn_ops.prompt_attention(q[r0:r1].view(1, L, H, dk), kk, vv, scale, out=a[r0:r1].view(1, L, H, dv), rule=rule,
                                      gate=None if gate is None else gate[r0:r1],
                                      head_gate=None if head_gate is None else head_gate[r0:r1])
        if sb.rd < T:
            paged_ops.paged_attention_decode(q[sb.rd:], kc, vc, sb.bt, sb.ctx, scale, out=a[sb.rd:], rule=rule,
                                             gate=None if gate is None else gate[sb.rd:],
                                             head_gate=None if head_gate is None else head_gate[sb.rd:])
        return a

    def attend_latent(self, l: int, q, kv, sb: StepBatch, m, w_ukv, table, gate=None) -> torch.Tensor:
        """Latent attention of layer `l` (`m`: models.layered.LatentSpec) for every row of `sb`.  q [rows, heads * qk_dim] (not rotated
        yet), kv [rows, cached]: the vectors and rotated key parts, already in the cache; w_ukv: the heads' key products, then their
        value products.  Prompt portions form keys and values of all positions they see and go through the flash kernel; decoded rows
        (and portions that it does not take) work on the cached vectors."""
        H, dn, dr, dv, R = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        cache, T, rd = self.cache.k[l], sb.rows, sb.rd
        a = torch.empty((T, H * dv), dtype=q.dtype, device=self.device)
        flash = False
        if sb.spans:
            slots, ends = sb.all_keys()
            keys = kv[:rd] if slots is None else ops.gather_rows(cache.view(-1, m.cached), slots)
            flash = attn_ops.split_supported(dn, dr, dv, q, keys, keys[:, R:], gate)
        if flash:
            both = gemm(keys[:, :R], w_ukv)                       # keys of all heads, then values of all heads
            rope_ops.rotate_pairs_(q[:rd], H, m.qk_dim, dn, table[:rd])
            for i, (r0, r1, _) in enumerate(sb.spans):
                L, k0, k1 = r1 - r0, ends[i], ends[i + 1]
                attn_ops.prompt_attention_split(q[r0:r1].view(1, L, H, dn + dr), both[k0:k1, :H * dn].view(1, -1, H, dn),
                                                both[k0:k1, H * dn:].view(1, -1, H, dv), keys[k0:k1, R:], m.scale,
                                                out=a[r0:r1].view(1, L, H, dv), gate=None if gate is None else gate[r0:r1])
        lo = rd if flash else 0                                   # rows that work on the cached vectors
        if lo < T:
            qa = latent_ops.head_product(q[lo:], m.qk_dim, w_ukv[:H * dn], H, R, dn, transposed=True, tail=dr, table=table[lo:])
            if lo == rd and latent_ops.latent_decode_supported(qa, R, dr):
                c = latent_ops.latent_decode(qa, cache, R, sb.bt, sb.ctx, m.scale)
            else:
                bt, seq = sb.row_tables()
                c = paged_ops.paged_attention_rows(qa, cache, self.cache.v[l], bt, seq[lo:], sb.pos[lo:], m.scale)
            latent_ops.head_product(c, R, w_ukv[H * dn:], H, dv, R, transposed=False, gate=None if gate is None else gate[lo:], out=a[lo:])
        return a

    # ---- one model pass ----------------------------------------------------------------------------------------------
    def _run(self, sb: StepBatch, rows) -> torch.Tensor | None:
        """All layers over the rows of `sb`; logits of the rows `rows` (int64 tensor, None: every row, [] : none)."""
        x = self.body.embed(sb)
        for l in range(self.body.depth):
            x = self.body.layer(l, x, sb)
        logits = None if isinstance(rows, list) else self.body.head(x, rows)
        if self.tp is not None:
            self.tp.end_step()
        return logits

    @torch.no_grad()
    def prefill(self, seq_id: int, tokens: list) -> torch.Tensor:
        """Runs the whole prompt, fills the cache slots of `seq_id` (which must have blocks reserved) and returns the
        logits of the last position, [vocab_padded]."""
        return self.step_mixed([(seq_id, tokens, 0, True)], [], [], [])[0][0]

    @torch.no_grad()
    def step_mixed(self, chunks: list, dec_ids: list, dec_tok: list, dec_len: list):
        """One model pass over several prompt chunks and the decode batch.

        `chunks`: list of (seq_id, tokens, start, want): `tokens` are positions [start, start + len) of the sequence's
        prefix; everything before `start` is already in the cache.  `want`: True for the logits of the last position,
        False for none, or a list of places among `tokens`.  `dec_*`: as for `decode`.  All rows go through the
        projections, the MLP and the collectives together (the weights are read once per step); attention runs per part.
        Returns (per chunk: logits [vocab_padded], None, or [len(want), vocab_padded]; decode logits
        [len(dec_ids), vocab_padded] or None).
        (Batched and chunked prefill of the reference's scheduler: crates/nn/src/continuous_batching.rs:248-295.)"""
        dev, bs = self.device, self.block_size
        ids_h, pos_h, slot_h, spans, tables = [], [], [], [], []
        for seq_id, tokens, start, _ in chunks:
            table = self.cache.block_table(seq_id)
            L = len(tokens)
            spans.append((len(ids_h), len(ids_h) + L, start))
            tables.append(table)
            ids_h += list(tokens)
            pos_h += list(range(start, start + L))
            slot_h += [table[p_ // bs] * bs + p_ % bs for p_ in range(start, start + L)]
        rd = len(ids_h)
        for seq_id, tok, n in zip(dec_ids, dec_tok, dec_len):
            table = self.cache.block_table(seq_id)
            ids_h.append(tok)
            pos_h.append(n - 1)
            slot_h.append(table[(n - 1) // bs] * bs + (n - 1) % bs)
        T = len(ids_h)
        host = torch.tensor([ids_h, pos_h, slot_h], dtype=torch.int64).to(dev)
        bt = ctx = None
        if dec_ids:
            width = max(len(self.cache.block_table(s_)) for s_ in dec_ids)
            bt = self._fill_tables(dec_ids, width).to(dev)
            ctx = torch.tensor(dec_len, dtype=torch.int32, device=dev)
        segments = None
        if self.recurrent:
            table = [(r0, r1 - r0, self.cache.state_slot(c[0]), start) for (r0, r1, start), c in zip(spans, chunks)]
            table += [(rd + i, 1, self.cache.state_slot(s_), n - 1) for i, (s_, n) in enumerate(zip(dec_ids, dec_len))]
            segments = Segments.of(table, dev)
        sb = StepBatch(host[0], host[1], host[2], spans, rd, tables, bt, ctx, bs, segments)
        # logits only where they are asked for: by default the last row of every chunk that completes its prompt, and the
        # decode rows
        want = []
        for (r0, r1, _), c in zip(spans, chunks):
            want.append([r1 - 1] if c[3] is True else [r0 + i for i in c[3]] if c[3] else [])
        rows = [r for w in want for r in w] + list(range(rd, T))
        if rows and rows != list(range(T)):
            sel = torch.tensor(rows, dtype=torch.int64, device=dev)
        else:
            sel = None if rows else []
        logits = self._run(sb, sel)
        out, at = [], 0
        for w, c in zip(want, chunks):
            part = logits[at:at + len(w)] if w else None
            out.append(part[0] if c[3] is True else part)
            at += len(w)
        return out, (logits[at:] if dec_ids else None)

    def step(self, chunks: list, dec_ids: list, dec_tok: list, dec_len: list):
        """One engine iteration: `step_mixed` when there is prompt work, else the graphed `decode`."""
        if chunks:
            return self.step_mixed(chunks, dec_ids, dec_tok, dec_len)
        return [], (self.decode(dec_ids, dec_tok, dec_len) if dec_ids else None)

    # ---- decode ------------------------------------------------------------------------------------------------------
    def _decode_segments(self, seq_ids, context_lens) -> list:
        return [(i, 1, self.cache.state_slot(s), n - 1) for i, (s, n) in enumerate(zip(seq_ids, context_lens))]

    def _decode_body(self, ids, ctx, bt, segments=None):
        """The device-side part of a decode step on static tensors (captured into a CUDA graph per batch size)."""
        B, bs = ids.shape[0], self.block_size
        pos = (ctx - 1).to(torch.int64)
        slots = bt.gather(1, (pos // bs).view(B, 1)).view(B).to(torch.int64) * bs + pos % bs
        return self._run(StepBatch(ids, pos, slots, [], 0, [], bt, ctx, bs, segments), None)

    def _fill_tables(self, seq_ids, width: int) -> torch.Tensor:
        tables = [self.cache.block_table(s) for s in seq_ids]
        bt_host = torch.zeros((len(seq_ids), width), dtype=torch.int32)
        for i, t in enumerate(tables):
            bt_host[i, :len(t)] = torch.tensor(t, dtype=torch.int32)
        return bt_host

    @torch.no_grad()
    def decode(self, seq_ids: list, last_tokens: list, context_lens: list) -> torch.Tensor:
        """One new token per sequence.  context_lens[i] counts the tokens in the cache AFTER this token is appended.
        Returns logits [batch, vocab_padded] (with CUDA graphs: valid until the next decode call)."""
        dev = self.device
        if self.use_graphs and dev.type == "cuda":
            return self._decode_graphed(seq_ids, last_tokens, context_lens)
        ids = torch.tensor(last_tokens, dtype=torch.int64, device=dev)
        ctx = torch.tensor(context_lens, dtype=torch.int32, device=dev)
        max_blocks = max(len(self.cache.block_table(s)) for s in seq_ids)
        bt = self._fill_tables(seq_ids, max_blocks).to(dev)
        seg = Segments.of(self._decode_segments(seq_ids, context_lens), dev) if self.recurrent else None
        return self._decode_body(ids, ctx, bt, seg)

    def _table_width(self, context_lens) -> int:
        """Block-table columns of a graphed decode step: the model's whole context when that is at most 1024 blocks, else
        the next power of two above what the batch needs now (a graph per width, so that the split-KV grid stays small)."""
        full = min((self.cfg.seq_len + self.block_size - 1) // self.block_size, self.cache.num_blocks)
        if full <= 1024:
            return full
        need = (max(context_lens) + self.block_size - 1) // self.block_size
        return min(full, max(64, 1 << (need - 1).bit_length()))

    def _decode_graphed(self, seq_ids, last_tokens, context_lens) -> torch.Tensor:
        """Replays one captured CUDA graph per batch size: the 10 to 20 launches per layer of a decode step are
        launch-bound from Python, the graph submits them in one call.  Inputs live in static device tensors that
        are refreshed (a few small copies) before each replay."""
        B = len(seq_ids)
        dev = self.device
        width = self._table_width(context_lens)
        g = self._graphs.get((B, width))
        if g is None:
            ids = torch.zeros(B, dtype=torch.int64, device=dev)
            ctx = torch.ones(B, dtype=torch.int32, device=dev)
            bt = torch.zeros((B, width), dtype=torch.int32, device=dev)
            g = {"ids": ids, "ctx": ctx, "bt": bt, "seg": None, "graph": None, "out": None}
            if self.recurrent:
                g["seg"] = Segments(torch.zeros((B, 4), dtype=torch.int32, device=dev), None)
            self._graphs[(B, width)] = g
        g["ids"].copy_(torch.tensor(last_tokens, dtype=torch.int64), non_blocking=True)
        g["ctx"].copy_(torch.tensor(context_lens, dtype=torch.int32), non_blocking=True)
        g["bt"].copy_(self._fill_tables(seq_ids, width), non_blocking=True)
        if g["seg"] is not None:
            g["seg"].table.copy_(torch.tensor(self._decode_segments(seq_ids, context_lens), dtype=torch.int32), non_blocking=True)
        if g["graph"] is None:
            # first use of this batch size: one eager run (lazy kernel configuration, tensor-map cache), then capture
            out = self._decode_body(g["ids"], g["ctx"], g["bt"], g["seg"])
            torch.cuda.current_stream().synchronize()
            graph = torch.cuda.CUDAGraph()
            # A collection in the middle of a capture could destroy an earlier runner's graphs, which ends the capture with an error
            collecting = gc.isenabled()
            gc.disable()
            try:
                with torch.cuda.graph(graph):
                    g["out"] = self._decode_body(g["ids"], g["ctx"], g["bt"], g["seg"])
            finally:
                if collecting:
                    gc.enable()
            g["graph"] = graph
            return out
        g["graph"].replay()
        return g["out"]


def load_runner(model: str, device=None, dtype=None, num_blocks: int = 1024, block_size: int = 16, weights: str | None = None,
                seed: int = 0, num_slots: int = 64, **overrides) -> ModelRunner:
    """Runner of a preset name or of a model folder (config.json + model.safetensors, the model class chosen by the
    configuration); `weights` names another safetensors file.  Without weights: random initialisation."""
    from ..models.registry import load_tensors, resolve_config
    cfg = resolve_config(model, **overrides)
    if device is None:
        device = "cuda" if torch.cuda.is_available() else "cpu"
    params = build_weights(cfg, device, dtype, load_tensors(model, weights), seed)
    return ModelRunner(cfg, params=params, device=device, num_blocks=num_blocks, block_size=block_size, seed=seed,
                       num_slots=num_slots)
