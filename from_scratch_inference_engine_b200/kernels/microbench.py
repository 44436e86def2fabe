"""Times single kernels at given sizes and prints achieved GB/s or TFLOP/s.

    python -m from_scratch_inference_engine_b200.kernels.microbench KERNEL [options]

KERNEL: attention_decode, attention_prefill, add_rmsnorm, rope_kv_write, swiglu, argmax,
sample, linear (the library product as the engine calls it), gemm_f32, gemm_decode,
gemm_decode_swiglu, gemm_tiles, gemm_tiles_swiglu (the engine's own tcgen05 products),
sum_layernorm, routed_experts (every kernel of a feed-forward of routed experts, one line for all),
state_space (every kernel of a state-space mixer, and the same scan with one decay per head beside it),
stream_norm (a residual of --streams streams settled, gathered and normed), scaled_attention (capped scores
inside chunks of --chunk positions, gated columns: a prompt of --tokens behind --context - --tokens cached
ones on tcgen05, or - --tokens 1 - decoded tokens of --batch requests on mma.sync; all flops are useful ones).

Each kernel is timed with CUDA events over --iters launches after --warmup launches; between
launches a buffer larger than L2 is read so that inputs come from HBM (read, not written:
dirty lines would be written back during the timed kernel).  One JSON line
per run: time, algorithmic bytes and flops, achieved rates and their fraction of the peaks
in MEASURED_PEAKS.json at the repository root (or of 6,650 GB/s and 1,590 TFLOP/s when that
file is absent).  The same command under `ncu` profiles exactly this kernel at this size.
"""

from __future__ import annotations

import argparse
import json
import math
import sys
from pathlib import Path

import torch

from . import ops

ROOT = Path(__file__).resolve().parents[2]


def peaks():
    values = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    path = ROOT / "MEASURED_PEAKS.json"
    if path.exists():
        try:
            data = json.loads(path.read_text())
            for key in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                value = data.get(key) if isinstance(data, dict) else None
                if isinstance(value, dict):        # a record with the figure inside
                    value = next((value[k] for k in ("value", "median", "mean") if k in value), None)
                if isinstance(value, (int, float)) and value > 0:
                    values[key] = float(value)
                    values["source"] = "measured"
        except (OSError, ValueError, TypeError):
            pass
    return values


class Timer:
    def __init__(self, warmup: int, iters: int, flush: bool = True):
        self.warmup, self.iters = warmup, iters
        self.flush = torch.zeros(256 * 1024 * 1024, dtype=torch.uint8, device="cuda") if flush else None

    def __call__(self, fn) -> float:
        for _ in range(self.warmup):
            fn()
        times = []
        for _ in range(self.iters):
            if self.flush is not None:
                self.flush.view(torch.int32).sum()
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            start.record()
            fn()
            end.record()
            torch.cuda.synchronize()
            times.append(start.elapsed_time(end))
        times.sort()
        return times[len(times) // 2]          # median, ms


def paged_inputs(batch, new, past, heads, kv_heads, hd, page, dtype):
    """Random pages, shuffled block tables and queries for `batch` requests with `past`
    cached tokens and `new` tokens each."""
    g = torch.Generator(device="cuda").manual_seed(0)
    total = past + new
    blocks = -(-total // page)
    pages = torch.randn((batch * blocks + 1, 1, 2, kv_heads, page, hd), generator=g, device="cuda",
                        dtype=torch.float32).to(dtype)
    order = torch.randperm(batch * blocks, generator=g, device="cuda").to(torch.int32)
    tables = order.view(batch, blocks).contiguous()
    q = torch.randn((batch * new, (heads + 2 * kv_heads) * hd), generator=g, device="cuda",
                    dtype=torch.float32).to(dtype)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    return pages, tables, q, i32([i * new for i in range(batch)]), i32([new] * batch), \
        i32([past] * batch)


def run_attention(args, timer, decode: bool):
    heads, kv_heads, hd, page = args.heads, args.kv_heads, args.head_dim, args.page
    new = 1 if decode else args.tokens
    past = args.context - new
    dtype = torch.bfloat16 if args.dtype == "bfloat16" else torch.float32
    pages, tables, q, qstart, qlen, pos0 = paged_inputs(args.batch, new, past, heads, kv_heads, hd,
                                                        page, dtype)
    group = heads // kv_heads
    tokens = args.batch * new
    out = torch.empty((tokens, heads * hd), dtype=dtype, device="cuda")
    rows = new * group
    sms = torch.cuda.get_device_properties(0).multi_processor_count
    if dtype is torch.bfloat16:
        row_class = next((c for c, r in enumerate(ops.ATTENTION_ROW_CLASSES) if rows <= r), 2)
        per_tile = ops.ATTENTION_ROW_CLASSES[row_class]
        if args.variant == "tc" and row_class == 2:
            per_tile = ops.ATTENTION_TC_ROWS
    else:
        rows16 = args.variant == "rows16" and rows <= ops.attention_rows16_rows()
        row_class, per_tile = -1, ops.attention_rows16_rows() if rows16 else ops.attention_rows_per_tile()
    tile_item, tile_row0 = [], []
    for i in range(args.batch):
        for r0 in range(0, rows, per_tile):
            tile_item.append(i)
            tile_row0.append(r0)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    # as the engine lists them: the tiles that see the most keys first
    by_keys = sorted(range(len(tile_item)), key=lambda n: -(past + (min(tile_row0[n] + per_tile, rows) - 1) // group))
    tile_item, tile_row0 = [tile_item[n] for n in by_keys], [tile_row0[n] for n in by_keys]
    tile_item, tile_row0 = i32(tile_item), i32(tile_row0)
    nsplit = args.nsplit
    if nsplit <= 0:
        from ..parts.attention import attention_splits
        nsplit = attention_splits(tile_item.numel() * kv_heads, args.context, sms, decode,
                                  1 if args.variant == "tc" and row_class == 2 else 2)
    part_o = torch.empty(max(1, nsplit * tokens * heads * hd), device="cuda")
    part_ml = torch.empty(max(1, nsplit * tokens * heads * 2), device="cuda")
    scale = 1.0 / math.sqrt(hd)

    use_tc = args.variant == "tc" and row_class == 2
    use_tcd = args.variant == "tc" and row_class == 0 and hd in ops.ATTENTION_TC_DECODE_HEAD_DIMS
    if use_tc or use_tcd:
        pages_map = ops.PagesMap(pages, "tc")
        error = torch.zeros(1, dtype=torch.int32, device="cuda")

    def launch():
        if use_tcd:
            ops.attention_tc_decode(pages_map, 0, q, q.stride(0), tables, tile_item, tile_row0,
                                    tile_item.numel(), qstart, qlen, pos0, out, tokens, heads,
                                    kv_heads, 0, scale, error, nsplit, part_o, part_ml, None, 0)
        elif use_tc:
            ops.attention_tc(pages_map, 0, q, q.stride(0), tables, tile_item, tile_row0,
                             tile_item.numel(), qstart, qlen, pos0, out, tokens, heads, kv_heads,
                             0, scale, error, nsplit, part_o, part_ml, None, 0)
        elif row_class >= 0:
            ops.attention_mma(row_class, q, q.stride(0), pages[:, 0, 0], pages[:, 0, 1],
                              pages.stride(0), page, tables, tile_item, tile_row0,
                              tile_item.numel(), qstart, qlen, pos0, out, tokens, heads, kv_heads,
                              hd, 0, scale, nsplit, part_o, part_ml, None, 0)
        else:
            ops.attention_generic(q, q.stride(0), pages[:, 0, 0], pages[:, 0, 1], pages.stride(0),
                                  page, tables, tile_item, tile_row0, tile_item.numel(), qstart,
                                  qlen, pos0, out, tokens, heads, kv_heads, hd, 0, scale, nsplit,
                                  part_o, part_ml, rows16=rows16)
    ms = timer(launch)
    extra = {}
    elem = 2 if dtype is torch.bfloat16 else 4
    kv_bytes = args.batch * args.context * 2 * kv_heads * hd * elem
    io_bytes = kv_bytes + 2 * tokens * heads * hd * elem
    # causal: query t of a portion sees past + t + 1 keys
    pairs = args.batch * (new * past + new * (new + 1) / 2)
    flops = 4.0 * heads * hd * pairs
    if use_tc or use_tcd:
        extra["error"] = int(error.item())
    extra.update({"nsplit": nsplit, "tiles": tile_item.numel(),
                  "variant": ("tc" if use_tc else "tc_decode" if use_tcd else "mma")
                  if row_class >= 0 else ("rows16" if rows16 else "generic")})
    return ms, io_bytes, flops, extra


def run_scaled_attention(args, timer):
    """Attention with 32-bit weights over shuffled pages: --softcap (0: none), chunks or a window, a gate per
    column or per head, sinks; --maps 2: two keys side by side in a row, their ranges left for the merge of
    differences, which is timed with it."""
    from ..parts.attention import attention_splits
    from ..parts.scaled_attention import key_splits
    heads, kv_heads, hd, page, new = args.heads, args.kv_heads, args.head_dim, args.page, args.tokens
    batch, past, chunk = args.batch if new == 1 else 1, args.context - new, args.chunk
    pages, tables, _, qstart, qlen, pos0 = paged_inputs(batch, new, past, heads, kv_heads, hd, page, torch.bfloat16)
    group, tokens = heads // kv_heads, batch * new
    wide = torch.randn(tokens, 2 * heads * hd, device="cuda").bfloat16()         # queries beside their gates
    gate = wide[:, heads * hd:] if args.gate else None
    head_gate = wide[:, heads * hd:heads * hd + heads] if args.head_gate else None
    maps, window = args.maps, args.window
    if maps == 2:                                  # as many query heads for every map, half as wide
        heads, group = 2 * heads, 2 * group
    scale = torch.full((heads,), hd ** -0.5, device="cuda")
    sink = torch.randn(heads, device="cuda") if args.sink else None
    out = torch.empty(tokens, heads * hd, dtype=torch.bfloat16, device="cuda")
    error = torch.zeros(1, dtype=torch.int32, device="cuda")
    sms = torch.cuda.get_device_properties(0).multi_processor_count
    per_tile = 16 if new == 1 else ops.ATTENTION_TC_ROWS
    tiles = [(i, r) for i in range(batch) for r in range(0, new * group, per_tile)]
    tiles.sort(key=lambda t: -t[1])
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    item, row0 = i32([t[0] for t in tiles]), i32([t[1] for t in tiles])
    seen = lambda pos: min(pos % chunk + 1 if chunk else pos + 1, window or pos + 1)
    reach = chunk or window
    longest = min(args.context, reach + per_tile) if reach else args.context
    nsplit = args.nsplit or (key_splits(len(tiles) * kv_heads, longest, sms, key_tile=64) if new == 1 else
                             attention_splits(len(tiles) * kv_heads, longest, sms, False, blocks_per_sm=1))
    parts = (torch.empty(nsplit * tokens * heads * hd, device="cuda"), torch.empty(nsplit * tokens * heads * 2, device="cuda"))
    options = dict(chunk=chunk, softcap=args.softcap, gate=gate, sink=sink, maps=maps, partial=maps == 2,
                   head_gate=None if maps == 2 else head_gate)

    def merged(attention):
        def run():
            attention()
            if maps == 2:
                ops.difference_merge(*parts, out, tokens, heads // 2, hd, nsplit, 0.6, 1e-6, 0.4, head_gate)
        return run
    if new == 1:
        slots = i32(list(range(batch)))
        ms = timer(merged(lambda: ops.scaled_attention(
            wide, wide.stride(0), scale, pages[:, 0, 0], pages[:, 0, 1], pages.stride(0), page, hd, hd, False, tables, item,
            row0, len(tiles), qstart, qlen, pos0, slots, out, tokens, heads, kv_heads, window, error, nsplit, *parts,
            form="mma_few", **options)))
    else:
        pages_map = ops.PagesMap(pages, "tc")
        ms = timer(merged(lambda: ops.attention_tc_scaled(
            pages_map, 0, wide, wide.stride(0), scale, tables, item, row0, len(tiles), qstart, qlen, pos0, out, tokens,
            heads, kv_heads, window, error, nsplit, *parts, **options)))
    keys = sum(seen(past + t) for t in range(new))
    read = batch * min(args.context, seen(args.context - 1) if new == 1 else args.context)
    nbytes = 2 * (read * 2 * kv_heads * hd + tokens * heads * hd * (3 if args.gate else 2))
    # a query of two maps is half as wide as its key row
    return ms, nbytes, (4.0 if maps == 1 else 3.0) * heads * hd * batch * keys, {"nsplit": nsplit, "tiles": len(tiles), "error": int(error.item())}


def run_routed_experts(args, timer, dtype):
    """Every kernel of a feed-forward of routed experts at --tokens, --hidden, --inter (an expert's
    width), --experts, --top, --groups, --keep with a random router: ms, and the share of the
    measured peak that the work a token asks for (no padding rows counted) reaches.  Steps with at
    least 32 rows per expert take the grouped tcgen05 products, others the tiles of 64 rows."""
    g = torch.Generator(device="cuda").manual_seed(0)
    rand = lambda *shape: torch.randn(shape, generator=g, device="cuda", dtype=torch.float32)
    elem = 2 if dtype is torch.bfloat16 else 4
    tokens, h, f, experts, top = args.tokens, args.hidden, args.inter, args.experts, args.top
    pairs = tokens * top
    y = rand(tokens, h).to(dtype)
    w_router = (rand(experts, h) / math.sqrt(h)).to(dtype)
    w_gu = (rand(experts, 2 * f, h) / math.sqrt(h)).to(dtype)
    w_d = (rand(experts, h, f) / math.sqrt(f)).to(dtype)
    correction = rand(experts) * 0.1
    ids = torch.zeros(tokens, top, dtype=torch.int32, device="cuda")
    weights = torch.zeros(tokens, top, device="cuda")
    logits = torch.nn.functional.linear(y, w_router).float()
    peak = peaks()
    rows = []

    def note(name, ms, nbytes, flops):
        gbs, tflops = nbytes / (ms * 1e-3) / 1e9, flops / (ms * 1e-3) / 1e12
        rows.append({"kernel": name, "ms": round(ms, 5), "GB/s": round(gbs, 1), "TFLOP/s": round(tflops, 2),
                     "frac_hbm": round(gbs / peak["hbm_gbs"], 3), "frac_bf16": round(tflops / peak["bf16_tflops"], 3)})

    note("moe_route", timer(lambda: ops.moe_route(None, None, correction, ids, weights, top, args.groups,
                                                  args.keep, 2.5, logits=logits)),
         tokens * (experts * 4 + top * 8), 0.0)
    used = int(torch.unique(ids).numel())
    shared = rand(tokens, h).to(dtype)
    out = torch.empty(tokens, h, dtype=dtype, device="cuda")
    error = torch.zeros(1, dtype=torch.int32, device="cuda")
    grouped = dtype is torch.bfloat16 and pairs >= 32 * experts and not args.no_grouped
    if grouped:
        tile = ops.GEMM_TILES_ROWS
        room = (pairs // tile + experts) * tile
        buffer = torch.zeros(ops.moe_lists_size(pairs, experts, tile, True), dtype=torch.int32, device="cuda")
        lists = ops.moe_align(ids, pairs, experts, buffer, tile, True)
        note("moe_align", timer(lambda: ops.moe_align(ids, pairs, experts, buffer, tile, True)), pairs * 12, 0.0)
        padded = int(lists[4].item()) * tile
        x_sorted = torch.empty(room, h, dtype=dtype, device="cuda")
        note("moe_gather", timer(lambda: ops.moe_gather(y, lists, tile, top, x_sorted)),
             (tokens + pairs) * h * elem, 0.0)
        gate_up, down = ops.GroupedTiledWeight(w_gu, True, "silu"), ops.GroupedTiledWeight(w_d, False)
        act = torch.empty(room, f, dtype=dtype, device="cuda")
        sms = torch.cuda.get_device_properties(0).multi_processor_count
        note("gemm_tiles_grouped gate,up", timer(lambda: ops.gemm_tiles_grouped(gate_up, x_sorted, act, lists[2], lists[4], error, sms)),
             (used * 2 * f * h + pairs * (h + f)) * elem, 2.0 * pairs * 2 * f * h)
        expert_out = torch.empty(room, h, dtype=dtype, device="cuda")
        note("gemm_tiles_grouped down", timer(lambda: ops.gemm_tiles_grouped(down, act, expert_out, lists[2], lists[4], error, sms)),
             (used * f * h + pairs * (h + f)) * elem, 2.0 * pairs * f * h)
        note("moe_combine", timer(lambda: ops.moe_combine(expert_out, weights, shared, out, top, place=lists[5])),
             (pairs + 2 * tokens) * h * elem, 2.0 * pairs * h)
        extra = {"rows_with_padding": padded}
    else:
        buffer = torch.zeros(ops.moe_lists_size(pairs, experts), dtype=torch.int32, device="cuda")
        lists = ops.moe_align(ids, pairs, experts, buffer)
        note("moe_align", timer(lambda: ops.moe_align(ids, pairs, experts, buffer)), pairs * 8, 0.0)
        act = torch.empty(pairs, f, dtype=dtype, device="cuda")
        note("moe_product gate,up", timer(lambda: ops.moe_product(y, w_gu, act, lists, pairs, top, True, "silu")),
             (used * 2 * f * h + tokens * h + pairs * f) * elem, 2.0 * pairs * 2 * f * h)
        expert_out = torch.empty(pairs, h, dtype=dtype, device="cuda")
        note("moe_product down", timer(lambda: ops.moe_product(act, w_d, expert_out, lists, pairs, top, False)),
             (used * f * h + pairs * (h + f)) * elem, 2.0 * pairs * f * h)
        note("moe_combine", timer(lambda: ops.moe_combine(expert_out, weights, shared, out, top)),
             (pairs + 2 * tokens) * h * elem, 2.0 * pairs * h)
        extra = {}
    print(json.dumps(dict({"kernel": "routed_experts", "dtype": args.dtype, "tokens": tokens, "hidden": h,
                           "inter": f, "experts": experts, "top": top, "groups": [args.groups, args.keep],
                           "experts_used": used, "error": int(error.item()), "peaks": peak["source"],
                           "kernels": rows}, **extra)))


def run_state_space(args, timer, dtype):
    """Every kernel between the two products of a state-space mixer for one prompt of --tokens
    tokens: --heads heads of --head-dim value columns over --state state rows, one group, four taps;
    and `lightning_scan` with one decay per head over as many state numbers (heads of 128 x 128), the
    like kernel of decaying linear attention.  ms, achieved rates, and the share of the measured copy
    rate (the scan: of the nominal 32-bit FMA peak, 4 flops per state number and token)."""
    g = torch.Generator(device="cuda").manual_seed(0)
    rand = lambda *shape: torch.randn(shape, generator=g, device="cuda", dtype=torch.float32)
    elem = 2 if dtype is torch.bfloat16 else 4
    tokens, heads, vdim, state, taps = args.tokens, args.heads, args.head_dim, args.state, 4
    inner, channels = heads * vdim, heads * vdim + 2 * state
    width = 2 * inner + 2 * state + heads
    proj = (rand(tokens, width) * 0.5).to(dtype)
    matrix = heads * state * vdim
    floats = -(-(matrix + (taps - 1) * channels) // 8) * 8
    slots = torch.zeros(1, floats, device="cuda")
    conv, conv_b = rand(channels, taps) * 0.5, rand(channels) * 0.1
    conv_by_tap = conv.t().contiguous()
    dt_bias, a_log, skip, gain = rand(heads), torch.linspace(-4.0, 0.5, heads, device="cuda"), rand(heads), rand(inner)
    dev = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    qstart, qlen, slot = dev([0]), dev([tokens]), dev([0])
    act = torch.empty(tokens, channels + inner, device="cuda")
    decay = torch.empty(tokens, heads, device="cuda")
    o = torch.empty(tokens, inner, device="cuda")
    y = torch.empty(tokens, inner, dtype=dtype, device="cuda")
    chunk = 64
    segs = -(-tokens // chunk)
    chunks = {}
    if tokens > 2 * chunk:
        chunks = dict(seg_item=dev([0] * segs), seg_row0=dev([i * chunk for i in range(segs)]), num_segs=segs,
                      seg_tokens=chunk, chunk_states=torch.empty(segs * (matrix + heads), device="cuda"))
    peak = peaks()
    ffma = 148 * 128 * 2 * 1.965e9 / 1e12
    rows = []

    def note(name, ms, nbytes, flops):
        gbs, tflops = nbytes / (ms * 1e-3) / 1e9, flops / (ms * 1e-3) / 1e12
        rows.append({"kernel": name, "ms": round(ms, 5), "GB/s": round(gbs, 1), "TFLOP/s": round(tflops, 2),
                     "frac_hbm": round(gbs / peak["hbm_gbs"], 3), "frac_ffma": round(tflops / ffma, 3)})

    note("ssd_prep", timer(lambda: ops.ssd_prep(proj, inner, inner + channels, qstart, qlen, slot, 1, slots, matrix,
                                                conv, conv_b, dt_bias, a_log, heads, vdim, act, decay,
                                                conv_wt=conv_by_tap)),
         tokens * ((channels + heads) * elem + (channels + inner + heads) * 4), 2.0 * tokens * channels * taps)
    note("ssd_tails", timer(lambda: ops.ssd_tails(proj, inner, channels, taps, qstart, qlen, slot, 1, slots, matrix)),
         2 * (taps - 1) * channels * 4, 0.0)
    scan_bytes = tokens * (inner + 2 * state + heads + inner) * 4 * (2 if chunks else 1)
    note("lightning_scan, decay per token", timer(lambda: ops.lightning_scan(
        act, inner + state, inner, channels, qstart, qlen, slot, 1, slots, None, o, heads, state, vdim,
        share=heads, decay_tok=decay, **chunks)), scan_bytes, 4.0 * tokens * matrix)
    note("ssd_gate_norm", timer(lambda: ops.ssd_gate_norm(o, act, proj, 0, skip, gain, y, vdim, 1, 1e-6)),
         tokens * inner * (8 + 2 * elem), 8.0 * tokens * inner)
    # the like kernel: one decay per head, heads of 128 x 128 over as many state numbers
    dim = 128
    like_heads = max(1, matrix // (dim * dim))
    like = rand(tokens, 3 * like_heads * dim)
    like_state = torch.zeros(1, like_heads, dim, dim, device="cuda")
    like_decay = torch.linspace(0.9, 0.999, like_heads, device="cuda")
    like_out = torch.empty(tokens, like_heads * dim, device="cuda")
    like_chunks = dict(chunks)
    if chunks:
        like_chunks["chunk_states"] = torch.empty(segs * like_heads * dim * dim, device="cuda")
    note("lightning_scan, decay per head", timer(lambda: ops.lightning_scan(
        like, 0, like_heads * dim, 2 * like_heads * dim, qstart, qlen, slot, 1, like_state, like_decay, like_out,
        like_heads, dim, dim, **like_chunks)),
         tokens * 4 * like_heads * dim * 4 * (2 if chunks else 1), 4.0 * tokens * like_heads * dim * dim)
    print(json.dumps({"kernel": "state_space", "dtype": args.dtype, "tokens": tokens, "heads": heads, "vdim": vdim,
                      "state": state, "taps": taps, "chunk_parallel": bool(chunks), "peaks": peak["source"],
                      "kernels": rows}))


def run_gated_linear(args, timer, dtype):
    """Every kernel of a gated linear attention mixer (--heads, --head-dim key columns, --vdim value columns, --rank)
    over one prompt of --tokens, or over --batch requests with one token each, beside the same scan with one
    decay per head at as many state numbers (heads of 128 x 128)."""
    heads, dim, vdim, rank = args.heads, args.head_dim, args.vdim, args.rank
    elem = 2 if dtype is torch.bfloat16 else 4
    items = args.batch if args.tokens == 1 else 1
    tokens = args.tokens * items
    g = torch.Generator(device="cuda").manual_seed(0)
    rand = lambda *shape: torch.randn(shape, generator=g, device="cuda", dtype=torch.float32)
    dev = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    qk, inner = heads * dim, heads * vdim
    proj = (rand(tokens, -(-(2 * qk + 2 * inner + rank) // 8) * 8) * 0.5).to(dtype)
    weight, bias, gain = rand(rank, qk) / rank ** 0.5, rand(qk), rand(vdim)
    decay, o = torch.empty(tokens, qk, device="cuda"), torch.empty(tokens, inner, device="cuda")
    y = torch.empty(tokens, inner, dtype=dtype, device="cuda")
    per = args.tokens
    qstart, qlen, slot = dev([i * per for i in range(items)]), dev([per] * items), dev(list(range(items)))
    chunk = 64
    segs = -(-per // chunk)

    def chunks(floats):
        if per <= 2 * chunk:
            return {}
        return dict(seg_item=dev([0] * segs), seg_row0=dev([i * chunk for i in range(segs)]), num_segs=segs,
                    seg_tokens=chunk, chunk_states=torch.empty(segs * floats, device="cuda"))
    peak, ffma, rows = peaks(), 148 * 128 * 2 * 1.965e9 / 1e12, []

    def note(name, ms, nbytes, flops):
        gbs, tflops = nbytes / (ms * 1e-3) / 1e9, flops / (ms * 1e-3) / 1e12
        rows.append({"kernel": name, "ms": round(ms, 5), "GB/s": round(gbs, 1), "TFLOP/s": round(tflops, 2),
                     "frac_hbm": round(gbs / peak["hbm_gbs"], 3), "frac_ffma": round(tflops / ffma, 3)})

    note("row_decay", timer(lambda: ops.row_decay(proj, 2 * qk + 2 * inner, rank, weight, bias, 1 / 16.0, decay)),
         tokens * (rank * elem + qk * 4), 2.0 * tokens * qk * rank)
    matrix = heads * dim * vdim
    state = torch.zeros(items, heads, dim, vdim, device="cuda")
    options = chunks(matrix + qk)
    carried = 2 * items * matrix * 4                         # the state in and out
    note("lightning_scan, decay per state row", timer(lambda: ops.lightning_scan(
        proj, 0, qk, 2 * qk, qstart, qlen, slot, items, state, None, o, heads, dim, vdim, decay_row=decay,
        out_scale=dim ** -0.5, **options)),
         tokens * ((2 * qk + inner) * elem + qk * 4 + inner * 4) * (2 if options else 1) + carried, 4.0 * tokens * matrix)
    note("head_norm_silu", timer(lambda: ops.head_norm_silu(o, proj, 2 * qk + inner, gain, 1e-6, y, heads)),
         tokens * inner * (4 + 2 * elem), 8.0 * tokens * inner)
    like_heads = max(1, matrix // (128 * 128))
    like, like_out = rand(tokens, 3 * like_heads * 128), torch.empty(tokens, like_heads * 128, device="cuda")
    like_state = torch.zeros(items, like_heads, 128, 128, device="cuda")
    like_decay = torch.linspace(0.9, 0.999, like_heads, device="cuda")
    options = chunks(like_heads * 128 * 128)
    note("lightning_scan, decay per head", timer(lambda: ops.lightning_scan(
        like, 0, like_heads * 128, 2 * like_heads * 128, qstart, qlen, slot, items, like_state, like_decay, like_out,
        like_heads, 128, 128, **options)),
         tokens * 4 * like_heads * 128 * 4 * (2 if options else 1) + 2 * items * like_heads * 128 * 128 * 4,
         4.0 * tokens * like_heads * 128 * 128)
    print(json.dumps({"kernel": "gated_linear", "dtype": args.dtype, "tokens": tokens, "requests": items, "heads": heads,
                      "dim": dim, "vdim": vdim, "rank": rank, "chunk_parallel": per > 2 * chunk, "peaks": peak["source"],
                      "kernels": rows}))


def run(args):
    timer = Timer(args.warmup, args.iters, not args.no_flush)
    dtype = torch.bfloat16 if args.dtype == "bfloat16" else torch.float32
    elem = 2 if dtype is torch.bfloat16 else 4
    extra = {}
    g = torch.Generator(device="cuda").manual_seed(0)
    rand = lambda *shape: torch.randn(shape, generator=g, device="cuda", dtype=torch.float32)
    if args.kernel in ("attention_decode", "attention_prefill"):
        ms, nbytes, flops, extra = run_attention(args, timer, args.kernel == "attention_decode")
    elif args.kernel == "add_rmsnorm":
        x, delta = rand(args.tokens, args.hidden), rand(args.tokens, args.hidden).to(dtype)
        gain, y = rand(args.hidden).to(dtype), torch.empty((args.tokens, args.hidden), dtype=dtype,
                                                           device="cuda")
        ms = timer(lambda: ops.add_rmsnorm(x, delta, gain, 1e-6, y))
        nbytes, flops = args.tokens * args.hidden * (8 + 2 * elem), 4.0 * args.tokens * args.hidden
    elif args.kernel == "swiglu":
        gu = rand(args.tokens, 2 * args.inter).to(dtype)
        act = torch.empty((args.tokens, args.inter), dtype=dtype, device="cuda")
        ms = timer(lambda: ops.swiglu(gu, act))
        nbytes, flops = 3 * args.tokens * args.inter * elem, 8.0 * args.tokens * args.inter
    elif args.kernel == "rope_kv_write":
        from ..parts.rope import rotary_table
        heads, kv_heads, hd, page = args.heads, args.kv_heads, args.head_dim, args.page
        qkv = rand(args.tokens, (heads + 2 * kv_heads) * hd).to(dtype)
        table = torch.from_numpy(rotary_table(1e6, hd, args.tokens + 1)).cuda()
        pages = torch.zeros((args.tokens // page + 1, 1, 2, kv_heads, page, hd), dtype=dtype,
                            device="cuda")
        pos = torch.arange(args.tokens, dtype=torch.int32, device="cuda")
        error = torch.zeros(1, dtype=torch.int32, device="cuda")
        ms = timer(lambda: ops.rope_kv_write(qkv, pos, table, pos, pages[:, 0, 0], pages[:, 0, 1],
                                             pages.stride(0), page, heads, kv_heads, hd, hd, error))
        nbytes = args.tokens * hd * elem * (2 * heads + 4 * kv_heads)
        flops = 6.0 * args.tokens * (heads + kv_heads) * hd
    elif args.kernel in ("argmax", "sample"):
        logits = rand(args.tokens, args.vocab)
        out = torch.empty(args.tokens, dtype=torch.int32, device="cuda")
        if args.kernel == "argmax":
            scratch = torch.empty(2 * args.tokens * ops.ARGMAX_PARTS, device="cuda")
            ms = timer(lambda: ops.argmax(logits, out, scratch))
        else:
            ones = torch.ones(args.tokens, device="cuda")
            k = torch.full((args.tokens,), args.top_k, dtype=torch.int32, device="cuda")
            u = torch.rand(args.tokens, generator=g, device="cuda")
            ms = timer(lambda: ops.sample(logits, ones * 0.8, k, ones * args.top_p, u, out))
        nbytes, flops = args.tokens * args.vocab * 4, float(args.tokens * args.vocab)
    elif args.kernel in ("gemm_decode", "gemm_decode_swiglu"):
        m, n, k = args.tokens, args.n, args.k
        swiglu = args.kernel == "gemm_decode_swiglu"
        x, w = rand(m, k).to(dtype), (rand(2 * n if swiglu else n, k) / math.sqrt(k)).to(dtype)
        weight = ops.DecodeWeight(w, swiglu=swiglu)
        out = torch.empty((m, n), dtype=dtype, device="cuda")
        error = torch.zeros(1, dtype=torch.int32, device="cuda")
        sms = torch.cuda.get_device_properties(0).multi_processor_count
        tiles = -(-n // (64 if swiglu else 128))
        splits = args.nsplit if args.nsplit > 0 else ops.gemm_decode_splits(tiles, k, sms)
        ms = timer(lambda: ops.gemm_decode(weight, x, out, None, error, splits))
        extra = {"splits": splits, "error": int(error.item())}
        nbytes, flops = (m * k + w.shape[0] * k + m * n) * elem, 2.0 * m * w.shape[0] * k
    elif args.kernel == "gemm_skinny":
        m, n, k = args.tokens, args.n, args.k
        x, w = rand(m, k).to(dtype), (rand(n, k) / math.sqrt(k)).to(dtype)
        out = torch.empty((m, n), dtype=dtype, device="cuda")
        ms = timer(lambda: ops.gemm_skinny(w, x, out, None))
        nbytes, flops = (m * k + n * k + m * n) * elem, 2.0 * m * n * k
    elif args.kernel in ("gemm_tiles", "gemm_tiles_swiglu"):
        m, n, k = args.tokens, args.n, args.k
        swiglu = args.kernel == "gemm_tiles_swiglu"
        # outputs of unit scale, as a layer sees them (the activation's exp stays in range)
        x, w = rand(m, k).to(dtype), (rand(2 * n if swiglu else n, k) / math.sqrt(k)).to(dtype)
        weight = ops.TiledWeight(w, swiglu=swiglu)
        out = torch.empty((m, n), dtype=dtype, device="cuda")
        error = torch.zeros(1, dtype=torch.int32, device="cuda")
        sms = torch.cuda.get_device_properties(0).multi_processor_count
        floats, ints = (0, 0) if args.variant == "whole_tiles" else \
            ops.gemm_tiles_workspace(m, n, k, swiglu, sms)
        workspace = torch.empty(floats, dtype=torch.float32, device="cuda") if floats else None
        counters = torch.zeros(max(ints, 1), dtype=torch.int32, device="cuda") if floats else None
        ms = timer(lambda: ops.gemm_tiles(weight, x, out, None, error, sms, workspace, counters))
        extra = {"error": int(error.item()), "workspace_floats": floats,
                 "counters_left": int(counters.abs().sum().item()) if floats else 0}
        nbytes, flops = (m * k + w.shape[0] * k + m * n) * elem, 2.0 * m * w.shape[0] * k
    elif args.kernel in ("linear", "gemm_f32"):
        m, n, k = args.tokens, args.n, args.k
        if args.kernel == "linear":
            x, w = rand(m, k).to(dtype), rand(n, k).to(dtype)
            ms = timer(lambda: torch.nn.functional.linear(x, w))
        else:
            x, w = rand(m, k), rand(n, k)
            ms = timer(lambda: ops.gemm_f32(x, w, None, kind=args.f32_kind, rows_per_warp=args.f32_rows_per_warp))
            elem = 4
            extra = {"frac_ffma": round(2.0 * m * n * k / (ms * 1e-3) / 74.4e12, 3), "f32_kind": args.f32_kind}
        nbytes, flops = (m * k + n * k + m * n) * elem, 2.0 * m * n * k
    elif args.kernel == "routed_experts":
        return run_routed_experts(args, timer, dtype)
    elif args.kernel == "state_space":
        return run_state_space(args, timer, dtype)
    elif args.kernel == "gated_linear":
        return run_gated_linear(args, timer, dtype)
    elif args.kernel == "norm_rotate_write":
        from ..parts.rope import rotary_table
        heads, kv_heads, hd, page = args.heads, args.kv_heads, args.head_dim, args.page
        own = 0 if args.keys_as_values else kv_heads * hd
        qkv = rand(args.tokens, (heads + kv_heads) * hd + own + -(-heads // 8) * 8).to(dtype)
        table = torch.from_numpy(rotary_table(1e6, hd // 2, args.tokens + 1)).cuda()
        pages = torch.zeros((args.tokens // page + 1, 1, 2, kv_heads, page, hd), dtype=dtype, device="cuda")
        pos = torch.arange(args.tokens, dtype=torch.int32, device="cuda")
        error = torch.zeros(1, dtype=torch.int32, device="cuda")
        q_gain, k_gain = (rand(heads * hd), rand(kv_heads * hd)) if args.whole_norm else (rand(hd), rand(hd))
        ms = timer(lambda: ops.norm_rotate_write(qkv, pos, table, pos, pages[:, 0, 0], pages[:, 0, 1], pages.stride(0), page,
                                                 heads, kv_heads, hd, hd, hd // 2, q_gain, k_gain, 1e-6, error,
                                                 whole=args.whole_norm, values_from_keys=args.keys_as_values))
        nbytes = args.tokens * elem * (2 * heads * hd + 3 * kv_heads * hd + own)
        flops = 10.0 * args.tokens * (heads + kv_heads) * hd
    elif args.kernel == "scaled_attention":
        ms, nbytes, flops, extra = run_scaled_attention(args, timer)
    elif args.kernel == "stream_norm":
        s = args.streams
        x, y = rand(args.tokens, s, args.hidden), rand(args.tokens, args.hidden).to(dtype)
        mix, spread, gather = torch.eye(s, device="cuda") + 0.01 * rand(s, s), rand(s) * 0.1, rand(s)
        gain, bias = rand(args.hidden), rand(args.hidden)
        out = torch.empty((args.tokens, args.hidden), dtype=dtype, device="cuda")
        scale = rand(args.hidden) if args.scaled else None
        ms = timer(lambda: ops.stream_norm(x, None, y, mix, spread, gather, gain, None if args.scaled else bias, 1e-6, out,
                                           centred=not args.scaled, delta_scale=scale))
        nbytes, flops = args.tokens * args.hidden * (8 * s + 2 * elem), 2.0 * args.tokens * args.hidden * s * (s + 2)
    elif args.kernel == "sum_layernorm":
        x, d1, d2 = rand(args.tokens, args.hidden), rand(args.tokens, args.hidden).to(dtype), \
            rand(args.tokens, args.hidden).to(dtype)
        gain, bias = rand(args.hidden), rand(args.hidden)
        y = torch.empty((args.tokens, args.hidden), dtype=dtype, device="cuda")
        ms = timer(lambda: ops.sum_layernorm(x, [d1, d2], gain, bias, 1e-6, y))
        nbytes, flops = args.tokens * args.hidden * (8 + 3 * elem), 8.0 * args.tokens * args.hidden
    else:
        raise SystemExit(f"unknown kernel {args.kernel}")
    peak = peaks()
    gbs, tflops = nbytes / (ms * 1e-3) / 1e9, flops / (ms * 1e-3) / 1e12
    record = {"kernel": args.kernel, "dtype": args.dtype, "ms": round(ms, 5), "bytes": int(nbytes),
              "flops": flops, "GB/s": round(gbs, 1), "TFLOP/s": round(tflops, 2),
              "frac_hbm": round(gbs / peak["hbm_gbs"], 3),
              "frac_bf16": round(tflops / peak["bf16_tflops"], 3), "peaks": peak["source"],
              "sizes": {k: v for k, v in vars(args).items()
                        if k not in ("kernel", "dtype", "warmup", "iters", "no_flush", "f32_kind", "f32_rows_per_warp")}}
    record.update(extra)
    print(json.dumps(record))


def main(argv=None) -> int:
    parser = argparse.ArgumentParser(description=__doc__,
                                     formatter_class=argparse.RawDescriptionHelpFormatter)
    parser.add_argument("kernel")
    parser.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--context", type=int, default=4096)
    parser.add_argument("--tokens", type=int, default=2048)
    parser.add_argument("--heads", type=int, default=28)
    parser.add_argument("--kv-heads", type=int, default=4)
    parser.add_argument("--head-dim", type=int, default=128)
    parser.add_argument("--page", type=int, default=16)
    parser.add_argument("--hidden", type=int, default=3584)
    parser.add_argument("--inter", type=int, default=18944)
    parser.add_argument("--vocab", type=int, default=152064)
    parser.add_argument("--n", type=int, default=37888)
    parser.add_argument("--k", type=int, default=3584)
    parser.add_argument("--nsplit", type=int, default=0, help="0 = the engine's choice")
    parser.add_argument("--state", type=int, default=128, help="state_space: state rows per head")
    parser.add_argument("--streams", type=int, default=4, help="stream_norm: residual streams")
    parser.add_argument("--chunk", type=int, default=0, help="scaled_attention: positions per chunk (0: none)")
    parser.add_argument("--softcap", type=float, default=0.0, help="scaled_attention: cap on the scores (0: none)")
    parser.add_argument("--gate", action="store_true", help="scaled_attention: a gate per column")
    parser.add_argument("--head-gate", action="store_true", help="scaled_attention: a gate per head")
    parser.add_argument("--sink", action="store_true", help="scaled_attention: a sink per head")
    parser.add_argument("--window", type=int, default=0, help="scaled_attention: keys a query sees (0: all)")
    parser.add_argument("--maps", type=int, default=1, choices=[1, 2],
                        help="scaled_attention: 2 = two keys of half the head size, with the merge of differences")
    parser.add_argument("--vdim", type=int, default=128, help="gated_linear: value columns per head")
    parser.add_argument("--rank", type=int, default=16, help="gated_linear: width of the narrow product of the decays")
    parser.add_argument("--whole-norm", action="store_true", help="norm_rotate_write: the norm over all heads at once")
    parser.add_argument("--keys-as-values", action="store_true", help="norm_rotate_write: values are the keys as projected")
    parser.add_argument("--scaled", action="store_true", help="stream_norm: outputs scaled by column, RMS norm")
    parser.add_argument("--experts", type=int, default=64)
    parser.add_argument("--top", type=int, default=6)
    parser.add_argument("--groups", type=int, default=8)
    parser.add_argument("--keep", type=int, default=4)
    parser.add_argument("--no-grouped", action="store_true",
                        help="routed_experts: tiles of 64 rows also where the grouped products would run")
    parser.add_argument("--variant", default="mma", choices=["mma", "tc", "rows16", "whole_tiles"],
                        help="bfloat16 attention: mma.sync with cp.async loads, or tcgen05; float32 "
                             "attention: rows16 takes the kernel for tiles of up to 16 rows; gemm_tiles: "
                             "whole_tiles leaves a partial last round of tiles to the pairs it falls to")
    parser.add_argument("--f32-kind", default="auto", choices=["auto", "rows", "tiles", "plain"],
                        help="gemm_f32: which of the float32 kernels (frac_ffma is of the nominal "
                             "74.4 TFLOP/s: 148 SMs x 128 lanes x 2 x 1.965 GHz)")
    parser.add_argument("--f32-rows-per-warp", type=int, default=0, choices=[0, 1, 2, 4])
    parser.add_argument("--top-k", type=int, default=0)
    parser.add_argument("--top-p", type=float, default=1.0)
    parser.add_argument("--warmup", type=int, default=3)
    parser.add_argument("--iters", type=int, default=20)
    parser.add_argument("--no-flush", action="store_true")
    args = parser.parse_args(argv)
    run(args)
    return 0


if __name__ == "__main__":
    sys.exit(main())
