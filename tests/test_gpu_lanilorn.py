"""The Lanilorn design in the engine against the plain implementation of the tests: every mechanism
alone, whole prompts against decoding token by token, portions down to two tokens, mixed batches with
pages and slots that are used again, keys far away, at page borders and on either side of a window's
edge in prompts and in decoding, the first tokens of a sequence, long decoding, and greedy generation
through the engine."""

import math

import numpy as np
import pytest
import torch

import helpers
import lanilorn_models as lm
import plain_lanilorn as plain

pytestmark = pytest.mark.gpu

F32_BOUND = 2e-4          # largest |engine - plain| of a row, relative to max(1, largest |plain|)
BF16_BOUND = 3e-2
# float32 runs the sharpened models (every mechanism far out in the logits); bfloat16 runs gentle ones, in
# which a rounding in one layer is not blown up by the next
SHARPEN = {"float32": True, "bfloat16": False}

_folders = {}
_plain = {}


def folder_of(tmp_path_factory, name, dtype="float32"):
    key = (name, SHARPEN[dtype])
    if key not in _folders:
        _folders[key] = lm.write_model(tmp_path_factory.mktemp(f"lanilorn_{name}"), name, sharpen=SHARPEN[dtype])
    return _folders[key]


def plain_rows(folder, ids):
    key = (str(folder), tuple(ids))
    if key not in _plain:
        _plain[key] = plain.logits_for(folder, ids)
    return _plain[key]


def runner_for(folder, dtype, num_pages, max_requests=4, page_size=16, **options):
    from from_scratch_inference_engine_b200 import LoadedModel, ModelRunner
    model = LoadedModel.from_pretrained(folder, dtype=dtype, max_positions=num_pages * page_size)
    return ModelRunner(model.model, model.runtime, page_size=page_size, num_pages=num_pages,
                       max_requests=max_requests, max_step_tokens=num_pages * page_size, **options)


def assert_rows(rows, requests, folder, bound):
    """Every row within `bound` of the plain logits.  bfloat16 rounds every product's result:
    there one row in ten may lie beyond the bound, none beyond three times it."""
    assert rows
    beyond = 0
    for (key, pos), row in sorted(rows.items()):
        want = plain_rows(folder, requests[key.split("~")[0]])[pos]
        base = max(1.0, float(np.abs(want).max()))
        diff = float(np.abs(row.astype(np.float64) - want).max())
        limit = bound * base * (3.0 if bound == BF16_BOUND else 1.0)
        assert diff <= limit, f"request {key} position {pos}: off by {diff:.3e} (bound {limit:.3e})"
        beyond += diff > bound * base
    assert beyond <= 0.1 * len(rows), f"{beyond} of {len(rows)} rows beyond the bound"


def vocab_of(name):
    return lm.CONFIGS[name]["vocab"]


def dev(values, dtype=torch.int32):
    return torch.tensor(values, dtype=dtype, device="cuda")


# ----------------------------------------------------------------- mechanisms, kernel by kernel
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams,width", [(1, 37), (2, 256), (4, 1000), (9, 100)])
def test_outputs_are_scaled_column_by_column_as_they_settle(dtype, streams, width):
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(streams + width)
    rand = lambda *shape: torch.randn(shape, generator=g)
    tokens, eps = 6, 1e-3
    held, delta, scale = rand(tokens, streams, width), rand(tokens, width).to(dtype), rand(width)
    mix, spread, gather, gain = rand(streams, streams), rand(streams), rand(streams), rand(width)
    parts = plain.spread_streams([held[:, s].double() for s in range(streams)], mix.double(), spread.double(),
                                 delta.double() * scale.double())
    want = plain.rms_norm(plain.gather_streams(parts, gather.double()), gain.double(), eps)
    x, out = held.clone().cuda(), torch.zeros(tokens, width, device="cuda", dtype=dtype)
    ops.stream_norm(x, None, delta.cuda(), mix.cuda(), spread.cuda(), gather.cuda(), gain.cuda(), None, eps, out,
                    centred=False, delta_scale=scale.cuda())
    tolerance = 5e-5 if dtype is torch.float32 else 2e-2
    assert (x.cpu().double() - torch.stack(parts, 1)).abs().max() < 1e-5 * max(1.0, float(held.abs().max()) * streams)
    assert (out.cpu().double() - want).abs().max() < tolerance * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,whole,from_keys,gains", [
    (6, 2, 16, 16, 8, True, True, True), (3, 1, 12, 12, 6, True, True, True), (4, 4, 64, 64, 64, True, True, True),
    (40, 8, 128, 128, 64, True, True, True), (3, 3, 8, 24, 0, False, False, False), (5, 1, 24, 16, 16, False, False, True),
    (2, 2, 40, 40, 32, False, True, True), (7, 1, 64, 128, 0, True, False, True), (3, 2, 16, 16, 16, False, False, False)])
def test_norm_over_the_projection_and_values_that_are_the_keys(dtype, heads, kv_heads, dim, vdim, dims, whole, from_keys,
                                                               gains):
    """q in place, k and v into the token's slot: the norm over all heads at once or head by head, with and
    without gains, values of their own or the keys as they were projected; sizes that fit the vector form and
    sizes that do not; columns behind are left alone; a token without a slot stores nothing."""
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(heads * dim)
    page, eps, tokens, pages = 4, 1e-2, 9, 8
    width = (heads + kv_heads) * dim + (0 if from_keys else kv_heads * vdim)
    extra = 8 if width % 8 == 0 else 5
    proj = (torch.randn(tokens, width + extra, generator=g) * 0.7).to(dtype)
    positions = torch.tensor([0, 3, 1, 20, 7, 9, 11, 31, 2], dtype=torch.int32)
    slots = torch.tensor([7, 2, 30, 12, 5, 21, -1, 0, 19], dtype=torch.int32)
    rot = lm.yarn(1000.0, dims, 3.0, 16, 4.0, 0.5) if dims else None
    freq, magnitude = plain.yarn_frequencies(rot) if rot else ([], 1.0)
    angles = torch.arange(32)[:, None].double() * torch.tensor(freq, dtype=torch.float64)[None]
    table = (torch.cat([angles.cos(), angles.sin()], 1) * magnitude).float().contiguous().cuda()
    q_gain = torch.rand(heads * dim if whole else dim, generator=g) + 0.5 if gains else None
    k_gain = torch.rand(kv_heads * dim if whole else dim, generator=g) + 0.5 if gains else None
    both = torch.zeros(pages, kv_heads * page * (dim + vdim), device="cuda", dtype=dtype)
    k_pages, v_pages = both[:, :kv_heads * page * dim], both[:, kv_heads * page * dim:]
    work, error = proj.clone().cuda(), torch.zeros(1, dtype=torch.int32, device="cuda")
    c = lambda t: None if t is None else t.cuda()
    ops.norm_rotate_write(work, positions.cuda(), table, slots.cuda(), k_pages, v_pages, both.stride(0), page, heads,
                          kv_heads, dim, vdim, dims, c(q_gain), c(k_gain), eps, error, whole=whole,
                          values_from_keys=from_keys)
    assert int(error.item()) == 0
    q, k = proj[:, :heads * dim].double(), proj[:, heads * dim:(heads + kv_heads) * dim].double()
    v = (k if from_keys else proj[:, (heads + kv_heads) * dim:width].double()).view(tokens, kv_heads, vdim)
    if gains and whole:
        q, k = plain.rms_norm(q, q_gain.double(), eps), plain.rms_norm(k, k_gain.double(), eps)
    q, k = q.view(tokens, heads, dim), k.view(tokens, kv_heads, dim)
    if gains and not whole:
        q, k = plain.rms_norm(q, q_gain.double(), eps), plain.rms_norm(k, k_gain.double(), eps)
    q, k = plain.rotate(q, rot, positions.tolist()), plain.rotate(k, rot, positions.tolist())
    tolerance = 2e-5 if dtype is torch.float32 else 3e-2
    assert (work[:, :heads * dim].cpu().double().view(tokens, heads, dim) - q).abs().max() < tolerance * float(q.abs().max())
    assert torch.equal(work[:, width:].cpu(), proj[:, width:])
    kp = k_pages.cpu().double().reshape(pages, kv_heads, page, dim)
    vp = v_pages.cpu().double().reshape(pages, kv_heads, page, vdim)
    for t, slot in enumerate(slots.tolist()):
        if slot < 0:
            continue
        assert (kp[slot // page, :, slot % page] - k[t]).abs().max() < tolerance * float(k.abs().max())
        assert torch.equal(vp[slot // page, :, slot % page], v[t])           # as projected, not a rounding more
    assert float(kp.abs().sum(dim=(1, 3)).ne(0).sum()) == 8                  # one token had no slot: nothing stored


def _paged(rows, page_size, order, pages_total):
    """rows [n, kv_heads, width] laid out as pages [kv_head][slot][width] at the given page ids."""
    n, kv_heads, width = rows.shape
    pages = torch.zeros(pages_total, kv_heads, page_size, width, dtype=rows.dtype)
    table = []
    for b in range(-(-n // page_size)):
        part = rows[b * page_size:(b + 1) * page_size]
        pages[order[b], :, :part.shape[0]] = part.transpose(0, 1)
        table.append(order[b])
    return pages, table


class Attention:
    """Requests of (cached, new) tokens over shuffled pages of two entries (the second one is read), and the
    plain result: `maps` keys side by side in a key row `dk` wide, a window, sinks, a factor on the scores by the
    query's position, a gate per head.  Some queries point at the first key of their window while the key
    before it would win if it were seen."""

    def __init__(self, lengths, heads, kv_heads, dk, dv, page, dtype, scale, window=0, sinks=False, temperature=None,
                 gated=False, maps=1, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.lengths, self.heads, self.kv_heads, self.dk, self.dv, self.page = lengths, heads, kv_heads, dk, dv, page
        self.dtype, self.window, self.maps = dtype, window, maps
        group, dim = heads // kv_heads, dk // maps
        total = sum(-(-(a + b) // page) for a, b in lengths) + 3
        order = torch.randperm(total, generator=g).tolist()
        keys, values = torch.zeros(total, kv_heads, page, dk, dtype=dtype), torch.zeros(total, kv_heads, page, dv, dtype=dtype)
        self.sink = (torch.rand(heads, generator=g) * 4 - 1) if sinks else None
        longest = max(a + b for a, b in lengths)
        factors = plain.query_temperature(longest, temperature)
        gate = torch.randn(sum(b for _, b in lengths), heads, generator=g).to(dtype) if gated else None
        tables, qs, want, used, at = [], [], [], 0, 0
        for cached, new in lengths:
            n = cached + new
            k = plain.unit_rms(torch.randn(n, kv_heads, maps, dim, generator=g).double(), 0.0).float()
            q = plain.unit_rms(torch.randn(new, heads, maps, dim, generator=g).double(), 0.0).float()
            for qi in sorted({0, new // 3, new - 1}):
                i = cached + qi
                first = max(0, i - window + 1) if window else 0
                q[qi] = k[first, :, None].expand(kv_heads, group, maps, dim).reshape(heads, maps, dim)
                if first > 0:
                    k[first - 1] = k[first] * 1.1                     # outside: it would win if it were seen
            q, k = q.to(dtype), k.to(dtype)
            v = torch.randn(n, kv_heads, dv, generator=g).to(dtype)
            blocks = -(-n // page)
            kp, table = _paged(k.reshape(n, kv_heads, dk), page, order[used:used + blocks], total)
            vp, _ = _paged(v, page, order[used:used + blocks], total)
            used += blocks
            keys += kp
            values += vp
            tables.append(table)
            qs.append(q.reshape(new, -1))
            mask = (plain.window_mask(n, window) if window else plain.causal_mask(n))[cached:]
            qd = q.double() * factors[cached:n, None, None, None]
            out = torch.stack([plain.sink_attention(qd[:, :, m], k[:, :, m].double(), v.double(), mask, scale,
                                                    None if self.sink is None else self.sink.double())
                               for m in range(maps)], dim=2)                   # [new, heads, maps, dv]
            if gated and maps == 1:
                out = out * torch.sigmoid(gate[at:at + new].double())[:, :, None, None]
            at += new
            want.append(out)
        self.want = torch.cat(want)
        self.tokens = self.want.shape[0]
        self.tables = torch.full((len(lengths), max(len(t) for t in tables)), -1, dtype=torch.int32)
        for i, t in enumerate(tables):
            self.tables[i, :len(t)] = torch.tensor(t, dtype=torch.int32)
        self.tables = self.tables.cuda()
        # q and the gate as columns of one wider tensor, as the engine's product leaves them
        wide = torch.zeros(self.tokens, heads * dk + 16 + -(-heads // 8) * 8, dtype=dtype)
        wide[:, :heads * dk] = torch.cat(qs)
        if gated:
            wide[:, heads * dk + 16:heads * dk + 16 + heads] = gate
        self.q = wide.cuda()
        self.gate = self.q[:, heads * dk + 16:heads * dk + 16 + heads] if gated else None
        self.keys, self.values = keys, values
        self.scale = torch.full((heads * maps,), scale, dtype=torch.float32, device="cuda")
        self.factors = None if temperature is None else factors.float().cuda()
        starts = np.cumsum([0] + [b for _, b in lengths])
        self.qstart, self.qlen = dev(starts[:-1].tolist()), dev([b for _, b in lengths])
        self.pos0, self.slots = dev([a for a, _ in lengths]), dev(list(range(len(lengths))))

    def tiles(self, rows, only):
        item, row0, toks, at = [], [], [], 0
        for i, (_, new) in enumerate(self.lengths):
            if i in only:
                for r in range(0, new * (self.heads * self.maps // self.kv_heads), rows):
                    item.append(i)
                    row0.append(r)
                toks += range(at, at + new)
            at += new
        return dev(item), dev(row0), len(item), dev(toks), len(toks)

    def forms(self):
        forms = ["plain"]
        if self.dtype is torch.bfloat16 and self.dk % 16 == 0 and self.dv in (32, 64, 96, 128, 192, 256):
            forms += ["mma", "mma_few"] + (["mma_split"] if self.dv % 64 == 0 else [])
            if self.dk == self.dv and self.dk in (64, 128) and self.maps <= 2:
                forms.append("tcgen05")
        return forms

    def launch(self, form, nsplit, only, partial=False):
        from from_scratch_inference_engine_b200.kernels import ops
        heads = self.heads * self.maps
        out = torch.full((self.tokens, heads * self.dv), 7.0, device="cuda", dtype=self.dtype)
        error = torch.zeros(1, dtype=torch.int32, device="cuda")
        part_o = torch.full((nsplit * self.tokens * heads * self.dv,), float("nan"), device="cuda")
        part_ml = torch.full((nsplit * self.tokens * heads * 2,), float("nan"), device="cuda")
        options = dict(head_gate=None if self.maps > 1 else self.gate, pos_scale=self.factors, maps=self.maps,
                       sink=None if self.sink is None else self.sink.cuda(), partial=partial)
        q_ld = self.q.stride(0)
        if form == "tcgen05":
            pages = torch.randn(self.keys.shape[0], 2, 2, *self.keys.shape[1:]).to(self.dtype)
            pages[:, 1, 0], pages[:, 1, 1] = self.keys, self.values
            item, row0, count, toks, n = self.tiles(ops.ATTENTION_TC_ROWS, only)
            ops.attention_tc_scaled(ops.PagesMap(pages.cuda()), 1, self.q, q_ld, self.scale, self.tables, item, row0, count,
                                    self.qstart, self.qlen, self.pos0, out, self.tokens, heads, self.kv_heads, self.window,
                                    error, nsplit, part_o, part_ml, combine_tokens=toks, num_combine=n, **options)
        else:
            both = torch.cat([self.keys.flatten(1), self.values.flatten(1)], dim=1).cuda()
            split = self.keys[0].numel()
            item, row0, count, toks, n = self.tiles(ops.scaled_attention_rows(self.dtype, self.dk, self.dv, False, form), only)
            ops.scaled_attention(self.q, q_ld, self.scale, both[:, :split], both[:, split:], both.stride(0), self.page,
                                 self.dk, self.dv, False, self.tables, item, row0, count, self.qstart, self.qlen,
                                 self.pos0, self.slots, out, self.tokens, heads, self.kv_heads, self.window, error,
                                 nsplit, part_o, part_ml, form=form, combine_tokens=toks, num_combine=n, **options)
        assert int(error.item()) == 0
        return out, part_o, part_ml, toks, n

    def run(self, form, nsplit, only=None):
        """[tokens, heads, dv]; `only`: the requests that the tiles hold."""
        out, _, _, toks, _ = self.launch(form, nsplit, range(len(self.lengths)) if only is None else only)
        return out.cpu().double().reshape(self.tokens, self.heads, self.dv), toks.cpu().long()

    def run_difference(self, form, nsplit, weight, eps, factor, only=None):
        from from_scratch_inference_engine_b200.kernels import ops
        untouched, part_o, part_ml, toks, n = self.launch(form, nsplit, range(len(self.lengths)) if only is None else only,
                                                          partial=True)
        assert (untouched == 7.0).all()
        out = torch.full((self.tokens, self.heads * self.dv), 7.0, device="cuda", dtype=self.dtype)
        ops.difference_merge(part_o, part_ml, out, self.tokens, self.heads, self.dv, nsplit, weight, eps, factor,
                             self.gate, None if only is None else toks, n)
        return out.cpu().double().reshape(self.tokens, self.heads, self.dv), toks.cpu().long()


LENGTHS = [(300, 177), (0, 90), (40, 2), (260, 1)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,heads,kv_heads,window,page", [
    (24, 6, 2, 37, 16), (96, 4, 1, 50, 8), (32, 6, 6, 1, 16), (64, 8, 2, 100, 32), (128, 6, 3, 129, 16), (128, 10, 1, 0, 16)])
def test_windows_sinks_and_gates_per_head(dtype, dim, heads, kv_heads, window, page):
    """Every form of the attention kernel that takes the sizes, whole and split over key ranges: a long
    portion behind 300 cached tokens, a first portion, two tokens behind 40, a token decoded at position
    260; the sinks count once whatever the number of ranges."""
    case = Attention(LENGTHS, heads, kv_heads, dim, dim, page, dtype, 2.0 / dim ** 0.5, window, sinks=True, gated=True,
                     seed=dim + heads)
    tolerance = 1e-4 if dtype is torch.float32 else 2e-2
    for form in case.forms():
        for nsplit in (1, 3, 34):
            got, _ = case.run(form, nsplit)
            assert (got - case.want[:, :, 0]).abs().max() < tolerance * max(1.0, float(case.want.abs().max())), (form, nsplit)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,dv,heads,kv_heads,page", [
    (12, 20, 4, 2, 16), (7, 5, 3, 1, 16), (48, 96, 6, 2, 8), (16, 32, 6, 3, 16), (32, 64, 8, 2, 16), (64, 128, 4, 1, 32),
    (64, 128, 4, 4, 16), (48, 192, 2, 2, 16), (8, 400, 2, 1, 16)])
def test_the_difference_of_two_maps(dtype, dim, dv, heads, kv_heads, page):
    """Every form of the attention over two keys side by side, its ranges merged, subtracted, normed and gated:
    the same requests; every token's queries with a factor of their own."""
    case = Attention(LENGTHS, heads, kv_heads, 2 * dim, dv, page, dtype, 1.5 / dim ** 0.5,
                     temperature={"coef": 0.3, "every": 9}, gated=True, maps=2, seed=dim + dv)
    weight, eps, factor = 0.7, 1e-3, 0.6
    want = plain.difference(case.want[:, :, 0], case.want[:, :, 1], weight, 1 - factor, eps)
    want = want * torch.sigmoid(case.gate.cpu().double())[:, :, None]
    tolerance = 2e-4 if dtype is torch.float32 else 2e-2
    for form in case.forms():
        for nsplit in (1, 3, 34):
            got, _ = case.run_difference(form, nsplit, weight, eps, factor)
            assert (got - want).abs().max() < tolerance * max(1.0, float(want.abs().max())), (form, nsplit)


def test_split_ranges_of_listed_tokens_only():
    """Tiles of some requests, split over key ranges and merged for their tokens: the other requests' rows
    stay as they were (another launch of the step fills them)."""
    lengths = [(90, 200), (333, 1), (0, 150), (251, 1)]
    sunk = Attention(lengths, 4, 2, 64, 64, 16, torch.bfloat16, 0.3, 70, sinks=True, gated=True, seed=5)
    apart = Attention(lengths, 4, 2, 64, 64, 16, torch.bfloat16, 0.3, gated=True, maps=2, seed=6)
    want = plain.difference(apart.want[:, :, 0], apart.want[:, :, 1], 0.4, 0.2, 1e-5) * \
        torch.sigmoid(apart.gate.cpu().double())[:, :, None]
    for form, only in (("tcgen05", (0, 2)), ("auto", (1, 3)), ("plain", (1, 3)), ("mma_few", (1, 3))):
        for got, toks, right in ((*sunk.run(form, 3, only), sunk.want[:, :, 0]),
                                 (*apart.run_difference(form, 3, 0.4, 1e-5, 0.8, only), want)):
            assert (got[toks] - right[toks]).abs().max() < 2e-2 * max(1.0, float(right.abs().max()))
            rest = torch.ones(right.shape[0], dtype=torch.bool)
            rest[toks] = False
            assert (got[rest] == 7.0).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank,columns,tokens", [(1, 5, 3), (16, 256, 33), (5, 130, 16), (64, 1024, 50)])
def test_decays_through_their_logarithms(dtype, rank, columns, tokens):
    """sigmoid(z)^(1 / tau), with biases so large that the sigmoid itself is 1 or 0 in 32-bit."""
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(rank)
    proj = torch.randn(tokens, rank + 7, generator=g).to(dtype)
    w, bias = torch.randn(columns, rank, generator=g) / rank ** 0.5, torch.randn(columns, generator=g)
    bias[0], bias[1], bias[2] = 95.0, -60.0, -300.0
    for tau in (1.0, 16.0):
        out = torch.empty(tokens, columns, device="cuda")
        ops.row_decay(proj.cuda(), 4, rank, w.t().contiguous().cuda(), bias.cuda(), 1.0 / tau, out)
        want = plain.key_decays(proj[:, 4:4 + rank].double(), {"a1": torch.eye(rank).double(), "a2": w.double(),
                                                               "a2.b": bias.double()}, "", tau)
        assert (out.cpu().double() - want).abs().max() < 2e-6
        assert torch.isfinite(out).all()
        for column in (1, 2) if tau > 1 else (1,):
            assert (out[:, column].cpu().double() / want[:, column] - 1).abs().max() < 1e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim", [(3, 10, 14), (3, 32, 40), (1, 64, 128), (2, 100, 36), (2, 200, 20), (1, 256, 64)])
def test_scan_with_a_decay_per_state_row(dtype, heads, dim, vdim):
    """Two requests' tokens as one batch - in one call, in three that carry the state, and chunk by
    chunk - against the recurrence token by token; slots in another order than the requests, one slot
    untouched."""
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(dim + vdim)
    lengths, slots = [150, 71], [2, 0]
    width = 2 * heads * dim + heads * vdim
    proj = torch.randn(sum(lengths), width + 3 * (dim % 4 != 0) + 8, generator=g).to(dtype)
    decay = torch.rand(sum(lengths), heads * dim, generator=g) ** 0.2
    decay[:, 0], decay[5:9, 1] = 1.0, 0.0                # a row that keeps everything, one that forgets at once
    start = torch.randn(3, heads, dim, vdim, generator=g)
    scale = dim ** -0.5
    want, state, at = [], start.double().clone(), 0
    for n, slot in zip(lengths, slots):
        rows = proj[at:at + n].double()
        q, k = rows[:, :heads * dim].reshape(n, heads, dim), rows[:, heads * dim:2 * heads * dim].reshape(n, heads, dim)
        v = rows[:, 2 * heads * dim:width].reshape(n, heads, vdim)
        a = decay[at:at + n].double().reshape(n, heads, dim)
        want.append(plain.decayed_recurrence(q * scale, k, v, a, state[slot].clone()).reshape(n, -1))
        s = state[slot]
        for t in range(n):
            s = a[t][:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
        state[slot] = s
        at += n
    want = torch.cat(want)

    def run(cuts, chunked):
        held = start.clone().cuda()
        rows, begin = torch.zeros(sum(lengths), heads * vdim), [0, 0]
        for cut in cuts:
            take = [list(range(sum(lengths[:i]) + begin[i], sum(lengths[:i]) + min(lengths[i], cut[i]))) for i in range(2)]
            begin = [min(lengths[i], cut[i]) for i in range(2)]
            index = torch.tensor(take[0] + take[1])
            counts = [len(t) for t in take]
            segments = {}
            if chunked:
                seg = [(i, r) for i in range(2) for r in range(0, counts[i], 64)]
                segments = dict(seg_item=dev([s[0] for s in seg]), seg_row0=dev([s[1] for s in seg]), num_segs=len(seg),
                                seg_tokens=64, chunk_states=torch.full((len(seg) * heads * dim * (vdim + 1),), float("nan"),
                                                                       device="cuda"))
            out = torch.zeros(len(index), heads * vdim, device="cuda")
            ops.lightning_scan(proj[index].cuda(), 0, heads * dim, 2 * heads * dim, dev([0, counts[0]]), dev(counts),
                               dev(slots), 2, held, None, out, heads, dim, vdim, decay_row=decay[index].cuda(),
                               out_scale=scale, **segments)
            rows[index] = out.cpu()
        return rows, held
    for cuts, chunked in (([(150, 71)], False), ([(40, 3), (41, 70), (150, 71)], False), ([(150, 71)], True),
                          ([(70, 65), (150, 71)], True)):
        rows, held = run(cuts, chunked)
        assert (rows.double() - want).abs().max() < 2e-5 * float(want.abs().max()), (cuts, chunked)
        assert (held.cpu().double() - state).abs().max() < 2e-5 * float(state.abs().max())
        assert torch.equal(held[1].cpu(), start[1])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_of_every_head_times_its_gate(dtype):
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(8)
    for heads, vdim, before in ((3, 10, 5), (4, 64, 8), (1, 200, 16), (5, 128, 4)):
        o, gain = torch.randn(7, heads * vdim, generator=g) * 3, torch.rand(vdim, generator=g) + 0.5
        proj = torch.randn(7, before + heads * vdim + 4, generator=g).to(dtype)
        out = torch.empty(7, heads * vdim, device="cuda", dtype=dtype)
        ops.head_norm_silu(o.cuda(), proj.cuda(), before, gain.cuda(), 1e-2, out, heads)
        want = plain.rms_norm(o.double().view(7, heads, vdim), gain.double(), 1e-2).reshape(7, -1) * \
            torch.nn.functional.silu(proj[:, before:before + heads * vdim].double())
        tolerance = 1e-5 if dtype is torch.float32 else 2e-2
        assert (out.cpu().double() - want).abs().max() < tolerance * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,n,k,options", [
    (5, 96, 64, {}), (12, 61, 37, {}), (16, 200, 96, {}), (3, 384, 256, {"few_token_min_elements": 1}),
    (30, 256, 512, {"few_token_min_elements": 1}), (40, 128, 64, {}), (300, 520, 192, {"tiled_min_tiles": 1}), (90, 77, 40, {})])
def test_squared_relu_behind_every_product(dtype, rows, n, k, options):
    """relu(x w^T)^2 through whichever product the runtime picks: the set-up-free one, the tcgen05 one for few
    tokens, the tiled one, the library's with a kernel behind it, the 32-bit ones."""
    from from_scratch_inference_engine_b200.engine.runtime import Runtime
    runtime = Runtime(dtype=dtype, max_positions=16, **options)
    g = torch.Generator().manual_seed(rows)
    x = torch.randn(rows, k, generator=g).to(runtime.dtype)
    w = (torch.randn(n, k, generator=g) / k ** 0.5 * 2).to(runtime.dtype)
    wd = w.cuda()
    runtime.prepare_weight(wd, plain_activation="relu2")
    got = runtime.linear_activated(x.cuda(), wd, "relu2", "test")
    want = torch.relu(x.double() @ w.double().T) ** 2
    tolerance = 1e-5 if dtype == "float32" else 2e-2
    assert got.dtype is runtime.dtype and int(runtime.error.item()) == 0
    assert (got.cpu().double() - want).abs().max() < tolerance * float(want.abs().max())
    assert (got.cpu()[want == 0] == 0).float().mean() > 0.99


# ------------------------------------------------------------------- each mechanism in a model
@pytest.mark.parametrize("name", ["window", "sinks", "difference", "difference_even", "recurrent", "recurrent_deep",
                                  "feed_forward", "all", "odd"])
def test_whole_prompt_and_token_by_token(tmp_path_factory, name):
    """The prompt in one step against the same tokens one by one: the first tokens of a sequence,
    page borders, window borders that fall on decoded tokens."""
    folder = folder_of(tmp_path_factory, name)
    requests = {"p": helpers.random_ids(vocab_of(name), 70, 11)}
    runner = runner_for(folder, "float32", num_pages=8)
    rows = helpers.run_trace_in_process(runner, helpers.trace_whole(requests))
    assert len(rows) == 70
    assert_rows(rows, requests, folder, F32_BOUND)
    rows = helpers.run_trace_in_process(runner, helpers.trace_tail_by_one(requests, tail=69))
    assert len(rows) == 70
    assert_rows(rows, requests, folder, F32_BOUND)


def test_faults_would_show_in_the_logits(tmp_path_factory):
    """The test models are sharp enough that a window one key off, a missing sink, values after the norm, a norm head by
    head, another rotation, a missing temperature or gate, swapped maps, a fixed weight of the difference, another
    tau, decays shared by the rows, outputs left unscaled, streams mixed with the transposed matrix, relu
    unsquared, other scales of embedding and logits and another eps move the logits far beyond the bound the engine
    is held to."""
    def moved(name, change=None, oracle=None):
        folder = folder_of(tmp_path_factory, name)
        config, weights = plain.load(folder)
        ids = helpers.random_ids(vocab_of(name), 60, 11)
        right = plain.forward(config, weights, ids)
        weights = dict(weights)
        kept = {k: getattr(plain, k) for k in (oracle or {})}
        if change is not None:
            change(config, weights)
        try:
            for k, f in (oracle or {}).items():
                setattr(plain, k, f)
            wrong = plain.forward(config, weights, ids)
        finally:
            for k, f in kept.items():
                setattr(plain, k, f)
        return float((wrong - right).abs().max()) / max(1.0, float(right.abs().max()))

    def mixer(index=0, **values):
        def change(config, weights):
            for key, value in values.items():
                at, keys = config["layers"][index]["mixer"], key.split("__")
                for part in keys[:-1]:
                    at = at[part]
                at[keys[-1]] = value
        return change

    def tensor(name, f):
        def change(config, weights):
            weights[name] = f(weights[name])
        return change

    def swapped_maps(config, weights):
        for which, heads in (("q", 4), ("k", 2)):
            t = weights[f"l0.mix.{which}"]
            weights[f"l0.mix.{which}"] = t.view(heads, 2, -1, t.shape[1]).flip(1).reshape(t.shape)

    def other_scale(key, value):
        def change(config, weights):
            config[key] = value
        return change

    def values_after_the_norm(q, k, v, mask, scale, sink):
        return kept_attention(q, k, k, mask, scale, sink)
    kept_attention = plain.sink_attention

    def head_by_head(x, w, eps):
        if x.dim() == 2 and x.shape[-1] in (96, 32):              # q and k of "window"
            return (plain.unit_rms(x.view(x.shape[0], -1, 16), eps).reshape(x.shape)) * w
        return plain.unit_rms(x, eps) * w

    def shared_decays(h, w, prefix, tau):
        a = kept_decays(h, w, prefix, tau)
        return a.mean(-1, keepdim=True).expand_as(a)
    kept_decays = plain.key_decays

    for name, change, oracle in (
            ("window", mixer(mask__size=12), None), ("window", mixer(mask__size=10), None),
            ("window", mixer(rot__dims=6), None), ("window", mixer(rot__scaling=None), None),
            ("window", None, {"rms_norm": head_by_head}), ("window", None, {"sink_attention": values_after_the_norm}),
            ("sinks", tensor("l0.mix.sink", lambda t: t - 40.0), None), ("sinks", tensor("l0.mix.g", torch.zeros_like), None),
            ("difference", mixer(q_temp__coef=0.0), None), ("difference", mixer(q_temp__every=8), None),
            ("difference", swapped_maps, None), ("difference", tensor("l0.mix.lq2", torch.zeros_like), None),
            ("difference", mixer(diff=0.4), None), ("difference", tensor("l0.mix.g", torch.zeros_like), None),
            ("recurrent", mixer(tau=4.2), None), ("recurrent", None, {"key_decays": shared_decays}),
            ("recurrent", tensor("l0.mix.norm", torch.ones_like), None), ("recurrent", other_scale("norm", {"eps": 3e-3}), None),
            ("all", tensor("l1.ls1", torch.ones_like), None), ("all", tensor("l0.ls2", torch.ones_like), None),
            ("all", tensor("l1.hc1.mix", lambda t: t.T), None), ("all", other_scale("embedding", {"scale": 1.4}), None),
            ("all", other_scale("logit_scale", 1.9), None),
            ("feed_forward", None, {"dense": lambda h, w, p: torch.relu(h @ w[p + "up"].T) @ w[p + "down"].T})):
        assert moved(name, change, oracle) > 50 * F32_BOUND, (name, change, oracle)


@pytest.mark.parametrize("dtype,name,bound", [("float32", "all", F32_BOUND), ("bfloat16", "wide", BF16_BOUND)])
def test_far_keys_page_borders_and_a_long_prompt(tmp_path_factory, dtype, name, bound):
    """A prompt of several hundred tokens, whole and cut inside a page, a window and a chunk of the recurrence,
    beside a short request in the same step, then decoding; in bfloat16 the long portions take the tcgen05
    attention and the chunk-parallel scan, the short ones the mma.sync attention - in one batch."""
    folder = folder_of(tmp_path_factory, name, dtype)
    requests = {"long": helpers.random_ids(vocab_of(name), 331, 3),
                "short": helpers.random_ids(vocab_of(name), 12, 4)}
    runner = runner_for(folder, dtype, num_pages=48)
    steps = [{"step": 0, "end": ["short"], "entries": [
                  {"id": "long", "tokens": requests["long"][:203], "want": [0, 15, 16, 20, 21, 63, 64, 99, 100, 127, 199, 202]},
                  {"id": "short", "tokens": requests["short"], "want": [0, 11]}]},
             {"step": 1, "end": [], "entries": [
                  {"id": "long", "tokens": requests["long"][203:329], "want": [0, 4, 5, 60, 63, 64, 98, 125]}]},
             {"step": 2, "end": [], "entries": [{"id": "long", "tokens": [requests["long"][329]], "want": [0]}]},
             {"step": 3, "end": ["long"], "entries": [{"id": "long", "tokens": [requests["long"][330]], "want": [0]}]}]
    rows = helpers.run_trace_in_process(runner, steps)
    assert len(rows) == 24
    assert_rows(rows, requests, folder, bound)


def test_the_forms_of_the_attention_agree_inside_a_model(tmp_path_factory):
    """The same long prompt with the tcgen05 attention, with mma.sync only and with the 32-bit kernel: the
    kernels are the only difference, so the logits agree far inside what bfloat16 rounding moves."""
    from from_scratch_inference_engine_b200.kernels import ops
    from from_scratch_inference_engine_b200.parts import scaled_attention
    folder = folder_of(tmp_path_factory, "wide", "bfloat16")
    ids = helpers.random_ids(vocab_of("wide"), 300, 9)
    rows, calls = {}, []
    inner = ops.attention_tc_scaled
    try:
        ops.attention_tc_scaled = lambda *a, **k: (calls.append(k["maps"]), inner(*a, **k))[1]
        for form in ("auto", "mma", "plain"):
            scaled_attention.FORM = form
            del calls[:]
            runner = runner_for(folder, "bfloat16", num_pages=24)
            rows[form] = helpers.run_trace_in_process(runner, helpers.trace_whole({"p": ids}))
            assert sorted(calls) == ([1, 1, 2, 2] if form == "auto" else [])
    finally:
        scaled_attention.FORM = "auto"
        ops.attention_tc_scaled = inner
    for form in ("mma", "plain"):
        for key, row in rows["auto"].items():
            assert np.abs(row - rows[form][key]).max() < BF16_BOUND * max(1.0, np.abs(row).max()), (form, key)


def test_sizes_that_fit_no_vector_in_bfloat16(tmp_path_factory):
    """Width 37, heads of 5 to 7 columns, nine streams: no row starts on 16 bytes.  The bfloat16 products and
    kernels take their plain forms."""
    folder = folder_of(tmp_path_factory, "odd", "bfloat16")
    requests = {"a": helpers.random_ids(vocab_of("odd"), 45, 6), "b": helpers.random_ids(vocab_of("odd"), 19, 7)}
    runner = runner_for(folder, "bfloat16", num_pages=8)
    for steps in (helpers.trace_whole(requests), helpers.trace_mixed(requests, seed=1, max_live=2)):
        rows = helpers.run_trace_in_process(runner, steps)
        assert len(rows) == 64
        assert_rows(rows, requests, folder, BF16_BOUND)


# ---------------------------------------------------------------------------- the whole design
@pytest.mark.parametrize("name", ["all", "wide"])
@pytest.mark.parametrize("dtype,bound", [("float32", F32_BOUND), ("bfloat16", BF16_BOUND)])
def test_portions_of_every_size(tmp_path_factory, name, dtype, bound):
    folder = folder_of(tmp_path_factory, name, dtype)
    requests = {"a": helpers.random_ids(vocab_of(name), 90, 1),
                "b": helpers.random_ids(vocab_of(name), 37, 2)}
    runner = runner_for(folder, dtype, num_pages=8)
    steps = helpers.trace_portions(requests, seed=3)
    assert min(len(e["tokens"]) for s in steps for e in s["entries"]) <= 2
    rows = helpers.run_trace_in_process(runner, steps)
    assert len(rows) == 127
    assert_rows(rows, requests, folder, bound)


@pytest.mark.parametrize("name,dtype,bound", [("all", "float32", F32_BOUND), ("wide", "bfloat16", BF16_BOUND)])
def test_mixed_batches_reuse_pages_and_slots(tmp_path_factory, name, dtype, bound):
    """Six unequal requests through two slots and a pool that holds little more than two of
    them: portions of one beside single tokens of another, requests that sit a step out, one
    that is released in the middle and fed again from its first token - every request's rows equal what
    it gives alone."""
    folder = folder_of(tmp_path_factory, name, dtype)
    lengths = {"a": 75, "b": 9, "c": 41, "d": 1, "e": 58, "f": 26}
    requests = {k: helpers.random_ids(vocab_of(name), n, i + 20)
                for i, (k, n) in enumerate(lengths.items())}
    steps, names = helpers.trace_mixed_with_recompute(requests, seed=5, max_live=2)
    need = helpers.live_tokens_needed(steps, round_to=16)
    runner = runner_for(folder, dtype, num_pages=need // 16, max_requests=2)
    rows = helpers.run_trace_in_process(runner, steps)
    assert len(rows) >= sum(lengths.values())
    assert_rows(rows, names, folder, bound)
    assert runner.cache.slots.num_free == 2
    assert all(free == need // 16 for free in runner.cache.free_pages())


def test_pages_behind_a_window_are_given_back(tmp_path_factory):
    """A request much longer than the pool: 400 tokens of windowed layers pass through pages for 80."""
    from from_scratch_inference_engine_b200 import LoadedModel, ModelRunner
    folder = folder_of(tmp_path_factory, "window")
    requests = {"long": helpers.random_ids(vocab_of("window"), 400, 8)}
    model = LoadedModel.from_pretrained(folder, dtype="float32", max_positions=512)
    runner = ModelRunner(model.model, model.runtime, page_size=16, num_pages=5, max_requests=2,
                         max_step_tokens=64)
    steps, at = [], 0
    for n in [40, 33, 40, 7, 40, 40, 25, 40, 40, 40, 40, 13]:
        steps.append({"step": len(steps), "end": [], "entries": [
            {"id": "long", "tokens": requests["long"][at:at + n], "want": [0, n - 1]}]})
        at += n
    steps.append({"step": len(steps), "end": ["long"], "entries": [
        {"id": "long", "tokens": requests["long"][at:], "want": [0]}]})
    rows = helpers.run_trace_in_process(runner, steps)
    assert_rows(rows, requests, folder, F32_BOUND)
    assert all(free == 5 for free in runner.cache.free_pages())


def test_long_decoding_through_graphs_and_without(tmp_path_factory):
    """A short prompt, then 150 tokens one by one through captured graphs - windows move over decoded tokens,
    the temperature steps up many times; the same without graphs gives the same rows up to the order of the
    sums."""
    folder = folder_of(tmp_path_factory, "all")
    requests = {"long": helpers.random_ids(vocab_of("all"), 157, 9)}
    steps = helpers.trace_tail_by_one(requests, tail=150)
    both = []
    for graphs in (True, False):
        runner = runner_for(folder, "float32", num_pages=12, cuda_graphs=graphs)
        assert runner.cuda_graphs == graphs
        rows = helpers.run_trace_in_process(runner, steps)
        assert_rows(rows, requests, folder, F32_BOUND)
        both.append(rows)
    for key in both[0]:
        assert float(np.abs(both[0][key] - both[1][key]).max()) < \
            F32_BOUND * max(1.0, float(np.abs(both[0][key]).max()))


def test_decode_batch_with_padding(tmp_path_factory):
    """Three requests decode together in a captured batch of four (bfloat16, mma.sync attention over
    split ranges in the graph): the padding entry writes no page and no state and changes nobody's rows."""
    folder = folder_of(tmp_path_factory, "wide", "bfloat16")
    requests = {k: helpers.random_ids(vocab_of("wide"), n, s)
                for k, n, s in (("a", 130, 1), ("b", 122, 2), ("c", 126, 3))}
    runner = runner_for(folder, "bfloat16", num_pages=28)
    steps = [{"step": 0, "end": [], "entries": [
        {"id": k, "tokens": ids[:92], "want": [91]} for k, ids in requests.items()]}]
    for t in range(92, 122):
        steps.append({"step": len(steps), "end": [], "entries": [
            {"id": k, "tokens": [ids[t]], "want": [0]} for k, ids in requests.items()]})
    steps[-1]["end"] = list(requests)
    rows = helpers.run_trace_in_process(runner, steps)
    assert runner._graphs
    assert_rows(rows, requests, folder, BF16_BOUND)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(tmp_path_factory, dtype):
    """Requests of unequal length through `Engine` and its scheduler with a small token budget
    (prompts go in portions) and two slots: every generated token is the plain implementation's
    choice; where the plain logits are a near tie the engine may pick either."""
    from from_scratch_inference_engine_b200 import Engine, LoadedModel, SamplingParams
    folder = folder_of(tmp_path_factory, "all", dtype)
    model = LoadedModel.from_pretrained(folder, dtype=dtype, max_positions=256)
    engine = Engine(model, block_size=16, num_blocks=16, max_batch=2, max_step_tokens=24)
    prompts = [helpers.random_ids(vocab_of("all"), n, s) for n, s in ((45, 1), (7, 2), (30, 3))]
    ids = [engine.add_request(p, SamplingParams(temperature=0.0), 8) for p in prompts]
    engine.run_until_done()
    config, weights = plain.load(folder)
    slack = 1e-3 if dtype == "float32" else 0.15
    for rid, prompt in zip(ids, prompts):
        seq = list(prompt)
        assert len(engine.output(rid)) == 8
        for token in engine.output(rid):
            logits = plain.forward(config, weights, seq)[-1]
            assert float(logits.max() - logits[token]) <= slack * max(1.0, float(logits.abs().max()))
            seq.append(token)


def test_llm_entry_point_reads_the_design_by_its_name(tmp_path_factory):
    from from_scratch_inference_engine_b200 import LLM, GenerationConfig, load_config
    folder = folder_of(tmp_path_factory, "odd")
    assert type(load_config(folder)).__name__ == "LanilornConfig"
    llm = LLM(folder, block_size=16, num_blocks=8, max_batch=2, dtype="float32", eos_id=-1)
    prompt = helpers.random_ids(vocab_of("odd"), 19, 4)
    got = llm.generate_ids(prompt, GenerationConfig(max_tokens=5))
    assert len(got) == 5
    config, weights = plain.load(folder)
    seq = list(prompt)
    for token in got:
        logits = plain.forward(config, weights, seq)[-1]
        assert float(logits.max() - logits[token]) <= 1e-3 * max(1.0, float(logits.abs().max()))
        seq.append(token)


@pytest.mark.parametrize("dtype,name,bound", [("float32", "all", F32_BOUND), ("bfloat16", "wide", BF16_BOUND)])
def test_trace_replay_program_runs_the_design(tmp_path_factory, tmp_path, dtype, name, bound):
    """bin/trace_run as a user runs it (a subprocess, steps on standard input, logits in files)
    on a mixed trace of five requests through four slots and a pool for the live tokens only."""
    import json
    import subprocess
    from pathlib import Path
    folder = folder_of(tmp_path_factory, name, dtype)
    vocab = vocab_of(name)
    requests = {key: helpers.random_ids(vocab, n, i)
                for i, (key, n) in enumerate({"a": 90, "b": 40, "c": 70, "d": 33, "e": 64}.items())}
    steps = helpers.trace_mixed(requests, seed=3)
    need = helpers.live_tokens_needed(steps, round_to=64)
    root = Path(__file__).resolve().parent.parent
    text = "".join(json.dumps(step) + "\n" for step in steps)
    done = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype,
                           "--out", str(tmp_path / "out"), "--max-tokens", str(need)],
                          input=text, capture_output=True, text=True, timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done ")] == \
        [f"done {s['step']}" for s in steps]
    outputs = {s["step"]: np.fromfile(tmp_path / "out" / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab)
               for s in steps if any(e["want"] for e in s["entries"])}
    rows = helpers.collect_rows(steps, outputs)
    assert len(rows) == sum(len(ids) for ids in requests.values())
    assert_rows(rows, requests, folder, bound)


@pytest.mark.parametrize("seed", range(1, 11))
def test_configurations_drawn_at_random(tmp_path_factory, seed):
    """Mixers, sizes, windows, rotations, constants and streams drawn at random (fixed seeds), in float32:
    a whole prompt, portions beside decoded tokens of other requests, and a tail token by token, against
    the plain implementation."""
    folder = lm.write_random(tmp_path_factory.mktemp(f"lanilorn_random{seed}"), seed)
    vocab = lm.CONFIGS[f"random{seed}"]["vocab"]
    requests = {"a": helpers.random_ids(vocab, 150, seed), "b": helpers.random_ids(vocab, 41, seed + 1),
                "c": helpers.random_ids(vocab, 67, seed + 2)}
    runner = runner_for(folder, "float32", num_pages=24)
    for steps in (helpers.trace_whole(requests), helpers.trace_mixed(requests, seed=seed, max_live=3),
                  helpers.trace_tail_by_one({"b": requests["b"]}, tail=30)):
        rows = helpers.run_trace_in_process(runner, steps)
        assert_rows(rows, requests, folder, F32_BOUND)
