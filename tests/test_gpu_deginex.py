"""The Deginex design in the engine against the plain implementation of the tests: every mechanism
alone, whole prompts against decoding token by token, portions down to two tokens, mixed batches with
pages and slots that are used again, keys far away, at page borders and on either side of a chunk's
edge in prompts and in decoding, the first tokens of a sequence, long decoding, and greedy generation
through the engine."""

import numpy as np
import pytest
import torch

import deginex_models as dm
import helpers
import plain_deginex as plain

pytestmark = pytest.mark.gpu

F32_BOUND = 2e-4          # largest |engine - plain| of a row, relative to max(1, largest |plain|)
BF16_BOUND = 6e-2
# float32 runs the sharpened routers (every token chooses its own experts); bfloat16 runs narrow ones,
# whose choice no rounding can turn
SHARPEN = {"float32": True, "bfloat16": False}

_folders = {}
_plain = {}


def folder_of(tmp_path_factory, name, **options):
    key = (name, tuple(sorted(options.items())))
    if key not in _folders:
        _folders[key] = dm.write_model(tmp_path_factory.mktemp(f"deginex_{name}"), name, **options)
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
    return dm.CONFIGS[name]["vocab"]


def dev(values, dtype=torch.int32):
    return torch.tensor(values, dtype=dtype, device="cuda")


# ----------------------------------------------------------------- mechanisms, kernel by kernel
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams,width", [(1, 36), (2, 37), (3, 256), (4, 1000), (4, 4104), (5, 64), (8, 520), (9, 100), (17, 41)])
def test_streams_settle_are_gathered_and_normed_in_one_pass(dtype, streams, width):
    """The first sublayer's input from streams that do not exist yet, the first output that brings them
    into being, an output onto existing streams, the sum on chosen rows only without touching them; a
    layer norm with gain and bias and an RMS norm."""
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(streams * 1000 + width)
    rand = lambda *shape: torch.randn(shape, generator=g)
    tokens, eps = 7, 1e-3
    start, held = rand(tokens, width) + 0.5, rand(tokens, streams, width) * 2
    mix, spread, gather = rand(streams, streams), rand(streams), rand(streams)
    gain, bias = rand(width), rand(width)
    delta = (rand(tokens, width) * 2).to(dtype)
    rows = torch.tensor([5, 0, 3], dtype=torch.int32)
    tolerance = 5e-5 if dtype is torch.float32 else 2e-2

    def expect(x, pending, a, centred):
        parts = [x[:, s].double() for s in range(streams)]
        if pending:
            parts = plain.spread_streams(parts, mix.double(), spread.double(), delta.double())
        u = plain.gather_streams(parts, torch.ones(streams).double() if a is None else a.double())
        y = plain.layer_norm(u, gain.double(), bias.double(), eps) if centred else \
            plain.unit_rms(u, eps) * gain.double()
        return torch.stack(parts, dim=1), y

    c = lambda t: None if t is None else t.cuda()
    for has_start, pending, a, centred, some in (
            (True, False, gather, True, None), (True, True, gather, True, None), (False, True, gather, True, None),
            (False, True, gather, False, None), (False, True, None, True, rows), (True, True, None, True, rows),
            (False, False, None, False, rows)):
        x0 = start[:, None].expand(tokens, streams, width) if has_start else held
        want_x, want_y = expect(x0, pending, a, centred)
        x = torch.full((tokens, streams, width), 3.0, device="cuda") if has_start else held.clone().cuda()
        before = x.clone()
        count = tokens if some is None else some.numel()
        out = torch.zeros(count, width, device="cuda", dtype=dtype)
        ops.stream_norm(x, c(start) if has_start else None, c(delta) if pending else None, c(mix) if pending else None,
                        c(spread) if pending else None, c(a), c(gain), c(bias) if centred else None, eps, out,
                        rows=c(some), write_x=some is None, centred=centred)
        want = want_y if some is None else want_y[some.long()]
        assert (out.cpu().double() - want).abs().max() < tolerance * max(1.0, float(want.abs().max()))
        if pending and some is None:
            assert (x.cpu().double() - want_x).abs().max() < 1e-5 * max(1.0, float(want_x.abs().max()))    # 32-bit
        else:
            assert torch.equal(x, before)
    x = held.clone().cuda()                            # the settling alone
    ops.stream_norm(x, None, c(delta), c(mix), c(spread), None, None, None, eps, None)
    want_x, _ = expect(held, True, None, True)
    assert (x.cpu().double() - want_x).abs().max() < 1e-5 * max(1.0, float(want_x.abs().max()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,vdim", [(12, 10), (64, 64), (128, 128)])
def test_heads_divided_by_their_root_mean_square_into_the_cache(dtype, dim, vdim):
    """q and k without a stored gain: q in place, k and v into the token's slot; columns behind q, k, v
    (the gate) are left alone; without `unit` nothing is divided."""
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    heads, kv_heads, page, eps, tokens = 3, 2, 4, 1e-2, 9
    width = (heads + kv_heads) * dim + kv_heads * vdim
    proj = (torch.randn(tokens, width + 6, generator=g) * 0.3).to(dtype)
    slots = torch.tensor([7, 2, 30, 12, 5, 21, -1, 0, 19], dtype=torch.int32)
    pages = 8
    table = torch.zeros(1, 0, device="cuda")
    for unit in (True, False):
        both = torch.zeros(pages, kv_heads * page * (dim + vdim), device="cuda", dtype=dtype)
        k_pages, v_pages = both[:, :kv_heads * page * dim], both[:, kv_heads * page * dim:]
        work = proj.clone().cuda()
        error = torch.zeros(1, dtype=torch.int32, device="cuda")
        ops.norm_rotate_write(work, torch.arange(tokens, dtype=torch.int32).cuda(), table, slots.cuda(), k_pages, v_pages,
                              both.stride(0), page, heads, kv_heads, dim, vdim, 0, None, None, eps, error, unit=unit)
        assert int(error.item()) == 0
        q = proj[:, :heads * dim].double().view(tokens, heads, dim)
        k = proj[:, heads * dim:(heads + kv_heads) * dim].double().view(tokens, kv_heads, dim)
        v = proj[:, (heads + kv_heads) * dim:width].double().view(tokens, kv_heads, vdim)
        if unit:
            q, k = plain.unit_rms(q, eps), plain.unit_rms(k, eps)
        tolerance = 1e-5 if dtype is torch.float32 else 2e-2
        assert (work[:, :heads * dim].cpu().double().view(tokens, heads, dim) - q).abs().max() < tolerance * 4
        assert torch.equal(work[:, width:].cpu(), proj[:, width:])
        kp = k_pages.cpu().double().reshape(pages, kv_heads, page, dim)
        vp = v_pages.cpu().double().reshape(pages, kv_heads, page, vdim)
        for t, slot in enumerate(slots.tolist()):
            if slot < 0:
                continue
            assert (kp[slot // page, :, slot % page] - k[t]).abs().max() < tolerance * 4
            assert (vp[slot // page, :, slot % page] - v[t]).abs().max() < 1e-6
        assert float(kp.abs().sum(dim=(1, 3)).ne(0).sum()) == 8      # one token had no slot: nothing stored


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
    """Requests of (cached, new) tokens over shuffled pages of two entries (the second one is read),
    with a query that points at the first key of its chunk while the key before the chunk would win if
    it were seen, and the plain result."""

    def __init__(self, lengths, heads, kv_heads, dk, dv, page, dtype, scales, chunk, window, softcap, gated, seed):
        g = torch.Generator().manual_seed(seed)
        self.lengths, self.heads, self.kv_heads, self.dk, self.dv, self.page = lengths, heads, kv_heads, dk, dv, page
        self.dtype, self.chunk, self.window, self.softcap = dtype, chunk, window, softcap
        group = heads // kv_heads
        total = sum(-(-(a + b) // page) for a, b in lengths) + 3
        order = torch.randperm(total, generator=g).tolist()
        keys, values = torch.zeros(total, kv_heads, page, dk, dtype=dtype), torch.zeros(total, kv_heads, page, dv, dtype=dtype)
        tables, qs, want, used = [], [], [], 0
        gates = [torch.randn(new, heads * dv, generator=g).to(dtype) for _, new in lengths]
        for (cached, new), gate in zip(lengths, gates):
            n = cached + new
            k = plain.unit_rms(torch.randn(n, kv_heads, dk, generator=g).double(), 0.0).float()
            q = plain.unit_rms(torch.randn(new, heads, dk, generator=g).double(), 0.0).float()
            for qi in sorted({0, new // 3, new - 1}):
                i = cached + qi
                first = max(i // chunk * chunk if chunk else 0, i - window + 1 if window else 0)
                q[qi] = k[first, :, None, :].expand(kv_heads, group, dk).reshape(heads, dk)
                if first > 0:
                    k[first - 1] = k[first] * 1.1                     # outside: it would win if it were seen
            q, k = q.to(dtype), k.to(dtype)
            v = torch.randn(n, kv_heads, dv, generator=g).to(dtype)
            blocks = -(-n // page)
            kp, table = _paged(k, page, order[used:used + blocks], total)
            vp, _ = _paged(v, page, order[used:used + blocks], total)
            used += blocks
            keys += kp
            values += vp
            tables.append(table)
            qs.append(q)
            mask = plain.chunk_mask(n, chunk or n)
            if window:
                mask &= torch.arange(n)[:, None] - torch.arange(n)[None, :] < window
            out = torch.zeros(new, heads, dv, dtype=torch.float64)
            for h in range(heads):
                s = q[:, h].double() @ k[:, h // group].double().T * scales[h]
                if softcap:
                    s = softcap * torch.tanh(s / softcap)
                out[:, h] = torch.softmax(s.masked_fill(~mask[cached:], -float("inf")), -1) @ v[:, h // group].double()
            if gated:
                out = out * torch.sigmoid(gate.double()).view(new, heads, dv)
            want.append(out)
        self.want = torch.cat(want)
        self.tokens = self.want.shape[0]
        self.tables = torch.full((len(lengths), max(len(t) for t in tables)), -1, dtype=torch.int32)
        for i, t in enumerate(tables):
            self.tables[i, :len(t)] = torch.tensor(t, dtype=torch.int32)
        self.tables = self.tables.cuda()
        # q and the gate as columns of one wider tensor, as the engine's product leaves them
        wide = torch.zeros(self.tokens, heads * dk + 16 + heads * dv, dtype=dtype)
        wide[:, :heads * dk] = torch.cat(qs).reshape(self.tokens, -1)
        wide[:, heads * dk + 16:] = torch.cat(gates)
        self.q = wide.cuda()
        self.gate = self.q[:, heads * dk + 16:] if gated else None
        self.keys, self.values = keys, values
        self.scales = torch.tensor(scales, dtype=torch.float32, device="cuda")
        starts = np.cumsum([0] + [b for _, b in lengths])
        self.qstart, self.qlen = dev(starts[:-1].tolist()), dev([b for _, b in lengths])
        self.pos0, self.slots = dev([a for a, _ in lengths]), dev(list(range(len(lengths))))

    def tiles(self, rows, only):
        item, row0, toks, at = [], [], [], 0
        for i, (_, new) in enumerate(self.lengths):
            if i in only:
                for r in range(0, new * (self.heads // self.kv_heads), rows):
                    item.append(i)
                    row0.append(r)
                toks += range(at, at + new)
            at += new
        return dev(item), dev(row0), len(item), dev(toks), len(toks)

    def scratch(self, nsplit):
        return (torch.full((nsplit * self.tokens * self.heads * self.dv,), float("nan"), device="cuda"),
                torch.full((nsplit * self.tokens * self.heads * 2,), float("nan"), device="cuda"))

    def run(self, form, nsplit, only=None):
        """`form` "tcgen05", or a form of `scaled_attention`; `only`: the requests that the tiles hold."""
        from from_scratch_inference_engine_b200.kernels import ops
        everyone = only is None
        only = range(len(self.lengths)) if everyone else only
        out = torch.full((self.tokens, self.heads * self.dv), 7.0, device="cuda", dtype=self.dtype)
        error = torch.zeros(1, dtype=torch.int32, device="cuda")
        q_ld = self.q.stride(0)
        if form == "tcgen05":
            pages = torch.randn(self.keys.shape[0], 2, 2, *self.keys.shape[1:]).to(self.dtype)
            pages[:, 1, 0], pages[:, 1, 1] = self.keys, self.values
            item, row0, count, toks, n = self.tiles(ops.ATTENTION_TC_ROWS, only)
            ops.attention_tc_scaled(ops.PagesMap(pages.cuda()), 1, self.q, q_ld, self.scales, self.tables, item, row0, count,
                                    self.qstart, self.qlen, self.pos0, out, self.tokens, self.heads, self.kv_heads,
                                    self.window, error, nsplit, *self.scratch(nsplit), chunk=self.chunk,
                                    softcap=self.softcap, gate=self.gate, combine_tokens=toks, num_combine=n)
        else:
            both = torch.cat([self.keys.flatten(1), self.values.flatten(1)], dim=1).cuda()
            split = self.keys[0].numel()
            item, row0, count, toks, n = self.tiles(ops.scaled_attention_rows(self.dtype, self.dk, self.dv, False, form), only)
            ops.scaled_attention(self.q, q_ld, self.scales, both[:, :split], both[:, split:], both.stride(0), self.page,
                                 self.dk, self.dv, False, self.tables, item, row0, count, self.qstart, self.qlen,
                                 self.pos0, self.slots, out, self.tokens, self.heads, self.kv_heads, self.window, error,
                                 nsplit, *self.scratch(nsplit), form=form, chunk=self.chunk, softcap=self.softcap,
                                 gate=self.gate, combine_tokens=None if everyone else toks, num_combine=n)
        assert int(error.item()) == 0
        return out.cpu().double().reshape(self.tokens, self.heads, self.dv), toks.cpu().long()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dk,dv,kv_heads,chunk,softcap,gated", [
    (24, 40, 2, 37, 6.0, True), (80, 56, 1, 150, 17.0, True), (48, 128, 2, 64, 3.0, True), (64, 64, 2, 100, 5.0, False),
    (128, 128, 3, 128, 15.0, True), (64, 64, 6, 300, 0.0, True)])
def test_capped_scores_chunks_and_gated_columns(dtype, dk, dv, kv_heads, chunk, softcap, gated):
    """Every form of the attention kernel that takes the sizes, whole and split over key ranges: a long
    portion behind 300 cached tokens, a first portion, two tokens behind 40, a token decoded at position
    260; scales of both signs."""
    scales = [0.5, 0.9, -0.4, 1.2, 0.7, 1.0] if dk < 64 else [0.3, 0.5, -0.2, 0.4, 0.25, 0.6]
    case = Attention([(300, 177), (0, 90), (40, 2), (260, 1)], 6, kv_heads, dk, dv, 16, dtype, scales, chunk, 0, softcap,
                     gated, seed=dk + chunk)
    forms = ["plain"]
    if dtype is torch.bfloat16 and dv % 64 == 0 and dk % 16 == 0:
        forms += ["mma", "mma_split", "mma_few"] + (["tcgen05"] if dk == dv else [])
    for form in forms:
        for nsplit in (1, 3):
            got, _ = case.run(form, nsplit)
            tolerance = 2e-4 if dtype is torch.float32 else 2e-2
            assert (got - case.want).abs().max() < tolerance * max(1.0, float(case.want.abs().max())), (form, nsplit)


@pytest.mark.parametrize("dim,heads,kv_heads,page,chunk,window,softcap,gated", [
    (64, 8, 1, 16, 0, 0, 0.0, False), (64, 4, 4, 8, 0, 70, 4.0, True), (128, 6, 2, 32, 256, 0, 30.0, True),
    (128, 4, 1, 16, 90, 130, 8.0, False), (64, 2, 2, 128, 33, 20, 2.0, True), (128, 12, 4, 64, 1, 0, 9.0, True)])
def test_tcgen05_attention_over_windows_chunks_and_split_ranges(dim, heads, kv_heads, page, chunk, window, softcap, gated):
    """The tcgen05 form against the plain result and the 32-bit kernel: long and short portions, windows
    and chunks that start inside a tile of keys, key ranges split unevenly, page sizes from 8 to 128; its
    32-bit weights keep it as close as the 32-bit kernel on the same bfloat16 operands."""
    scales = [(0.9 if h % 2 else 0.4) * (64 / dim) ** 0.5 for h in range(heads)]
    case = Attention([(517, 310), (0, 411), (129, 3)], heads, kv_heads, dim, dim, page, torch.bfloat16, scales, chunk, window,
                     softcap, gated, seed=dim + heads)
    base, _ = case.run("plain", 1)
    for nsplit in (1, 2, 5):
        got, _ = case.run("tcgen05", nsplit)
        assert (got - case.want).abs().max() < 1.5e-2 * max(1.0, float(case.want.abs().max())), nsplit
        # element by element no further than a bfloat16 rounding of the result from the 32-bit kernel
        assert ((got - base).abs() <= 1.6e-2 * base.abs() + 1e-3).all(), nsplit


def test_split_ranges_of_listed_tokens_only():
    """Tiles of some requests, split over key ranges and merged for their tokens: the other requests' rows
    stay as they were (another launch of the step fills them)."""
    case = Attention([(90, 200), (333, 1), (0, 150), (251, 1)], 4, 2, 64, 64, 16, torch.bfloat16, [0.4] * 4, 120, 0, 9.0,
                     True, seed=5)
    for form, only in (("tcgen05", (0, 2)), ("auto", (1, 3)), ("plain", (1, 3)), ("mma_few", (1, 3))):
        got, toks = case.run(form, 3, only)
        assert (got[toks] - case.want[toks]).abs().max() < 2e-2 * max(1.0, float(case.want.abs().max()))
        rest = torch.ones(case.tokens, dtype=torch.bool)
        rest[toks] = False
        assert (got[rest] == 7.0).all()


def test_weights_over_the_chosen_experts_alone():
    """Choice on the logits with the router's bias; weights a softmax over the chosen; the largest logit
    far above the rest, hundreds below zero and equal ones (ties go to the lower index)."""
    from from_scratch_inference_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(7)
    for experts, top in ((4, 1), (5, 5), (16, 4), (100, 7)):
        tokens = 40
        logits, bias = torch.randn(tokens, experts, generator=g) * 3, torch.randn(experts, generator=g) * 2
        logits[0] *= 100.0
        logits[1] -= 500.0
        ids = torch.empty(tokens, top, dtype=torch.int32, device="cuda")
        weights = torch.empty(tokens, top, device="cuda")
        ops.moe_route(None, None, None, ids, weights, top, 1, 1, 1.0, "chosen_softmax", True, logits=logits.cuda(),
                      bias=bias.cuda())
        w = {"r.router": torch.eye(experts, dtype=torch.float64), "r.router.b": bias.double()}
        want_ids, want_w = plain.route(logits.double(), w, "r.", top)
        for t in range(tokens):
            have = dict(zip(ids[t].tolist(), weights[t].tolist()))
            assert set(have) == set(want_ids[t].tolist()), t
            for e, value in zip(want_ids[t].tolist(), want_w[t].tolist()):
                assert abs(have[e] - value) < 1e-4
    ids, weights = torch.empty(1, 2, dtype=torch.int32, device="cuda"), torch.empty(1, 2, device="cuda")
    ops.moe_route(None, None, None, ids, weights, 2, 1, 1, 3.0, "chosen_softmax", True, logits=torch.zeros(1, 4).cuda())
    assert sorted(ids[0].tolist()) == [0, 1] and weights[0].tolist() == [1.5, 1.5]


# ------------------------------------------------------------------- each mechanism in a model
@pytest.mark.parametrize("name", ["chunk", "capped", "experts", "loop", "loop_first", "loop_last", "odd"])
def test_whole_prompt_and_token_by_token(tmp_path_factory, name):
    """The prompt in one step against the same tokens one by one: the first tokens of a sequence,
    page borders, chunk borders that fall on decoded tokens, every pass with its own cache."""
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
    """The test models are sharp enough that a chunk one key off, q and k left undivided, a missing cap, a
    missing gate, streams mixed with the transposed matrix, coefficients of the other sublayer, a pass
    left out, norms without their bias, a router without its bias, weights over all experts, another eps
    move the logits far beyond the bound the engine is held to."""
    def moved(name, change, oracle=None):
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

    def wider_chunk(config, weights):
        config["layers"][0]["mixer"]["mask"]["size"] += 1

    def higher_cap(config, weights):
        config["layers"][0]["mixer"]["softcap"] = 1e6

    def no_gate(config, weights):
        weights["l0.mix.g"] = torch.zeros_like(weights["l0.mix.g"])

    def mix_transposed(config, weights):
        weights["l1.hc1.mix"] = weights["l1.hc1.mix"].T

    def other_sublayer(config, weights):
        for part in ("in", "out", "mix"):
            a, b = f"l0.hc1.{part}", f"l0.hc2.{part}"
            weights[a], weights[b] = weights[b], weights[a]

    def one_pass_less(config, weights):
        config["loop"]["times"] -= 1

    def no_norm_bias(config, weights):
        weights["l0.norm1.b"] = torch.zeros_like(weights["l0.norm1.b"])

    def no_router_bias(config, weights):
        weights["l0.mlp.router.b"] = torch.zeros_like(weights["l0.mlp.router.b"])

    def other_eps(config, weights):
        config["norm"]["eps"] *= 30.0

    def over_all(h, w, prefix, top):
        z = h @ w[prefix + "router"].T + w[prefix + "router.b"]
        ids = torch.topk(z, top, dim=-1).indices
        return ids, torch.softmax(z, -1).gather(1, ids)

    for name, change, oracle in (
            ("chunk", wider_chunk, None), ("chunk", no_gate, None), ("chunk", None, {"unit_rms": lambda x, eps: x}),
            ("capped", higher_cap, None), ("loop", mix_transposed, None), ("loop", other_sublayer, None),
            ("loop", one_pass_less, None), ("loop", no_norm_bias, None), ("experts", no_router_bias, None),
            ("experts", None, {"route": over_all}), ("loop_last", other_eps, None)):
        assert moved(name, change, oracle) > 50 * F32_BOUND, (name, change, oracle)


@pytest.mark.parametrize("dtype,name,bound", [("float32", "loop", F32_BOUND), ("bfloat16", "wide", BF16_BOUND)])
def test_far_keys_page_borders_and_a_long_prompt(tmp_path_factory, dtype, name, bound):
    """A prompt of several hundred tokens, whole and cut inside a page and a chunk, beside a short
    request in the same step, then decoding; chunks start inside pages that earlier steps filled; in
    bfloat16 the long portions take the tcgen05 attention and the experts' grouped product, the short
    ones the mma.sync attention and tiles of 64 rows - in one batch."""
    folder = folder_of(tmp_path_factory, name, sharpen=SHARPEN[dtype])
    requests = {"long": helpers.random_ids(vocab_of(name), 331, 3),
                "short": helpers.random_ids(vocab_of(name), 12, 4)}
    runner = runner_for(folder, dtype, num_pages=48)
    steps = [{"step": 0, "end": ["short"], "entries": [
                  {"id": "long", "tokens": requests["long"][:203], "want": [0, 15, 16, 99, 100, 101, 127, 199, 200, 202]},
                  {"id": "short", "tokens": requests["short"], "want": [0, 11]}]},
             {"step": 1, "end": [], "entries": [
                  {"id": "long", "tokens": requests["long"][203:329], "want": [0, 4, 5, 60, 96, 97, 98, 125]}]},
             {"step": 2, "end": [], "entries": [{"id": "long", "tokens": [requests["long"][329]], "want": [0]}]},
             {"step": 3, "end": ["long"], "entries": [{"id": "long", "tokens": [requests["long"][330]], "want": [0]}]}]
    rows = helpers.run_trace_in_process(runner, steps)
    assert len(rows) == 22
    assert_rows(rows, requests, folder, bound)


def test_the_forms_of_the_attention_agree_inside_a_model(tmp_path_factory):
    """The same long prompt with the tcgen05 attention, with mma.sync only and with the 32-bit kernel: the
    kernels are the only difference, so the logits agree far inside what bfloat16 rounding moves."""
    from from_scratch_inference_engine_b200.kernels import ops
    from from_scratch_inference_engine_b200.parts import scaled_attention
    folder = folder_of(tmp_path_factory, "wide", sharpen=False)
    ids = helpers.random_ids(vocab_of("wide"), 300, 9)
    rows, calls = {}, []
    inner = ops.attention_tc_scaled
    try:
        ops.attention_tc_scaled = lambda *a, **k: (calls.append(1), inner(*a, **k))[1]
        for form in ("auto", "mma", "plain"):
            scaled_attention.FORM = form
            del calls[:]
            runner = runner_for(folder, "bfloat16", num_pages=24)
            rows[form] = helpers.run_trace_in_process(runner, helpers.trace_whole({"p": ids}))
            assert bool(calls) == (form == "auto")
    finally:
        scaled_attention.FORM = "auto"
        ops.attention_tc_scaled = inner
    for form in ("mma", "plain"):
        for key, row in rows["auto"].items():
            assert np.abs(row - rows[form][key]).max() < BF16_BOUND * max(1.0, np.abs(row).max()), (form, key)


def test_sizes_that_fit_no_vector_in_bfloat16(tmp_path_factory):
    """Width 37, heads of 6 and 10 columns, nine streams, experts of 13: no row starts on 16 bytes.  The
    bfloat16 products and kernels take their plain forms."""
    folder = folder_of(tmp_path_factory, "odd", sharpen=False)
    requests = {"a": helpers.random_ids(vocab_of("odd"), 45, 6), "b": helpers.random_ids(vocab_of("odd"), 19, 7)}
    runner = runner_for(folder, "bfloat16", num_pages=8)
    for steps in (helpers.trace_whole(requests), helpers.trace_mixed(requests, seed=1, max_live=2)):
        rows = helpers.run_trace_in_process(runner, steps)
        assert len(rows) == 64
        assert_rows(rows, requests, folder, BF16_BOUND)


# ---------------------------------------------------------------------------- the whole design
@pytest.mark.parametrize("name", ["loop", "wide"])
@pytest.mark.parametrize("dtype,bound", [("float32", F32_BOUND), ("bfloat16", BF16_BOUND)])
def test_portions_of_every_size(tmp_path_factory, name, dtype, bound):
    folder = folder_of(tmp_path_factory, name, sharpen=SHARPEN[dtype])
    requests = {"a": helpers.random_ids(vocab_of(name), 90, 1),
                "b": helpers.random_ids(vocab_of(name), 37, 2)}
    runner = runner_for(folder, dtype, num_pages=8)
    steps = helpers.trace_portions(requests, seed=3)
    assert min(len(e["tokens"]) for s in steps for e in s["entries"]) <= 2
    rows = helpers.run_trace_in_process(runner, steps)
    assert len(rows) == 127
    assert_rows(rows, requests, folder, bound)


@pytest.mark.parametrize("dtype,bound", [("float32", F32_BOUND), ("bfloat16", BF16_BOUND)])
def test_mixed_batches_reuse_pages_and_slots(tmp_path_factory, dtype, bound):
    """Six unequal requests through two slots and a pool that holds little more than two of
    them: portions of one beside single tokens of another, requests that sit a step out, one
    that is released in the middle and fed again from its first token - every request's rows equal what
    it gives alone."""
    folder = folder_of(tmp_path_factory, "loop", sharpen=SHARPEN[dtype])
    lengths = {"a": 75, "b": 9, "c": 41, "d": 1, "e": 58, "f": 26}
    requests = {k: helpers.random_ids(vocab_of("loop"), n, i + 20)
                for i, (k, n) in enumerate(lengths.items())}
    steps, names = helpers.trace_mixed_with_recompute(requests, seed=5, max_live=2)
    need = helpers.live_tokens_needed(steps, round_to=16)
    runner = runner_for(folder, dtype, num_pages=need // 16, max_requests=2)
    rows = helpers.run_trace_in_process(runner, steps)
    assert len(rows) >= sum(lengths.values())
    assert_rows(rows, names, folder, bound)
    assert runner.cache.slots.num_free == 2
    assert all(free == need // 16 for free in runner.cache.free_pages())


def test_pages_behind_chunks_are_given_back(tmp_path_factory):
    """A request much longer than the pool: every cache group keeps a chunk's worth of pages, so 400
    tokens pass through pages for 96."""
    from from_scratch_inference_engine_b200 import LoadedModel, ModelRunner
    folder = folder_of(tmp_path_factory, "loop")
    requests = {"long": helpers.random_ids(vocab_of("loop"), 400, 8)}
    model = LoadedModel.from_pretrained(folder, dtype="float32", max_positions=512)
    runner = ModelRunner(model.model, model.runtime, page_size=16, num_pages=6, max_requests=2,
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
    assert all(free == 6 for free in runner.cache.free_pages())


def test_long_decoding_through_graphs_and_without(tmp_path_factory):
    """A short prompt, then 150 tokens one by one through captured graphs - chunks begin and end on
    decoded tokens many times; the same without graphs gives the same rows up to the order of the sums."""
    folder = folder_of(tmp_path_factory, "loop")
    requests = {"long": helpers.random_ids(vocab_of("loop"), 157, 9)}
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
    split ranges in the graph): the padding entry writes no page and changes nobody's rows."""
    folder = folder_of(tmp_path_factory, "wide", sharpen=False)
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
    folder = folder_of(tmp_path_factory, "loop", sharpen=SHARPEN[dtype])
    model = LoadedModel.from_pretrained(folder, dtype=dtype, max_positions=256)
    engine = Engine(model, block_size=16, num_blocks=16, max_batch=2, max_step_tokens=24)
    prompts = [helpers.random_ids(vocab_of("loop"), n, s) for n, s in ((45, 1), (7, 2), (30, 3))]
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
    assert type(load_config(folder)).__name__ == "DeginexConfig"
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


@pytest.mark.parametrize("dtype,name,bound", [("float32", "loop", F32_BOUND), ("bfloat16", "wide", BF16_BOUND)])
def test_trace_replay_program_runs_the_design(tmp_path_factory, tmp_path, dtype, name, bound):
    """bin/trace_run as a user runs it (a subprocess, steps on standard input, logits in files)
    on a mixed trace of five requests through four slots and a pool for the live tokens only."""
    import json
    import subprocess
    from pathlib import Path
    folder = folder_of(tmp_path_factory, name, sharpen=SHARPEN[dtype])
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


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_configurations_drawn_at_random(tmp_path_factory, seed):
    """Layers, sizes, chunks, caps, routers, streams and loops drawn at random (fixed seeds), in float32:
    a whole prompt, portions beside decoded tokens of other requests, and a tail token by token, against
    the plain implementation."""
    folder = dm.write_random(tmp_path_factory.mktemp(f"deginex_random{seed}"), seed)
    vocab = dm.CONFIGS[f"random{seed}"]["vocab"]
    requests = {"a": helpers.random_ids(vocab, 150, seed), "b": helpers.random_ids(vocab, 41, seed + 1),
                "c": helpers.random_ids(vocab, 67, seed + 2)}
    runner = runner_for(folder, "float32", num_pages=24)
    for steps in (helpers.trace_whole(requests), helpers.trace_mixed(requests, seed=seed, max_live=3),
                  helpers.trace_tail_by_one({"b": requests["b"]}, tail=30)):
        rows = helpers.run_trace_in_process(runner, steps)
        assert_rows(rows, requests, folder, F32_BOUND)
