"""The Zasudra decoder in the engine against the plain implementation (``plain_zasudra.py``, float64): each mechanism
alone, whole prompts, token-by-token decoding, portions down to two tokens, unequal batches, pages and slots used again,
keys far away, at page borders and just inside and outside a chunk (in prompts and decoded), sinks, state carried over
hundreds of tokens, prompts in segments, decoding over key segments, several shapes, and greedy generation through the
entry point."""

import itertools
import math

import pytest
import torch

import helpers as H
import plain_zasudra as plain
import zasudra_cases as Z

pytestmark = pytest.mark.gpu
DTYPES = [pytest.param(torch.float32, id="f32"), pytest.param(torch.bfloat16, id="bf16")]
DEV = "cuda"


def case(tmp_path, name, seed, sharp=None, slow=False, decided=False):
    cfg = Z.CONFIGS[name] if sharp is None else Z.sharpen(Z.CONFIGS[name], sharp)
    if decided:
        cfg = Z.decided(cfg)
    W = Z.weights_for(cfg, seed, slow=slow)
    return cfg, W, Z.write_model(str(tmp_path), cfg, W)


def requests_for(cfg, lengths, seed):
    return {f"r{i}": H.random_tokens(cfg["vocab"], n, seed + i) for i, n in enumerate(lengths)}


def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def _rel(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max())


def _portions(sizes_of_steps):
    """For steps given as {slot: tokens}: (positions, q_start, slots, request of each token) per step, and per step the
    (slot, first, end) of every request's rows."""
    done = {}
    for sizes in sizes_of_steps:
        spans = []
        for s, n in sizes.items():
            spans.append((s, done.get(s, 0), done.get(s, 0) + n))
            done[s] = done.get(s, 0) + n
        yield (_i32([p for _s, a, b in spans for p in range(a, b)]), _i32([0] + list(itertools.accumulate(b - a for _s, a, b in spans))),
               _i32(list(sizes)), _i32([i for i, (_s, a, b) in enumerate(spans) for _ in range(a, b)]), spans)


STEPS = [{3: 1}, {3: 2, 1: 5}, {1: 1}, {3: 4, 1: 1}, {3: 1, 1: 2}, {3: 15, 1: 6}]          # even and odd portions, together and in turns


# ---- kernels alone ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, buckets, muls", [(37, 11, (5, 2)), (300, 1, (3, 4)), (1040, 997, (1000003, 998244353))], ids=str)
def test_bigram_embedding_carries_the_last_token(dtype, width, buckets, muls):
    """Two requests in slots that are not theirs by number; a request's first token takes the table's last row; products
    beyond 32 bits; other slots stay as they are."""
    from llm_pipeline_b200.ops import kernels
    vocab = 60
    gen = torch.Generator().manual_seed(width)
    W = {"embed": torch.randn(vocab, width, generator=gen).to(dtype), "bigram": torch.randn(buckets + 1, width, generator=gen).to(dtype)}
    tokens = {3: H.random_tokens(vocab, 23, 1), 1: H.random_tokens(vocab, 15, 2)}
    rule = {"buckets": buckets, "mul_prev": muls[0], "mul_cur": muls[1]}
    want = {s: plain.embed(t, W, rule) for s, t in tokens.items()}
    state = torch.full((5, 2), -7, dtype=torch.int32, device=DEV)
    state[[3, 1]] = 0
    table, bigram = W["embed"].to(DEV), W["bigram"].to(DEV)
    for positions, q_start, slots, request, spans in _portions(STEPS):
        ids = _i32([t for s, a, b in spans for t in tokens[s][a:b]])
        out = torch.empty(ids.numel(), width, device=DEV)
        kernels.embedding_bigram(ids, table, bigram, q_start, slots, positions, request, state, muls[0], muls[1], buckets, out)
        assert _rel(out, torch.cat([want[s][a:b] for s, a, b in spans])) < 1e-6
    assert (state[[0, 2, 4]] == -7).all()
    assert int(state[3, 22 & 1]) == tokens[3][22] and int(state[1, 14 & 1]) == tokens[1][14]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [54, 256, 3072, 5000])
def test_a_normed_addend_and_the_sum_itself_for_the_next_reader(dtype, width):
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(width)
    res, y, w = torch.randn(7, width, generator=gen) * 3.0, torch.randn(7, width, generator=gen) * 40.0, torch.randn(width, generator=gen)
    want = res.double() + plain.rms(y.double(), 1e-5, w.double())
    for delta in (y.to(DEV), y.to(DEV).to(dtype)):
        residual, out = res.to(DEV), torch.empty(7, width, device=DEV, dtype=dtype)
        kernels.add_norm_mix(residual, delta=delta, delta_weight=w.to(DEV), delta_eps=1e-5, out=out)
        tol = 1e-6 if delta.dtype == torch.float32 else 1e-2
        assert _rel(residual, want) < tol and _rel(out, want) < (tol if dtype == torch.float32 else 1e-2)
    # the general form and the one with the row in registers agree where a second norm follows
    second, residual = torch.randn(width, generator=gen), res.to(DEV)
    out = torch.empty(7, width, device=DEV, dtype=dtype)
    kernels.add_norm_mix(residual, delta=y.to(DEV), delta_weight=w.to(DEV), delta_eps=1e-5, weight=second.to(DEV), eps=1e-5, out=out)
    assert _rel(out, plain.rms(want, 1e-5, second.double())) < (1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 8), (3, 1, 10, 14, 6), (2, 2, 32, 32, 32), (6, 3, 20, 20, 0), (5, 5, 7, 3, 2), (16, 2, 128, 64, 64)], ids=str)
def test_row_norms_rotation_and_the_rows_write_alone(dtype, interleaved, sizes):
    """Norms over whole rows, the rotation of a part of every head, values from their own columns or the projected keys
    before norm and rotation, the [k | v] rows in their page slots; then a layer that has queries alone."""
    from llm_pipeline_b200.ops import kernels
    heads, kv_heads, dim, vdim, rot = sizes
    n, page, eps, base = 21, 8, 1e-5, 30.0
    gen = torch.Generator().manual_seed(dim)
    nq, nk = heads * dim, kv_heads * dim
    qw, kw = torch.randn(nq, generator=gen) * 0.3 + 1.0, torch.randn(nk, generator=gen) * 0.3 + 1.0
    pages_n = -(-n // page)
    order = torch.randperm(pages_n + 2, generator=gen)[:pages_n]
    slots = torch.tensor([int(order[t // page]) * page + t % page for t in range(n)], dtype=torch.int32, device=DEV)
    cos = sin = None
    if rot:
        inv = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], device=DEV)
        cos, sin = torch.empty(n, rot // 2, device=DEV), torch.empty(n, rot // 2, device=DEV)
        kernels.rope_tables(torch.arange(n, dtype=torch.int32, device=DEV), inv, 1.0, cos, sin)

    def turn(x):                                     # [n, heads, dim]
        if not rot:
            return x
        if interleaved:
            return plain.rotate_interleaved(x, rot, base)
        places = [c for i in range(rot // 2) for c in (i, i + rot // 2)] + list(range(rot, dim))        # pair (i, i + rot / 2) as neighbours
        back = [places.index(c) for c in range(dim)]
        return plain.rotate_interleaved(x[..., places], rot, base)[..., back]

    for keys_are_values, beside in itertools.product([False, True] if vdim == dim else [False], (4, 5)):     # rows of 16-byte pieces, and not
        width = nq + nk + (0 if keys_are_values else kv_heads * vdim)
        proj = torch.randn(n, width + beside, generator=gen) * 2.0       # a gate's columns follow
        P = proj.double()
        q = turn(plain.rms(P[:, :nq], eps, qw.double()).view(n, heads, dim))
        k = turn(plain.rms(P[:, nq:nq + nk], eps, kw.double()).view(n, kv_heads, dim))
        v = (P[:, nq:nq + nk] if keys_are_values else P[:, nq + nk:width]).reshape(n, kv_heads, vdim)
        pages = torch.full((pages_n + 2, kv_heads, page, dim + vdim), float("nan"), device=DEV, dtype=dtype)
        out = torch.empty(n, nq, device=DEV, dtype=dtype)
        v_at = nq if keys_are_values else nq + nk
        kernels.capped_rows_post(proj.to(DEV), qw.to(DEV), kw.to(DEV), eps, cos, sin, rot, interleaved, out, slots, pages, v_at, heads, kv_heads, dim, vdim)
        tol = 3e-6 if dtype == torch.float32 else 1e-2
        rows = pages.transpose(1, 2).reshape(-1, kv_heads, dim + vdim)[slots.long()]
        assert _rel(out, q.reshape(n, -1)) < tol and _rel(rows, torch.cat([k, v], dim=-1)) < tol
        assert torch.isnan(pages).sum() == pages.numel() - n * kv_heads * (dim + vdim)          # nothing else was written
    alone = torch.empty_like(out)
    kernels.capped_rows_post(proj[:, :nq].contiguous().to(DEV), qw.to(DEV), None, eps, cos, sin, rot, interleaved, alone, None, None, 0, heads, kv_heads, dim, vdim)
    assert _rel(alone, out.double().cpu()) < tol


def _attention_case(dtype, heads, kv_heads, dim, vdim, n, page, seed, chunk, sink, plant=None, rows=None, gate=None, scale=None):
    """Queries, keys and values as they enter the scores, written into shuffled pages; (engine output, plain output) for
    the token rows ``rows`` (all by default), launched as the portion they are."""
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(seed)
    q, k = torch.randn(n, heads, dim, generator=gen), torch.randn(n, kv_heads, dim, generator=gen)
    v, g = torch.randn(n, kv_heads, vdim, generator=gen), torch.randn(n, heads, generator=gen)
    sinks = torch.randn(heads, generator=gen) + 1.0 if sink == "learned" else torch.zeros(heads)
    if plant is not None:
        plant(q, k, v)
    q, k, v = (t.to(torch.bfloat16).float() for t in (q, k, v))
    scale = scale or 1.0 / math.sqrt(dim)
    want = plain.attend(q.double(), k.double(), v.double(), scale, chunk, sinks.double())
    if gate:
        want = want * torch.sigmoid(g.double())[..., None]
    want = want.reshape(n, -1)
    rows = list(range(n)) if rows is None else rows
    pages_n = -(-n // page)
    order = torch.randperm(pages_n + 3, generator=gen)[:pages_n]              # the request's pages lie anywhere in the pool
    pages = torch.full((pages_n + 3, kv_heads, page, dim + vdim), float("nan"))  # other pages hold what must never be read
    for t in range(n):
        pages[order[t // page], :, t % page] = torch.cat([k[t], v[t]], dim=-1)
    table = order.to(torch.int32).view(1, -1).clone()
    if chunk is not None:                                                      # pages no asked row sees are gone, as in the engine
        for p in range(min(rows) // chunk * chunk // page):
            pages[order[p]] = float("nan")
            table[0, p] = -1
    qd, pd = q.reshape(n, -1).to(DEV).to(dtype)[rows].contiguous(), pages.to(DEV).to(dtype)
    gd = g.to(DEV)[rows].contiguous() if gate else None
    sd, td = sinks.to(DEV), table.to(DEV)
    out = torch.empty(len(rows), heads * vdim, device=DEV, dtype=dtype)
    kernels.capped_attention(qd, pd, td, torch.zeros(len(rows), dtype=torch.int32, device=DEV), _i32(rows), out, heads, kv_heads, dim, vdim, 0, 0,
                             scale, 0.0, sink=sd, gate=gd, chunk=chunk or 0)
    got = out.float().cpu()
    if kernels.capped_mma_supports(dtype, dim, vdim) and rows == list(range(rows[0], rows[0] + len(rows))):
        per = kernels.capped_mma_tokens_per_tile(heads, kv_heads)
        tok0 = torch.arange(0, len(rows), per, dtype=torch.int32, device=DEV)
        reach = min(n, chunk + kernels.CAPPED_TILE_KEYS) if chunk else n
        ways = [(False, 0)]
        if len(rows) == 1:          # one row: also the warps sharing its keys, in one block and in segments with blocks of their own
            ways += [(True, 0), (True, -(-reach // kernels.CAPPED_SEGMENT_KEYS))]
        for split, segments in ways:
            for _ in range(2 if segments else 1):                              # twice: the counters are left as they were found
                tensor = torch.empty_like(out)
                kernels.capped_attention_mma(qd, pd, td, _i32([0, len(rows)]), _i32([rows[-1] + 1]), torch.zeros_like(tok0), tok0, tensor, heads, kv_heads,
                                             dim, vdim, 0, 0, scale, 0.0, sink=sd, gate=gd, split=split, chunk=chunk or 0, segments=segments)
                assert not torch.isnan(tensor).any(), "the tensor-core kernel read a row of a page that is gone"
                assert _rel(tensor, want[rows]) < 3e-2, ("tensor cores", split, segments)
    return got, want[rows]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 2, 16, 16, 40, "learned", False), (3, 3, 12, 20, None, 0.0, True), (6, 1, 48, 48, 9, "learned", True),
                                   (8, 2, 128, 128, 100, "learned", False), (2, 2, 96, 96, None, 0.0, True), (40, 2, 16, 64, 33, 0.0, True),
                                   (12, 3, 32, 128, 1, "learned", False), (5, 5, 10, 3, 64, 0.0, True), (1, 1, 64, 16, 65, "learned", True)], ids=str)
def test_chunked_and_gated_attention_alone(dtype, sizes):
    """Grouped heads, chunks shorter and longer than a page, of one token and none, learned and fixed sinks, a gate per
    head, over shuffled pages: a whole prompt, portions, single rows whose old pages are gone."""
    heads, kv_heads, dim, vdim, chunk, sink, gate = sizes
    for rows in (None, list(range(150, 200)), [150, 151, 199], [199], [100], [99], [64], [63]):
        got, want = _attention_case(dtype, heads, kv_heads, dim, vdim, 200, 16, 3, chunk, sink, rows=rows, gate=gate)
        assert not torch.isnan(got).any(), "a row of a page that is gone, or of another request, was read"
        assert _rel(got, want) < (1e-5 if dtype == torch.float32 else 2e-2), rows


@pytest.mark.parametrize("sizes", [(16, 8, 128, 128, None, 0.0, True), (8, 2, 48, 48, None, "learned", False), (4, 1, 64, 32, 700, "learned", True)], ids=str)
def test_single_rows_over_several_key_segments(sizes):
    heads, kv_heads, dim, vdim, chunk, sink, gate = sizes
    for row in (1500, 1279, 1280, 699, 700, 701, 255, 256, 0):
        got, want = _attention_case(torch.bfloat16, heads, kv_heads, dim, vdim, 1501, 16, 5, chunk, sink, rows=[row], gate=gate)
        assert _rel(got, want) < 2e-2, row


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk, page", [(40, 16), (16, 16), (33, 8), (5, 16)])
def test_a_key_just_inside_and_just_outside_a_chunk(dtype, chunk, page):
    """One key holds nearly all of a query's weight; whether it is the first key of the query's own chunk or the last of the
    chunk before decides the output. In a prompt and for single rows."""
    heads, kv_heads, dim, vdim, n = 2, 1, 32, 16, 170
    asked = {}
    for c in range(2, (n - 1) // chunk):
        first = c * chunk
        asked[first] = first - 1                      # the chunk's first token asks for the last key of the chunk before: unseen
        if chunk > 4 and first + 2 < n:
            asked[first + 2] = first                  # and a later one for the chunk's first key: seen
            asked[first + chunk - 1] = first          # the chunk's last token too
    asked = {i: j for i, j in list(asked.items())[:9] if i < n}

    def plant(q, k, v):
        for i, j in asked.items():
            q[i] = k[j, 0] * 40.0 / k[j, 0].norm()
        for j in set(asked.values()):
            k[j] = k[j] * 4.0 / k[j].norm() * math.sqrt(dim)

    rows = sorted(asked)
    whole, want = _attention_case(dtype, heads, kv_heads, dim, vdim, n, page, 7, chunk, 0.0, plant=plant)
    tol = 1e-4 if dtype == torch.float32 else 3e-2
    assert _rel(whole[rows], want[rows]) < tol
    # the premise, on the plain implementation: without chunks, or with chunks one longer, the asked rows differ much
    _, causal = _attention_case(dtype, heads, kv_heads, dim, vdim, n, page, 7, None, 0.0, plant=plant, rows=rows)
    outside = [r for r, i in enumerate(rows) if asked[i] // chunk != i // chunk]
    assert outside and (causal[outside] - want[rows][outside]).abs().max(dim=1).values.min() > 0.05
    inside = [i for i in rows if asked[i] // chunk == i // chunk]
    for i in inside[:2]:
        _, longer = _attention_case(dtype, heads, kv_heads, dim, vdim, n, page, 7, chunk + 1, 0.0, plant=plant, rows=[i])
        if asked[i] // (chunk + 1) != i // (chunk + 1):
            assert (longer[0] - want[i]).abs().max() > 0.05
    for i in rows:                                          # decoded alone: one row, old pages gone
        got, ref = _attention_case(dtype, heads, kv_heads, dim, vdim, n, page, 7, chunk, 0.0, plant=plant, rows=[i])
        assert _rel(got, ref) < tol, i


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sink_weighs_and_counts_once(dtype):
    """Scores near zero: the sink takes a share of the weight that shows, and it is the same however the keys are cut."""
    for n in (1, 2, 65, 600):
        got, want = _attention_case(dtype, 4, 2, 32, 32, n, 16, 9, None, "learned", rows=[n - 1], scale=0.01)
        assert _rel(got, want) < (1e-5 if dtype == torch.float32 else 2e-2), n
    gen = torch.Generator().manual_seed(1)
    q, k, v = torch.randn(3, 2, 8, generator=gen).double(), torch.randn(3, 1, 8, generator=gen).double(), torch.randn(3, 1, 8, generator=gen).double()
    low, high = (plain.attend(q, k, v, 1.0, None, torch.full((2,), s, dtype=torch.float64)) for s in (-50.0, 1.0))
    assert (low - high).abs().max() > 0.1 * low.abs().max()                    # the premise


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [54, 64, 1028])
def test_mixes_with_the_row_before_are_carried_from_step_to_step(dtype, width):
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(width)
    mu = torch.rand(5, width, generator=gen)
    xs = {3: torch.randn(23, width, generator=gen), 1: torch.randn(15, width, generator=gen)}
    want = {s: torch.stack([plain.token_shift(x.double(), mu[i].double()) for i in range(5)]) for s, x in xs.items()}
    offset = 4
    state = torch.full((5, offset + 2 * width + 3), 9.0, device=DEV)
    state[[3, 1]] = 0.0
    for positions, q_start, slots, request, spans in _portions(STEPS):
        rows = torch.cat([xs[s][a:b] for s, a, b in spans]).to(DEV)
        out = torch.empty(5, rows.shape[0], width, device=DEV, dtype=dtype)
        kernels.wkv_shift(rows, mu.to(DEV), state, offset, q_start, slots, positions, request, out)
        assert _rel(out, torch.cat([want[s][:, a:b] for s, a, b in spans], dim=1)) < (1e-6 if dtype == torch.float32 else 1e-2)
    assert (state[[0, 2, 4]] == 9.0).all() and (state[[3, 1], :offset] == 0.0).all() and (state[[3, 1], offset + 2 * width:] == 0.0).all()


@pytest.mark.parametrize("tokens, channels, rank", [(1, 40, 3), (17, 130, 12), (8, 256, 64), (70, 100, 150)])
def test_decays_alone(tokens, channels, rank):
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(rank)
    low, w2, w0 = torch.randn(tokens, rank, generator=gen), torch.randn(channels, rank, generator=gen) / math.sqrt(rank), torch.randn(channels, generator=gen) - 2.0
    want = torch.exp(-torch.exp(torch.tanh(low.double()) @ w2.double().T + w0.double()))
    wide = torch.full((tokens, rank + 3), float("nan"))
    wide[:, 2:2 + rank] = low
    out = kernels.wkv_decay(wide.to(DEV)[:, 2:2 + rank], w2.t().contiguous().to(DEV), w0.to(DEV), torch.empty(tokens, channels, device=DEV))
    assert _rel(out, want) < 1e-6


@pytest.mark.parametrize("sizes", [(3, 16), (2, 20), (1, 5), (2, 64), (1, 100), (2, 33), (1, 200), (5, 1), (2, 128)], ids=str)
def test_the_wkv_recurrence_alone(sizes, monkeypatch):
    """On given rows, whole, cut into portions down to one token, and in segments side by side, in a slot that is not the
    first; the state of other slots and the entries around the piece stay as they are."""
    from llm_pipeline_b200.ops import kernels
    heads, dim = sizes
    gen = torch.Generator().manual_seed(heads * dim)
    n, C = 75, heads * dim
    r, k, v = (torch.randn(n, C, generator=gen) for _ in range(3))
    w = torch.exp(-torch.exp(torch.randn(n, C, generator=gen) * 1.5 - 2.5))
    u = torch.randn(heads, dim, generator=gen)
    want, _ = plain.wkv_scan(*(t.double().view(n, heads, dim) for t in (r, k, v, w)), u.double())
    want = want.reshape(n, C)
    rd, kd, vd, wd, ud = (t.to(DEV) for t in (r, k, v, w, u))
    monkeypatch.setattr(kernels, "WKV_SEGMENT_TOKENS", 16)
    for cuts, segments in (((), 1), ((1,), 1), ((1, 2, 4, 9, 10, 41), 1), (tuple(range(1, n)), 1), ((), 5), ((5, 50), 3), ((2,), 7)):
        out = torch.full((n, C), float("nan"), device=DEV)
        offset, entries = 6, 2 * kernels.wkv_state_entries(heads, dim)
        state = torch.full((4, offset + entries + 3), 5.0, device=DEV)
        state[2] = 0.0
        edges = [0] + list(cuts) + [n]
        for lo, hi in zip(edges[:-1], edges[1:]):
            kernels.wkv_scan(rd[lo:hi], kd[lo:hi], vd[lo:hi], wd[lo:hi], ud, state, offset, _i32([0, hi - lo]), _i32([2]), _i32(list(range(lo, hi))),
                             out[lo:hi], heads, dim, segments)
        assert _rel(out, want) < 5e-6, (cuts, segments)
        assert (state[[0, 1, 3]] == 5.0).all() and (state[2, :offset] == 0.0).all() and (state[2, offset + entries:] == 0.0).all()


def test_the_wkv_recurrence_of_several_requests_at_once(monkeypatch):
    """Requests of unequal length in one step, from the states earlier steps left, with and without segments."""
    from llm_pipeline_b200.ops import kernels
    heads, dim = 2, 24
    C = heads * dim
    gen = torch.Generator().manual_seed(3)
    u = torch.randn(heads, dim, generator=gen)
    rows = {s: [torch.randn(n, C, generator=gen) for _ in range(3)] + [torch.rand(n, C, generator=gen)] for s, n in ((4, 60), (0, 1 + 33), (2, 2 + 8))}
    want = {s: plain.wkv_scan(*(t.double().view(-1, heads, dim) for t in x), u.double())[0].reshape(-1, C) for s, x in rows.items()}
    monkeypatch.setattr(kernels, "WKV_SEGMENT_TOKENS", 16)
    for segments in (1, 4):
        state = torch.zeros(5, 2 * kernels.wkv_state_entries(heads, dim), device=DEV)
        for positions, q_start, slots, _request, spans in _portions([{4: 7}, {0: 1, 2: 2}, {4: 53, 0: 33, 2: 8}]):
            args = [torch.cat([rows[s][i][a:b] for s, a, b in spans]).to(DEV) for i in range(4)]
            out = torch.empty(args[0].shape[0], C, device=DEV)
            kernels.wkv_scan(*args, u.to(DEV), state, 0, q_start, slots, positions, out, heads, dim, segments)
            assert _rel(out, torch.cat([want[s][a:b] for s, a, b in spans])) < 5e-6, segments


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim", [(3, 16), (2, 20), (1, 100), (3, 7), (1, 200), (4, 128)])
def test_heads_norm_and_gate_alone(dtype, heads, dim):
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(dim)
    n, C, eps = 9, heads * dim, 1e-5
    o, z, w = torch.randn(n, C, generator=gen) * 30.0, torch.randn(n, C, generator=gen) * 2.0, torch.randn(C, generator=gen) + 1.0
    want = plain.rms(o.double().view(n, heads, dim), eps).reshape(n, C) * w.double() * z.double() * torch.sigmoid(z.double())
    out = kernels.wkv_gate(o.to(DEV), z.to(DEV), w.to(DEV), torch.empty(n, C, device=DEV, dtype=dtype), heads, dim, eps)
    assert _rel(out, want) < (3e-6 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, width, experts, top", [(3, 64, 5, 2), (70, 54, 9, 4), (200, 256, 33, 8), (65, 40, 3, 3), (130, 48, 40, 1)])
def test_router_with_a_softmax_over_the_chosen_logits(dtype, tokens, width, experts, top):
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(experts)
    h, wr, b = torch.randn(tokens, width, generator=gen).to(dtype), torch.randn(experts, width, generator=gen) / math.sqrt(width), torch.randn(experts, generator=gen)
    ids = torch.full((tokens, top), -1, dtype=torch.int32, device=DEV)
    weights = torch.full((tokens, top), float("nan"), device=DEV)
    kernels.route_topk(h.to(DEV), wr.to(DEV), top, ids, weights, score="chosen_softmax", bias=b.to(DEV))
    chosen, want = plain.route(h.double(), wr.double(), b.double(), top)
    z = torch.sort(h.double() @ wr.double().T + b.double(), dim=-1, descending=True).values
    clear = (z[:, :min(top + 1, experts)].diff(dim=1).abs() > 1e-4).all(dim=1)          # no close call among the chosen and the next
    assert clear.float().mean() > 0.9
    assert torch.equal(ids.cpu().long()[clear], chosen[clear]) and _rel(weights.cpu()[clear], want[clear]) < 2e-5
    assert (weights.sum(dim=1) - 1.0).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, width, ff, experts, top", [(3, 64, 40, 5, 2), (90, 54, 22, 7, 5), (150, 72, 264, 4, 4), (300, 264, 136, 9, 1), (260, 64, 520, 3, 2)])
def test_squared_relu_experts_alone(dtype, tokens, width, ff, experts, top):
    """Every kernel that serves the sizes: a warp per output entry, the mma.sync and the tcgen05 grouped products; experts
    nobody chose, and one that everybody chose."""
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(ff)
    W = {f"f.e{e}.{n}": (torch.randn(*s, generator=gen) / math.sqrt(s[1])).to(torch.bfloat16).float()
         for e in range(experts) for n, s in (("up", (ff, width)), ("down", (width, ff)))}
    h = torch.randn(tokens, width, generator=gen).to(torch.bfloat16).float()
    ids = torch.stack([torch.randperm(experts, generator=gen)[:top] for _ in range(tokens)])
    if experts > top:
        ids[ids == experts - 1] = torch.where((ids == 0).any(dim=1, keepdim=True).expand_as(ids), ids, torch.zeros_like(ids))[ids == experts - 1]
    wts = torch.rand(tokens, top, generator=gen) + 0.1
    want = torch.zeros(tokens, width, dtype=torch.float64)
    for t in range(tokens):
        for e, w in zip(ids[t].tolist(), wts[t].double()):
            want[t] += w * (W[f"f.e{e}.down"].double() @ torch.relu(W[f"f.e{e}.up"].double() @ h[t].double()) ** 2)
    up = torch.stack([W[f"f.e{e}.up"] for e in range(experts)]).to(DEV).to(dtype)
    down = torch.stack([W[f"f.e{e}.down"] for e in range(experts)]).to(DEV).to(dtype)
    args = (h.to(DEV).to(dtype), up, down, ids.to(torch.int32).to(DEV), wts.to(DEV), 0.0)
    ways = [kernels.expert_rows]
    if kernels.expert_grouped_supports(dtype, width, ff):
        ways.append(kernels.expert_grouped)
    if kernels.expert_tc_supports(dtype, width, ff):
        ways.append(kernels.expert_tc)
    assert len(ways) == (1 if dtype == torch.float32 or width % 8 or ff % 8 else 3)
    for fn in ways:
        out = torch.full((tokens, width), float("nan"), device=DEV)
        fn(*args, out, "relu_squared")
        assert _rel(out, want) < (1e-5 if dtype == torch.float32 else 1.5e-2), fn.__name__
    torch.cuda.synchronize()
    kernels.check_error_flag()


@pytest.mark.parametrize("form, limit, identity", [("silu", 0.0, 3), ("clamped", 2.0, 0)])
def test_tcgen05_experts_of_the_other_forms(form, limit, identity):
    """Gate and up rows in one tile, identity experts left out of the sorted order, against the kernel of the few rows."""
    from llm_pipeline_b200.ops import kernels
    gen = torch.Generator().manual_seed(identity)
    tokens, width, ff, experts, top = 333, 136, 200, 6, 3
    h = torch.randn(tokens, width, generator=gen).to(torch.bfloat16).to(DEV)
    gu = (torch.randn(experts, 2 * ff, width, generator=gen) / math.sqrt(width) * 2.0).to(torch.bfloat16).to(DEV)
    down = (torch.randn(experts, width, ff, generator=gen) / math.sqrt(ff)).to(torch.bfloat16).to(DEV)
    ids = torch.stack([torch.randperm(experts + identity, generator=gen)[:top] for _ in range(tokens)]).to(torch.int32).to(DEV)
    wts = (torch.rand(tokens, top, generator=gen) + 0.1).to(DEV)
    a, b = (torch.full((tokens, width), float("nan"), device=DEV) for _ in range(2))
    kernels.expert_rows(h, gu, down, ids, wts, limit, a, form)
    kernels.expert_tc(h, gu, down, ids, wts, limit, b, form, identity)
    assert _rel(b, a.double().cpu()) < 1e-2
    torch.cuda.synchronize()
    kernels.check_error_flag()


# ---- one layer of each kind ------------------------------------------------------------------------------------------
ONE_LAYER = {
    "chunked": Z.config([Z.chunked(4, 2, 16, 12, 8, mlp=Z.moe(40, 4, 2))], width=40, vocab=50),
    "chunked, bare": Z.config([Z.chunked(3, 1, 12, 5, 12)], width=24, vocab=50, bigram=None),
    "no chunk, no rotation": Z.config([Z.chunked(2, 2, 16, None, None)], width=24, vocab=50),
    "wkv": Z.config([Z.wkv(3, 16, mlp=Z.moe(24, 3, 1))], width=40, vocab=50),
    "wkv, bare": Z.config([Z.wkv(2, 11)], width=30, vocab=50, bigram=None),
    "causal": Z.config([Z.causal(4, 2, 16, 24, mlp=Z.moe(40, 4, 4))], width=40, vocab=50),
    "causal twice": Z.config([Z.causal(4, 1, 12, 20), Z.causal(4, 1, 12, 20, kv_from=0, mlp=Z.moe(16, 3, 2))], width=32, vocab=50),
}


@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_one_layer_alone(tmp_path, name):
    cfg = ONE_LAYER[name]
    W = Z.weights_for(cfg, 11)
    folder = Z.write_model(str(tmp_path), cfg, W)
    requests = requests_for(cfg, [1, 2, 33, 70], 50)
    want = Z.oracle(cfg, W, requests)
    runner = H.make_runner(folder, torch.float32, page_size=8, num_pages=24, max_request_tokens=96, max_requests=2)
    Z.assert_matches(H.replay(runner, H.cut_whole(requests)), want, torch.float32, f"{name}, whole")
    Z.assert_matches(H.replay(runner, H.cut_portions(requests, (2, 5, 1, 16))), want, torch.float32, f"{name}, portions")


# ---- whole models ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(Z.CONFIGS))
def test_prefill_decoding_portions_and_batches(tmp_path, name, dtype):
    cfg, W, folder = case(tmp_path, name, 3)
    requests = requests_for(cfg, [1, 2, 3, 19, 64, 65, 150], 100)
    want = Z.oracle(cfg, W, requests)
    page = 8
    share = 1.0 if dtype == torch.float32 else 0.97     # bfloat16: a router's close call may fall the other way
    runner = H.make_runner(folder, dtype, page_size=page, num_pages=2 * (-(-150 // page)) + 6, max_request_tokens=160, max_requests=4)
    Z.assert_matches(H.replay(runner, H.cut_whole(requests)), want, dtype, f"{name}: whole prompts", share)
    Z.assert_matches(H.replay(runner, H.cut_tail_one_by_one(requests, tail=40)), want, dtype, f"{name}: last tokens one by one", share)
    Z.assert_matches(H.replay(runner, H.cut_portions(requests, (1,))), want, dtype, f"{name}: token by token", share)
    Z.assert_matches(H.replay(runner, H.cut_portions(requests, (2, 7, 3, 64, 2, 33))), want, dtype, f"{name}: portions", share)
    # unequal requests side by side, four live at most, so the slots and pages of finished ones go to later ones
    got = H.replay(runner, H.cut_mixed(requests, (2, 5, 16, 3, 31), max_live=4, decode_tail=9))
    Z.assert_matches(got, want, dtype, f"{name}: mixed batches", share)
    assert runner.cache.num_live == 0                                   # seven requests went through four slots
    assert runner.cache.pages_reused > 0 or all(layer["type"] == "wkv" for layer in cfg["layers"])


def test_the_same_logits_alone_and_in_a_batch(tmp_path):
    """float32: a request's logits beside others, or cut into portions, are those it has alone, to rounding of sums."""
    cfg, W, folder = case(tmp_path, "mixed", 4)
    requests = requests_for(cfg, [5, 40, 77, 130], 200)
    runner = H.make_runner(folder, torch.float32, page_size=16, num_pages=24, max_request_tokens=144, max_requests=4)
    alone = H.replay(runner, H.cut_whole(requests))
    mixed = H.replay(runner, H.cut_mixed(requests, (3, 2, 17), max_live=4, decode_tail=5))
    for rid in requests:
        assert (alone[rid] - mixed[rid]).abs().max() < 2e-4 * alone[rid].abs().max(), rid


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "causal_first", "wide_heads"])
def test_far_keys_page_borders_and_chunk_edges_under_a_sharp_softmax(tmp_path, name, dtype):
    """Scores of a wide spread: a query's weight sits on one or two keys, often hundreds of tokens back (the causal layers) or
    at a chunk's far edge, so a key that is lost, off by one or read from another request's page changes the logits by its
    whole value. Prompts as long as many pages, positions around every page border, decoded alone and in portions while
    chunks begin and end over decoded tokens and pages go back."""
    cfg, W, folder = case(tmp_path, name, 5, sharp=4.0, decided=dtype == torch.bfloat16)
    page = 16
    requests = requests_for(cfg, [4 * page, 4 * page + 1, 330, 17], 300)
    want = Z.oracle(cfg, W, requests)
    # the premise: in the plain implementation itself the far keys matter (without the first 3 pages the late logits differ much)
    late = plain.forward(cfg, W, requests["r2"][3 * page:]).float()
    assert Z.row_errors(late[-40:], want["r2"][-40:]).median() > 0.03
    runner = H.make_runner(folder, dtype, page_size=page, num_pages=2 * 21 + 4, max_request_tokens=336, max_requests=4)
    share = 1.0 if dtype == torch.float32 else 0.95
    Z.assert_matches(H.replay(runner, H.cut_whole(requests)), want, dtype, "sharp: whole", share)
    Z.assert_matches(H.replay(runner, H.cut_tail_one_by_one(requests, tail=3 * page + 2)), want, dtype, "sharp: decoding across borders", share)
    Z.assert_matches(H.replay(runner, H.cut_portions(requests, (page - 1, 2, page + 1, 2 * page, 3))), want, dtype, "sharp: portions", share)
    Z.assert_matches(H.replay(runner, H.cut_mixed(requests, (page, 2, page + 1), max_live=3, decode_tail=page + 3)), want, dtype, "sharp: mixed", share)


def test_a_chunk_that_ends_gives_its_pages_back(tmp_path):
    """While a request decodes, the pages of the chunks before its own return to the pool and go to the next request; the
    logits stay those of the plain implementation."""
    from llm_pipeline_b200.engine import StepEntry
    cfg = Z.sharpen(Z.config([Z.chunked(4, 2, 16, 20, 8, mlp=Z.moe(24, 3, 2)), Z.chunked(2, 2, 16, 20, 16)], width=40, vocab=50), 3.0)
    W = Z.weights_for(cfg, 21)
    folder = Z.write_model(str(tmp_path), cfg, W)
    requests = requests_for(cfg, [150, 90], 70)
    want = Z.oracle(cfg, W, requests)
    page = 8
    runner = H.make_runner(folder, torch.float32, page_size=page, num_pages=10, max_request_tokens=160, max_requests=2)   # 10 pages: 80 tokens
    got = {rid: [] for rid in requests}
    for rid, toks in requests.items():
        out = runner.step([StepEntry(rid, toks[:30], list(range(30)))])
        got[rid].append(out.float().cpu())
    for t in range(30, 150):
        live = [rid for rid, toks in requests.items() if t < len(toks)]
        out = runner.step([StepEntry(rid, [requests[rid][t]], [0]) for rid in live])
        for k, rid in enumerate(live):
            got[rid].append(out[k:k + 1].float().cpu())
        if t == 87:
            first = 80 // page                                              # token 88 is of the chunk that begins with token 80
            table = list(runner.cache.block_table("r1", 0))
            assert all(p < 0 for p in table[:first]) and all(p >= 0 for p in table[first:])
        if t == 89:
            runner.release("r1")
        runner.cache.check()
    assert runner.cache.pages_reused > 0
    Z.assert_matches({rid: torch.cat(rows) for rid, rows in got.items()}, want, torch.float32, "chunks over decoded tokens")


def test_states_carry_what_was_written_hundreds_of_tokens_back(tmp_path):
    """Decays close to one: what the first tokens wrote into the states still weighs in the logits 300 tokens later, so a
    state that is lost, zeroed at a cut or taken from another slot shows. Checked whole, in portions and in mixed batches."""
    cfg = Z.CONFIGS["wkv_only"]
    W = Z.weights_for(cfg, 12, slow=True)
    folder = Z.write_model(str(tmp_path), cfg, W)
    requests = requests_for(cfg, [320, 301, 47], 900)
    want = Z.oracle(cfg, W, requests)
    other = list(requests["r0"])
    other[:8] = H.random_tokens(cfg["vocab"], 8, 77)                    # the premise: the first tokens still matter at the end
    assert Z.row_errors(plain.forward(cfg, W, other).float()[-20:], want["r0"][-20:]).median() > 0.01
    runner = H.make_runner(folder, torch.float32, page_size=16, num_pages=50, max_request_tokens=336, max_requests=3)
    Z.assert_matches(H.replay(runner, H.cut_whole(requests)), want, torch.float32, "long memory: whole")
    Z.assert_matches(H.replay(runner, H.cut_portions(requests, (2, 63, 1, 130, 5))), want, torch.float32, "long memory: portions")
    Z.assert_matches(H.replay(runner, H.cut_mixed(requests, (40, 2, 9), max_live=2, decode_tail=20)), want, torch.float32, "long memory: mixed")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_in_segments_and_decoding_over_key_segments(tmp_path, dtype, monkeypatch):
    """Prompts long enough for the recurrence's segments and the grouped expert products, and contexts long enough for the
    causal layers' key segments in decoding, eager and replayed; sharp enough that a far key shows."""
    from llm_pipeline_b200.ops import kernels
    cfg = Z.sharpen(Z.config([Z.causal(4, 2, 16, 16, mlp=Z.moe(32, 4, 2)), Z.wkv(2, 24), Z.chunked(4, 2, 32, 300, 16, mlp=Z.moe(24, 3, 1)),
                              Z.causal(4, 2, 16, 16, kv_from=0)], width=48, vocab=90), 2.5)
    W = Z.weights_for(cfg, 31)
    folder = Z.write_model(str(tmp_path), cfg, W)
    requests = requests_for(cfg, [700, 640], 500)
    want = Z.oracle(cfg, W, requests)
    used = {"segments": 0, "keys": 0}
    scan, attend = kernels.wkv_scan, kernels.capped_attention_mma

    def counted_scan(*args, **kwargs):
        used["segments"] += args[13] > 1
        return scan(*args, **kwargs)

    def counted_attend(*args, **kwargs):
        used["keys"] += kwargs.get("segments", 0) > 1
        return attend(*args, **kwargs)

    monkeypatch.setattr(kernels, "wkv_scan", counted_scan)
    monkeypatch.setattr(kernels, "capped_attention_mma", counted_attend)
    runner = H.make_runner(folder, dtype, page_size=16, num_pages=90, max_request_tokens=720, max_requests=2)
    share = 1.0 if dtype == torch.float32 else 0.97
    Z.assert_matches(H.replay(runner, H.cut_whole(requests)), want, dtype, "long: whole", share)
    Z.assert_matches(H.replay(runner, H.cut_portions(requests, (513, 2, 61, 1))), want, dtype, "long: portions", share)
    Z.assert_matches(H.replay(runner, H.cut_mixed(requests, (520, 33), max_live=2, decode_tail=30)), want, dtype, "long: side by side", share)
    assert used["segments"] > 0 and (used["keys"] > 0) == (dtype == torch.bfloat16) and runner.graph_replays > 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_replayed_graphs(tmp_path, dtype):
    """Two requests decode side by side for 220 steps over many pages and chunks, the states, the rows before and the last
    tokens taking turns between their two copies: from the third step on a captured graph is replayed."""
    cfg, W, folder = case(tmp_path, "mixed", 6, decided=dtype == torch.bfloat16)
    requests = requests_for(cfg, [260, 231], 400)
    want = Z.oracle(cfg, W, requests)
    runner = H.make_runner(folder, dtype, page_size=16, num_pages=40, max_request_tokens=272, max_requests=2)
    from llm_pipeline_b200.engine import StepEntry
    rows = {rid: [] for rid in requests}
    out = runner.step([StepEntry(rid, toks[:11], list(range(11))) for rid, toks in requests.items()])
    for k, rid in enumerate(requests):
        rows[rid].append(out[11 * k:11 * (k + 1)].float().cpu())
    for t in range(11, 231):
        out = runner.step([StepEntry(rid, [toks[t]], [0]) for rid, toks in requests.items()])
        for k, rid in enumerate(requests):
            rows[rid].append(out[k:k + 1].float().cpu())
    assert runner.graph_replays > 200
    share = 1.0 if dtype == torch.float32 else 0.97
    for rid in requests:
        Z.assert_matches({rid: torch.cat(rows[rid])}, {rid: want[rid][:231]}, dtype, f"long decoding of {rid}", share)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(tmp_path, dtype):
    """Through the scheduler, the sampler and steps whose tokens the host has not seen yet (the bigram's previous token is
    carried on the device)."""
    from llm_pipeline_b200.inference import InferenceConfig, InferenceEngine
    cfg, W, folder = case(tmp_path, "causal_first" if dtype == torch.float32 else "mixed", 7)
    engine = InferenceEngine(InferenceConfig(model_path=folder, dtype=dtype, block_size=8, num_blocks=64, max_sequence_length=128,
                                             max_batch_size=4, max_num_batched_tokens=32))
    prompts = [H.random_tokens(cfg["vocab"], n, 600 + n) for n in (1, 7, 30, 45, 12)]       # five requests for four slots
    got = engine.generate(prompts, max_tokens=10, temperature=0.0)
    checked = 0
    for prompt, tokens in zip(prompts, got):
        ids = list(prompt)
        for token in tokens:
            logits = plain.forward(cfg, W, ids)[-1]
            top2 = torch.topk(logits, 2).values
            if dtype == torch.bfloat16 and float(top2[0] - top2[1]) < 0.04 * float(logits.std()) * 4:
                break                                                   # a near tie: the two sequences may part here
            assert token == int(logits.argmax()), (len(prompt), len(ids) - len(prompt))
            ids.append(token)
            checked += 1
    assert checked >= (50 if dtype == torch.float32 else 20)
    assert engine.engine.cache.num_live == 0
    info = engine.get_model_info()
    assert info["vocab_size"] == cfg["vocab"] and info["num_layers"] == len(cfg["layers"]) and info["total_parameters"] > 0


def test_generation_with_a_preempted_request(tmp_path):
    """Too few pages for all requests: one is preempted and computed again, its state and last token from nothing."""
    from llm_pipeline_b200.inference import InferenceConfig, InferenceEngine
    cfg, W, folder = case(tmp_path, "mixed", 8)
    engine = InferenceEngine(InferenceConfig(model_path=folder, dtype=torch.float32, block_size=8, num_blocks=12, max_sequence_length=64,
                                             max_batch_size=3, max_num_batched_tokens=32))
    prompts = [H.random_tokens(cfg["vocab"], n, 700 + n) for n in (25, 27, 21)]
    got = engine.generate(prompts, max_tokens=16, temperature=0.0)
    for prompt, tokens in zip(prompts, got):
        ids = list(prompt)
        for token in tokens:
            assert token == int(plain.forward(cfg, W, ids)[-1].argmax())
            ids.append(token)
        assert len(tokens) == 16
    assert engine.engine.cache.num_live == 0
