"""Every mechanism of the Lizazen family alone, against the plain oracle (oracle/lizazen_ref.py): the bigram embedding with the
token before kept in slots, norms over whole projections with values taken from the raw keys, capped scores with a sink,
differential attention in all its kernels, chunked attention with values wider than the keys, retention with rotated fp32 keys,
the residual norm of two halves, routing without renormalisation, and experts weighted on their input beside a shared expert.
Sequences are fed in portions over shuffled pages whose foreign slots hold NaN; loud keys sit just inside and just outside
every window, kept prefix and chunk.  fp32 compares tightly; bf16 against the same oracle fed the rounded inputs."""
import math

import pytest
import torch

import lizazen_ref as R
import lizazen_util as U

pytestmark = pytest.mark.gpu

F64 = torch.float64
DTYPES = [torch.float32, torch.bfloat16]
NAN = float("nan")
PORTIONS = [[(1, 1), (0, 70)], [(1, 20), (0, 2)], [(0, 1), (1, 1)], [(1, 37), (0, 1)], [(0, 33)], [(0, 1), (1, 2)], [(0, 1)], [(0, 1)], [(0, 40)]]


def _ops():
    from b200attn import ops
    return ops


def _close(got, want, tol, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max() / (want.abs().max() + 1e-30))
    assert err <= tol, f"{what}: relative error {err:.3e} above {tol:.1e}"


def _rows(T, n, dt, seed, amp=1.0):
    return (torch.randn(T, n, generator=torch.Generator().manual_seed(seed)) * amp).to(dt)


def _pool(cuda, dt, n, G, bs, d):
    return torch.full((n, G, bs, d), NAN, dtype=dt, device=cuda)


def _tables(bs, lens, seed):
    perm = U.pages(sum(-(-n // bs) for n in lens) + 5, seed)
    out, at = [], 0
    for n in lens:
        out.append(perm[at:at - (-n // bs)])
        at += -(-n // bs)
    return out, len(perm)


# ------------------------------------------------------------------------------------------------ bigram embedding
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D", [30, 64, 1028])
@pytest.mark.parametrize("vocab,buckets,mp,mc", [(50, 31, 17, 5), (40, 1, 3, 2), (40, 97, 0, 1), (30, 64, 999999999989, 1000003)])
def test_bigram_embedding_in_portions(cuda, dt, D, vocab, buckets, mp, mc):
    """Three sequences share two slots one after the other (dirty with tokens of their own); cuts before, after and between
    tokens; products beyond 32 bits; padding rows leave their slot alone."""
    ops = _ops()
    b = {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}
    w = {"embed": _rows(vocab, D, dt, 1), "bigram": _rows(buckets + 1, D, dt, 2)}
    last = torch.tensor([7, 11, 13], dtype=torch.int64, device=cuda)
    seqs = [torch.tensor(U.tokens(n, vocab, 9 + n)) for n in (40, 23, 17)]

    def step(tok, batch, pos, _):
        return ops.embed_bigram(w["embed"].to(cuda), w["bigram"].to(cuda), tok, batch, mp, mc, last)
    first = U.feed(cuda, seqs[:2], [[(0, 1), (1, 5)], [(1, 1), (0, 30)], [(0, 2), (1, 17)], [(0, 1)], [(0, 6)]], step, slots=[0, 2])
    assert last.tolist() == [int(seqs[0][-1]), 11, int(seqs[1][-1])]
    second = U.feed(cuda, seqs[2:], [[(0, 1)], [(0, 1)], [(0, 15)]], step, slots=[2])
    w64 = {k: v.to(F64) for k, v in w.items()}
    for got, s in zip(first + second, seqs):
        assert got.dtype == torch.float32
        _close(got, R.embedding(s.tolist(), w64, b), 1e-6)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    batch = ops.SeqBatch(i32([0, 1, 2]), i32([3, -1]), None, i32([0, 0]), 2, 2)
    before = int(last[0])
    x = ops.embed_bigram(w["embed"].to(cuda), w["bigram"].to(cuda), torch.tensor([4, 0], device=cuda), batch, mp, mc, last)
    assert last.tolist()[0] == 4
    _close(x[0], w64["embed"][4] + w64["bigram"][R.bigram_row(before, 4, b)], 1e-6)


# ------------------------------------------------------------------------------------------------ capped window attention on its own keys
def _window_case(cuda, dt, H, G, dk, size, cap, rot, scale, bs, n_pages, eps=1e-4, seed=0):
    ops = _ops()
    g = torch.Generator().manual_seed(seed)
    qw, kw = 1 + 0.4 * torch.randn(H * dk, generator=g), 1 + 0.4 * torch.randn(G * dk, generator=g)
    sinks = 1.5 * torch.randn(H, generator=g)
    kc, vc = _pool(cuda, dt, n_pages, G, bs, dk), _pool(cuda, dt, n_pages, G, bs, dk)
    table = ops.rotary_table(2048, rot["dims"], rot["base"], rot.get("scaling"), cuda) if rot else None

    def step(x, batch, pos, slots):
        q = ops.qk_rope_cache(x, H, G, dk, dk, pos, table, rot["dims"] if rot else 0, slots, kc, vc, v_from_k=True, q_norm=qw.to(cuda),
                              k_norm=kw.to(cuda), eps=eps)
        return ops.chunk_attention(q, kc, vc, batch, scale, window=size, sink=1.0, sink_logits=sinks.to(cuda), softcap=cap)

    def oracle(rows, capped=True):
        T, r = rows.shape[0], rows.to(F64)
        k = r[:, H * dk:(H + G) * dk]
        q = R.rotate(R.rms_norm(r[:, :H * dk], qw.to(F64), eps).view(T, H, dk), rot)
        kr = R.rotate(R.rms_norm(k, kw.to(F64), eps).view(T, G, dk), rot)
        seen = R.mask_matrix(T, lambda i, j: R.in_window(i, j, size) if size else j <= i)
        return R.attention(q, kr, k.view(T, G, dk), seen, scale, cap if capped else None, sinks.to(F64))
    return step, oracle


@pytest.mark.parametrize("H,G,dk,bs", [(4, 1, 24, 16), (3, 3, 40, 8), (4, 2, 64, 16), (8, 1, 128, 32), (12, 1, 32, 16), (6, 3, 6, 8), (2, 2, 96, 16)])
@pytest.mark.parametrize("size,cap", [(0, 4.0), (1, 2.0), (9, 3.0), (16, 50.0), (17, 0.0), (64, 1.0), (500, 6.0)])
@pytest.mark.parametrize("dt", DTYPES)
def test_capped_attention_in_mixed_batches(cuda, H, G, dk, bs, size, cap, dt):
    """Scores of standard deviation ~3 under caps below and above them; the values are the raw keys, the keys normed and rotated."""
    rot = U.rot(dk // 2 // 2 * 2, 300.0, U.zones(4.0, 1.0, 4.0, 120))
    seqs = [_rows(150, (H + G) * dk, dt, H + dk), _rows(61, (H + G) * dk, dt, 99)]
    tables, n = _tables(bs, (150, 61), size + dk)
    step, oracle = _window_case(cuda, dt, H, G, dk, size, cap, rot, 3 * dk ** -0.5, bs, n, seed=dk)
    for o, rows in zip(U.feed(cuda, seqs, PORTIONS, step, bs, tables), seqs):
        want = oracle(rows)
        _close(o, want, 2e-5 if dt == torch.float32 else 2e-2, f"window {size} cap {cap}")
        if 0 < cap <= 4.0 and size != 1:
            assert float((oracle(rows, False) - want).abs().max() / want.abs().max()) > 0.1      # the cap matters


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dk", [(2, 1, 16), (4, 2, 64), (1, 1, 10)])
@pytest.mark.parametrize("loud,seen", [("window_in", True), ("window_out", False), ("far", True)])
@pytest.mark.parametrize("how", ["prompt", "portion", "decoded"])
def test_a_loud_key_at_the_window_edge(cuda, dt, H, G, dk, loud, seen, how):
    """One key matches the last row's query with a capped score of ~30 above everything else, sink included; at a page border, or 600
    positions back.  Seen: the output is that key as projected."""
    ops = _ops()
    bs, T = 16, 704
    size = 0 if loud == "far" else 64
    i = T - 1
    j = {"window_in": i - size + 1, "window_out": i - size, "far": 99}[loud]
    rows = _rows(T, (H + G) * dk, torch.float32, 7, 0.05)
    rows[j, H * dk:] = 0
    rows[i, :H * dk] = 0
    rows[j, H * dk + dk - 1::dk] = 6.0                               # an entry that does not turn
    rows[i, dk - 1:H * dk:dk] = 30.0
    rows = rows.to(dt)
    tables, n = _tables(bs, (T,), 3)
    kc, vc = _pool(cuda, dt, n, G, bs, dk), _pool(cuda, dt, n, G, bs, dk)
    sinks = torch.full((H,), -2.0, device=cuda)
    table = ops.rotary_table(1024, dk // 4 * 2, 1e4, None, cuda)

    def step(x, batch, pos, slots):
        q = ops.qk_rope_cache(x, H, G, dk, dk, pos, table, dk // 4 * 2, slots, kc, vc, v_from_k=True)
        return ops.chunk_attention(q, kc, vc, batch, 1.0, window=size, sink=1.0, sink_logits=sinks, softcap=30.0)
    steps = {"prompt": [T], "portion": [T - 2, 2], "decoded": [T - 1, 1]}[how]
    got = U.feed(cuda, [rows], [[(0, m)] for m in steps], step, bs, tables)[0][-1].double().cpu()
    value = rows[j, H * dk:].double().view(G, dk)
    for h in range(H):
        want = value[h // (H // G)]
        if seen:
            assert float((got[h] - want).abs().max()) <= 2e-2, f"head {h} ({loud}, {how})"
        else:
            assert float(got[h].abs().max()) <= 0.3


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T", [1, 40])
def test_a_sink_is_neither_scaled_nor_capped(cuda, dt, T):
    """Zero scores: n keys weigh 1 / (n + e^sink) each, for sinks far above the cap and far below it."""
    ops = _ops()
    H, G, dk, bs = 4, 2, 32, 16
    sinks = torch.tensor([0.0, 7.0, -60.0, 60.0])
    kc, vc = (torch.zeros(4, G, bs, dk, dtype=dt, device=cuda) for _ in range(2))
    vc += 1.0
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    batch = ops.SeqBatch(i32([0, T]), i32([0]), i32([[3, 1, 0]]), None, 1, T)
    o = ops.chunk_attention(torch.zeros(T, H, dk, dtype=dt, device=cuda), kc, vc, batch, 0.01, sink=1.0, sink_logits=sinks.to(cuda), softcap=2.0)
    n = torch.arange(1, T + 1, dtype=F64).view(T, 1, 1)
    _close(o, (n / (n + sinks.to(F64).exp().view(1, H, 1))).expand(T, H, dk), 1e-5 if dt == torch.float32 else 5e-3)


# ------------------------------------------------------------------------------------------------ differential attention
def _diff_case(cuda, dt, H, G, dk, dv, size, keep, rot, scale, lam, part, eps, bs, n_pages):
    ops = _ops()
    kc, vc = _pool(cuda, dt, n_pages, 2 * G, bs, dk), _pool(cuda, dt, n_pages, G, bs, dv)
    table = ops.rotary_table(2048, rot["dims"], rot["base"], rot.get("scaling"), cuda) if rot else None

    def step(x, batch, pos, slots):
        q = ops.qk_rope_cache(x, 2 * H, 2 * G, dk, dv, pos, table, rot["dims"] if rot else 0, slots, kc, vc)
        return ops.chunk_attention(q, kc, vc, batch, scale, window=size, keep_first=keep, maps=2, map_lambda=lam, map_eps=eps,
                                   map_scale=1.0 - part)

    def oracle(rows):
        T, r = rows.shape[0], rows.to(F64)
        a, b = 2 * H * dk, 2 * (H + G) * dk
        q, k = R.rotate(r[:, :a].view(T, H, 2, dk), rot), R.rotate(r[:, a:b].view(T, G, 2, dk), rot)
        seen = R.mask_matrix(T, lambda i, j: R.in_window_or_kept(i, j, size, keep) if size else j <= i)
        return R.differential_attention(q, k, r[:, b:].view(T, G, dv), seen, scale, lam, part, eps)
    return step, oracle


DIFF_SHAPES = [(3, 1, 16, 40, 16), (2, 2, 8, 4, 8), (4, 2, 32, 64, 16), (6, 1, 64, 128, 16), (2, 1, 128, 128, 32), (3, 3, 6, 10, 8), (4, 4, 96, 32, 16),
               (2, 1, 64, 256, 16), (12, 1, 32, 96, 16), (1, 1, 20, 12, 8)]


@pytest.mark.parametrize("H,G,dk,dv,bs", DIFF_SHAPES)
@pytest.mark.parametrize("size,keep", [(0, 0), (1, 0), (9, 3), (16, 16), (17, 40), (64, 20), (33, 0), (500, 4)])
@pytest.mark.parametrize("dt", DTYPES)
def test_differential_attention_in_mixed_batches(cuda, H, G, dk, dv, bs, size, keep, dt):
    rot = U.rot(dk // 2 // 2 * 2, 300.0)
    width = 2 * (H + G) * dk + G * dv
    seqs = [_rows(150, width, dt, H + dk + size), _rows(61, width, dt, 99)]
    tables, n = _tables(bs, (150, 61), size + dk)
    step, oracle = _diff_case(cuda, dt, H, G, dk, dv, size, keep, rot, 1.5 * dk ** -0.5, 0.45, 0.3, 1e-5, bs, n)
    for o, rows in zip(U.feed(cuda, seqs, PORTIONS, step, bs, tables), seqs):
        _close(o, oracle(rows), 5e-5 if dt == torch.float32 else 3e-2, f"window {size} + {keep}")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv", [(3, 1, 16, 24), (4, 2, 64, 64), (1, 1, 6, 10)])
@pytest.mark.parametrize("lam,part,eps", [(-0.7, 0.1, 1e-6), (0.0, 0.9, 1e-5), (1.6, 0.5, 1e-3), (0.98, 0.0, 2.0)])
def test_lambda_and_the_norm_of_the_difference(cuda, dt, H, G, dk, dv, lam, part, eps):
    """lambda negative, zero and above one; an eps that outweighs the difference's mean square."""
    width = 2 * (H + G) * dk + G * dv
    rows = _rows(90, width, dt, dk)
    tables, n = _tables(16, (90,), 1)
    step, oracle = _diff_case(cuda, dt, H, G, dk, dv, 40, 2, None, dk ** -0.5, lam, part, eps, 16, n)
    got = U.feed(cuda, [rows], [[(0, 60)], [(0, 2)]] + [[(0, 1)]] * 5 + [[(0, 23)]], step, 16, tables)[0]
    _close(got[8:], oracle(rows)[8:], 5e-5 if dt == torch.float32 else 4e-2)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv", [(2, 1, 16, 24), (4, 2, 64, 32), (8, 1, 32, 128)])
@pytest.mark.parametrize("loud,seen", [("window_in", True), ("window_out", False), ("first_in", True), ("first_out", False)])
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("how", ["prompt", "portion", "decoded"])
def test_a_loud_key_of_one_map(cuda, dt, H, G, dk, dv, loud, seen, which, how):
    """One key of one map stands out for the last row, just inside or outside the window or the kept prefix (page borders).  All values
    are small except that key's: seen, the head is the key's value, normed, with the sign of its map; unseen, it is not."""
    bs, T, size, keep = 16, 416, 64, 32
    i = T - 1
    j = {"window_in": i - size + 1, "window_out": i - size, "first_in": keep - 1, "first_out": keep}[loud]
    a, b = 2 * H * dk, 2 * (H + G) * dk
    rows = _rows(T, b + G * dv, torch.float32, 7, 0.05)
    rows[i, :a] = 0
    for h in range(H):
        rows[i, (2 * h + which) * dk + dk - 1] = 8.0
    rows[j, a:b] = 0
    for g in range(G):
        rows[j, a + (2 * g + which) * dk + dk - 1] = 6.0
    value = torch.randn(G, dv, generator=torch.Generator().manual_seed(5))
    rows[j, b:] = value.flatten()
    rows = rows.to(dt)
    tables, n = _tables(bs, (T,), 3)
    step, oracle = _diff_case(cuda, dt, H, G, dk, dv, size, keep, U.rot(dk // 2, 1e4), 1.0, 0.6, 0.2, 1e-6, bs, n)
    steps = {"prompt": [T], "portion": [T - 2, 2], "decoded": [T - 1, 1]}[how]
    got = U.feed(cuda, [rows], [[(0, m)] for m in steps], step, bs, tables)[0][-1].double().cpu()
    _close(got, oracle(rows)[-1], 1e-4 if dt == torch.float32 else 8e-2, f"{loud}, map {which}, {how}")
    unit = R.unit_rms(value.to(dt).to(F64), 1e-6) * 0.8 * (1 if which == 0 else -1)
    for h in range(H):
        off = float((got[h] - unit[h // (H // G)]).abs().max())
        assert off < 0.25 if seen else off > 0.5, f"head {h}: {off}"


def test_map_and_cap_arguments_are_checked(cuda):
    ops = _ops()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    batch = ops.SeqBatch(i32([0, 1]), i32([0]), i32([[0]]), None, 1, 1)
    kc, vc, q = torch.zeros(1, 2, 16, 8, device=cuda), torch.zeros(1, 1, 16, 8, device=cuda), torch.zeros(1, 4, 8, device=cuda)
    with pytest.raises(ValueError, match="maps"):
        ops.chunk_attention(q, kc, vc, batch, 1.0)
    with pytest.raises(ValueError, match="maps"):
        ops.chunk_attention(q[:, :3].contiguous(), kc, vc, batch, 1.0, maps=2)
    with pytest.raises(Exception, match="maps per head"):
        ops.chunk_attention(torch.zeros(1, 3, 8, device=cuda), torch.zeros(1, 3, 16, 8, device=cuda), vc, batch, 1.0, maps=3)
    with pytest.raises(Exception, match="cap"):
        ops.chunk_attention(q, vc, vc, batch, 1.0, softcap=2.0, weight_kind=ops.WEIGHT_SIGMOID)


# ------------------------------------------------------------------------------------------------ chunked attention, wide values
@pytest.mark.parametrize("H,G,dk,dv,bs", [(4, 2, 24, 16, 16), (2, 1, 64, 192, 16), (2, 2, 96, 256, 32), (4, 1, 128, 256, 16), (3, 1, 32, 160, 8),
                                          (1, 1, 14, 2, 8), (2, 1, 32, 192, 16), (8, 2, 96, 192, 16)])
@pytest.mark.parametrize("size", [1, 16, 17, 48, 400])
@pytest.mark.parametrize("dt", DTYPES)
def test_chunked_attention_with_wide_values(cuda, H, G, dk, dv, bs, size, dt):
    ops = _ops()
    rot = U.rot(dk // 2 // 2 * 2, 500.0)
    width = (H + G) * dk + G * dv
    seqs = [_rows(150, width, dt, H + dk), _rows(61, width, dt, 99)]
    tables, n = _tables(bs, (150, 61), size)
    kc, vc = _pool(cuda, dt, n, G, bs, dk), _pool(cuda, dt, n, G, bs, dv)
    table = ops.rotary_table(256, rot["dims"], rot["base"], None, cuda)

    def step(x, batch, pos, slots):
        q = ops.qk_rope_cache(x, H, G, dk, dv, pos, table, rot["dims"], slots, kc, vc)
        return ops.chunk_attention(q, kc, vc, batch, dk ** -0.5, size)
    for o, rows in zip(U.feed(cuda, seqs, PORTIONS, step, bs, tables), seqs):
        T, r = rows.shape[0], rows.to(F64)
        q, k = R.rotate(r[:, :H * dk].view(T, H, dk), rot), R.rotate(r[:, H * dk:(H + G) * dk].view(T, G, dk), rot)
        want = R.attention(q, k, r[:, (H + G) * dk:].view(T, G, dv), R.mask_matrix(T, lambda i, j: R.in_chunk(i, j, size)), dk ** -0.5)
        _close(o, want, 2e-5 if dt == torch.float32 else 1.5e-2, f"chunk {size}")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("dk,dv", [(16, 24), (64, 192), (96, 256)])
@pytest.mark.parametrize("row,key,seen", [("last", "first", True), ("first", "before", False), ("second", "first", True), ("last", "before", False)])
@pytest.mark.parametrize("how", ["prompt", "portion", "decoded"])
def test_a_loud_key_at_the_chunk_edge(cuda, dt, dk, dv, row, key, seen, how):
    """The chunk of 100 positions starts inside a page; the querying row is its first, second or last, the loud key its first or the
    one before."""
    ops = _ops()
    bs, size, H, G = 16, 100, 2, 1
    start = 300
    i = {"last": start + size - 1, "first": start, "second": start + 1}[row]
    j = start if key == "first" else start - 1
    T = i + 1
    rows = _rows(T, (H + G) * dk + G * dv, torch.float32, 3, 0.05)
    rows[i, :H * dk] = 0
    rows[j, H * dk:(H + G) * dk] = 0
    rows[i, dk - 1:H * dk:dk] = 6.0
    rows[j, (H + G) * dk - 1] = 6.0
    rows[j, (H + G) * dk:] = 1.0
    rows = rows.to(dt)
    tables, n = _tables(bs, (T,), 3)
    kc, vc = _pool(cuda, dt, n, G, bs, dk), _pool(cuda, dt, n, G, bs, dv)
    table = ops.rotary_table(512, dk // 2, 1e4, None, cuda)

    def step(x, batch, pos, slots):
        q = ops.qk_rope_cache(x, H, G, dk, dv, pos, table, dk // 2, slots, kc, vc)
        return ops.chunk_attention(q, kc, vc, batch, 1.0, size)
    steps = {"prompt": [T], "portion": [T - 2, 2], "decoded": [T - 1, 1]}[how]
    got = U.feed(cuda, [rows], [[(0, m)] for m in steps], step, bs, tables)[0][-1].double().cpu()
    assert float((got - 1.0).abs().max()) < 0.02 if seen else float(got.abs().max()) < 0.3


# ------------------------------------------------------------------------------------------------ retention
def _retention_step(cuda, H, dk, dv, decay, rot, eps, state):
    ops = _ops()
    table = ops.rotary_table(2048, rot["dims"], rot["base"], rot.get("scaling"), cuda) if rot else None
    d = torch.tensor(decay, dtype=torch.float32, device=cuda)
    n = 2 * H * dk + H * dv

    def step(x, batch, pos, _):
        qkv, beta, dec = ops.recur_prep(x[:, :n], H, H, dk, dv, batch, k_scale=dk ** -0.5, decay_mode=ops.DECAY_HEAD_CONST, decay_bias=d,
                                        cos_sin=table)
        assert beta is None and qkv.dtype == torch.float32
        s = ops.channel_scan(qkv, None, dec, H, H, dk, dv, batch, state, delta=False)
        return ops.gated_head_norm(s, x[:, n:n + H * dv], None, eps, ops.GATE_SILU)
    return step


def _retention_oracle(rows, H, dk, dv, decay, rot, eps):
    T, r, n = rows.shape[0], rows.to(F64), H * dk
    q, k = R.rotate(r[:, :n].view(T, H, dk), rot), R.rotate(r[:, n:2 * n].view(T, H, dk), rot) * dk ** -0.5
    o, _ = R.retention(q, k, r[:, 2 * n:2 * n + H * dv].view(T, H, dv), decay)
    return R.unit_rms(o, eps).reshape(T, H * dv) * R.silu(r[:, 2 * n + H * dv:2 * n + 2 * H * dv])


@pytest.mark.parametrize("H,dk,dv,dims", [(3, 16, 24, 8), (2, 20, 12, 0), (4, 64, 64, 64), (2, 128, 128, 32), (3, 10, 6, 10), (2, 96, 32, 64), (1, 8, 600, 2),
                                          (2, 256, 16, 256)])
@pytest.mark.parametrize("dt", DTYPES)
def test_retention_in_portions_over_dirty_slots(cuda, H, dk, dv, dims, dt):
    decay = [0.999, 0.5, 0.97, 1.0][:H]
    rot = U.rot(dims, 90.0) if dims else None
    width = 2 * H * (dk + dv)
    seqs = [_rows(150, width, dt, dk), _rows(61, width, dt, 9)]
    state = torch.full((3, H, dk, dv), 1e4, device=cuda)
    got = U.feed(cuda, seqs, PORTIONS, _retention_step(cuda, H, dk, dv, decay, rot, 1e-5, state), slots=[2, 0])
    assert bool((state[1] == 1e4).all())
    for o, rows in zip(got, seqs):
        _close(o, _retention_oracle(rows, H, dk, dv, decay, rot, 1e-5), 5e-5 if dt == torch.float32 else 1.5e-2)
    again = U.feed(cuda, [seqs[1]], [[(0, 61)]], _retention_step(cuda, H, dk, dv, decay, rot, 1e-5, state), slots=[2])[0]
    _close(again, got[1], 2e-5 if dt == torch.float32 else 1e-2, "the slot of another sequence")


@pytest.mark.parametrize("dt", DTYPES)
def test_retention_remembers_and_forgets(cuda, dt):
    """One loud token 700 single-token steps back: the head with decay 1 still answers it, the one with decay 0.95 has lost it."""
    H, dk, dv, T = 2, 16, 16, 760
    rows = _rows(T, 2 * H * (dk + dv), torch.float32, 1, 0.02)
    n = H * dk
    rows[59] = 0
    value = torch.randn(H * dv, generator=torch.Generator().manual_seed(2)) * 8
    rows[59, n + dk - 1:2 * n:dk] = 8.0
    rows[59, 2 * n:2 * n + H * dv] = value
    rows[T - 1, dk - 1:n:dk] = 5.0
    rows[:, 2 * n + H * dv:] = 20.0                                  # an open gate: silu(20) = 20
    rows = rows.to(dt)
    state = torch.full((1, H, dk, dv), NAN, device=cuda)
    rot = U.rot(dk // 2, 1e4)
    got = U.feed(cuda, [rows], [[(0, 58)]] + [[(0, 1)]] * (T - 58), _retention_step(cuda, H, dk, dv, [1.0, 0.95], rot, 1e-6, state), slots=[0])[0]
    want = _retention_oracle(rows, H, dk, dv, [1.0, 0.95], rot, 1e-6)
    _close(got, want, 1e-4 if dt == torch.float32 else 2e-2)
    unit = 20.0 * R.unit_rms(value.to(dt).to(F64).view(H, dv), 1e-6)
    last = got[-1].double().cpu().view(H, dv)
    assert float((last[0] - unit[0]).abs().max()) < 2.0 and float((last[1] - unit[1]).abs().max()) > 10.0


@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("unit", [False, True])
def test_rotation_in_the_recurrence_preparation(cuda, interleaved, unit):
    """Both pair layouts, beside unit vectors and scales, at positions far into a sequence."""
    ops = _ops()
    H, G, dk, dv, dims = 2, 2, 24, 8, 12
    rows = _rows(5, 2 * G * dk + H * dv, torch.float32, 4)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    batch = ops.SeqBatch(i32([0, 3, 5]), i32([1000, 0]), None, i32([0, 1]), 2, 5)
    qkv, _, _ = ops.recur_prep(rows.to(cuda), H, G, dk, dv, batch, unit=unit, unit_eps=1e-6, q_scale=2.0, k_scale=0.5,
                               decay_mode=ops.DECAY_HEAD_CONST, decay_bias=torch.ones(H, device=cuda),
                               cos_sin=ops.rotary_table(1100, dims, 40.0, None, cuda), interleaved=interleaved)
    x = rows.to(F64)[:, :2 * G * dk].view(5, 2 * G, dk)
    if unit:
        x = x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    perm = list(range(dk))
    if interleaved:                                                  # pairs (2i, 2i + 1) are the half layout on reordered entries
        perm = list(range(0, dims, 2)) + list(range(1, dims, 2)) + list(range(dims, dk))
    y = torch.empty_like(x)
    y[..., perm] = R.rotate(x[..., perm], U.rot(dims, 40.0), [1000, 1001, 1002, 0, 1])
    y[:, :G] *= 2.0
    y[:, G:] *= 0.5
    _close(qkv[:, :2 * G * dk].reshape(5, 2 * G, dk), y, 3e-6)


# ------------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D", [30, 64, 1028, 4096, 9000])
@pytest.mark.parametrize("post,pre", [(True, True), (True, False), (False, True)])
@pytest.mark.parametrize("slices", [False, True])
def test_residual_norm_of_two_halves(cuda, dt, D, post, pre, slices):
    """The halves differ by a factor of a thousand: each has its own root mean square.  Rows of their own, or odd column slices."""
    ops = _ops()
    g = torch.Generator().manual_seed(D)
    T, eps = 5, 1e-3
    off = 3 if slices else 0
    y1, y2 = _rows(T, D + off, dt, 1, 30.0), _rows(T, D + off, dt, 2, 0.03)
    x = torch.randn(T, D, generator=g)
    w1, w2, wp, wn = (1 + 0.3 * torch.randn(D, generator=g) for _ in range(4))
    xd = x.to(cuda)
    h = ops.sandwich_norm_pair(xd, y1.to(cuda)[:, off:], w1.to(cuda), y2.to(cuda)[:, off:], w2.to(cuda), 0.5, wp.to(cuda) if post else None,
                               wn.to(cuda) if pre else None, eps)
    y = 0.5 * (R.rms_norm(y1[:, off:].to(F64), w1.to(F64), eps) + R.rms_norm(y2[:, off:].to(F64), w2.to(F64), eps))
    want = x.to(F64) + (R.rms_norm(y, wp.to(F64), eps) if post else y)
    _close(xd, want, 2e-6)
    assert (h is not None) == pre
    if pre:
        assert h.dtype == dt
        _close(h, R.rms_norm(want, wn.to(F64), eps), 3e-6 if dt == torch.float32 else 1e-2)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,dv", [(3, 24), (2, 192), (1, 1000), (2, 514)])
def test_head_norm_without_a_weight(cuda, dt, H, dv):
    ops = _ops()
    o, gate = torch.randn(7, H, dv, generator=torch.Generator().manual_seed(dv)) * 4, _rows(7, H * dv + 2, dt, 3, 2.0)
    got = ops.gated_head_norm(o.to(cuda), gate.to(cuda)[:, 2:], None, 1e-4, ops.GATE_SILU)
    want = R.unit_rms(o.to(F64), 1e-4).reshape(7, H * dv) * R.silu(gate[:, 2:].to(F64))
    _close(got, want, 3e-6 if dt == torch.float32 else 1e-2)


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T", [1, 5, 40, 1100])
@pytest.mark.parametrize("E,top,D", [(5, 2, 64), (12, 1, 30), (3, 3, 48), (64, 6, 128)])
@pytest.mark.parametrize("dt", DTYPES)
def test_sigmoid_routing_without_renormalisation(cuda, dt, T, E, top, D):
    """The ids of the largest scores and the scores themselves; one token's logits saturate high, one's low."""
    ops = _ops()
    h, w = _rows(T, D, dt, T), _rows(E, D, dt, E, 2.0 * D ** -0.5)
    h[0] *= 40.0
    ids, wts = ops.moe_route(h.to(cuda), w.to(cuda), None, top, scoring=ops.ROUTE_SIGMOID_PLAIN, weight_scale=1.5)
    z = h.to(F64) @ w.to(F64).T
    got = z.gather(1, ids.long().cpu())
    _close(wts, 1.5 * R.sigmoid(got), 3e-6 if dt == torch.float32 else 1e-4)
    want = torch.topk(z, top, dim=-1).values
    clear = (R.sigmoid(want) - R.sigmoid(got)).abs().max()           # equal sets up to scores that fp32 cannot tell apart
    assert float(clear) < 1e-5 and all(len(set(r.tolist())) == top for r in ids)


@pytest.mark.parametrize("T,E,top,D,F", [(1, 5, 2, 64, 24), (7, 12, 1, 30, 22), (40, 3, 3, 48, 40), (70, 16, 4, 128, 16), (1100, 4, 2, 64, 32),
                                         (1030, 8, 2, 96, 40)])
@pytest.mark.parametrize("glu", ["silu", "relu_sq"])
@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("dt", DTYPES)
def test_experts_weighted_on_their_input(cuda, dt, T, E, top, D, F, glu, shared):
    """expert(w h) differs from w expert(h) for both activations; small batches run on the tiled kernels, large bf16 ones on grouped
    library products; the shared rows are a column slice."""
    ops = _ops()
    h = _rows(T, D, dt, 1, 2.0)
    wg, wu, wd = (_rows(E * a, b, dt, 5 + i, b ** -0.5).view(E, a, b) for i, (a, b) in enumerate(((F, D), (F, D), (D, F))))
    g = torch.Generator().manual_seed(T)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    wts = torch.rand(T, top, generator=g) * 0.6 + 0.05
    extra = _rows(T, D + 4, dt, 8)
    c = lambda t: t.to(cuda)      # noqa: E731
    gu = torch.cat([wg, wu], dim=1).contiguous() if glu == "silu" else None
    gud = c(gu) if gu is not None else None
    y = ops.moe_experts(c(h), c(ids), c(wts), gud[:, :F] if gu is not None else None, gud[:, F:] if gu is not None else c(wu), c(wd),
                        w_gate_up=gud, glu=ops.GLU_SILU if glu == "silu" else ops.FF_RELU_SQ, weight_on_input=True,
                        add=c(extra)[:, 4:] if shared else None)
    h64, want, plain = h.to(F64), torch.zeros(T, D, dtype=F64), torch.zeros(T, D, dtype=F64)
    for e in range(E):
        t, k = torch.where(ids == e)
        for scaled, acc in ((True, want), (False, plain)):
            s = wts[t, k].to(F64).unsqueeze(1)
            x = h64[t] * (s if scaled else 1.0)
            a, u = x @ wg[e].to(F64).T, x @ wu[e].to(F64).T
            o = (R.silu(a) * u if glu == "silu" else torch.clamp(u, min=0) ** 2) @ wd[e].to(F64).T
            acc.index_add_(0, t, o if scaled else s * o)
    assert float((want - plain).abs().max() / want.abs().max()) > 0.05
    if shared:
        want = want + extra[:, 4:].to(F64)
    _close(y, want, 5e-6 if dt == torch.float32 else 2e-2)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("limit", [0.3, 1.0, 7.0])
@pytest.mark.parametrize("ff", [22, 324])
def test_bounded_units(cuda, dt, limit, ff):
    from b200attn.lizazen import GLU_ALPHA
    ops = _ops()
    gu = _rows(6, 2 * ff, dt, ff, 4.0)
    gu[0, :4] = torch.tensor([limit, -limit, 50.0, -50.0]).to(dt)
    got = ops.glu_and_mul(gu.to(cuda), ops.GLU_CLAMPED, GLU_ALPHA, limit)
    _close(got, R.bounded_glu(gu[:, :ff].to(F64), gu[:, ff:].to(F64), limit), 3e-6 if dt == torch.float32 else 1e-2)
    assert math.isclose(GLU_ALPHA, 1.702)
