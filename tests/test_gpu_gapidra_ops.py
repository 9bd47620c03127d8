"""Every mechanism of the Gapidra family alone, against the plain oracle (oracle/gapidra_ref.py): the norm over whole
projections before the rotation, sigmoid-weighted attention with a bias per head, the sink per head of latent attention in
all its kernels, the latent write in the half layout, the gate per channel, the joint input of the output projection with
xIELU.  Sequences are fed in portions over shuffled pages whose foreign slots hold NaN; one loud key sits just inside or
just outside every window.  fp32 compares tightly; bf16 against the same oracle fed the rounded inputs."""
import math

import pytest
import torch

import gapidra_ref as R
import gapidra_util as U

pytestmark = pytest.mark.gpu

F64 = torch.float64
DTYPES = [torch.float32, torch.bfloat16]
NAN = float("nan")


def _ops():
    from b200attn import ops
    return ops


def _close(got, want, tol, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max() / (want.abs().max() + 1e-30))
    assert err <= tol, f"{what}: relative error {err:.3e} above {tol:.1e}"


def _rot(dims, base, scaling=None):
    return {"dims": dims, "base": base, "scaling": scaling}


# ------------------------------------------------------------------------------------------------ joint projection input
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n_mix,n_ff,pad", [(40, 72, 0), (12, 20, 4), (13, 30, 1), (0, 64, 0), (48, 0, 8), (7, 0, 0), (1024, 4100, 0)])
@pytest.mark.parametrize("rows", ["all", "some", "none"])
def test_parallel_join(cuda, dt, n_mix, n_ff, pad, rows):
    """Gated heads beside xIELU units, both column ranges of wider rows; the heads' columns of rows past the gated ones stay
    as another kernel left them."""
    ops = _ops()
    g = torch.Generator().manual_seed(n_mix + n_ff)
    T, p, q = 9, 0.6, -0.4
    k = {"all": T, "some": 4, "none": 0}[rows]
    wide = (torch.randn(T, n_mix + n_ff + pad, generator=g) * 5).to(dt)
    if n_ff:
        z = torch.tensor([0.0, -0.0, 1e-3, -1e-3, 30.0, -90.0, 7.5, -7.5])
        wide[0, n_mix:n_mix + min(8, n_ff)] = z[:min(8, n_ff)].to(dt)
    mix = torch.randn(T, max(n_mix, 1), generator=g).to(dt)[:, :n_mix]
    out = torch.full((T, n_mix + n_ff), 77.0, dtype=dt, device=cuda)
    w = wide.to(cuda)
    a, b = R.softplus(p), 0.5 + R.softplus(q)
    ops.parallel_join(out, mix.to(cuda)[:k] if k else None, w[:k, :n_mix] if k else None, n_mix,
                      w[:, n_mix:n_mix + n_ff] if n_ff else None, ops.FF_XIELU, a, b)
    tol = 2e-6 if dt == torch.float32 else 6e-3
    if n_mix and k:
        _close(out[:k, :n_mix], mix[:k].to(F64) * R.sigmoid(wide[:k, :n_mix].to(F64)), tol, "gated heads")
    assert bool((out[k:, :n_mix] == 77.0).all())
    if n_ff:
        want = R.xielu(wide[:, n_mix:n_mix + n_ff].to(F64), p, q)
        _close(out[:, n_mix:], want, tol, "xielu")
        small = want.abs() < 0.1                                    # no cancellation near zero
        d = (out[:, n_mix:].double().cpu() - want).abs()[small]
        assert d.numel() == 0 or float(d.max()) <= (2e-7 if dt == torch.float32 else 5e-4)
    # without a gate the heads pass; squared ReLU is the other activation
    if n_mix and n_ff:
        ops.parallel_join(out, mix.to(cuda), None, n_mix, w[:, n_mix:n_mix + n_ff], ops.FF_RELU_SQ)
        assert torch.equal(out[:, :n_mix].cpu(), mix)
        _close(out[:, n_mix:], torch.clamp(wide[:, n_mix:n_mix + n_ff].to(F64), min=0) ** 2, tol)


# ------------------------------------------------------------------------------------------------ norm, rotation, pool write
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,dims", [(4, 1, 24, 16, 12), (6, 3, 6, 10, 2), (2, 2, 16, 16, 0), (5, 5, 40, 12, 20), (8, 1, 128, 64, 96),
                                            (3, 3, 16, 28, 16), (1, 1, 14, 2, 6)])
@pytest.mark.parametrize("layout", ["interleaved", "half"])
@pytest.mark.parametrize("pad", [3, 8])
def test_norm_over_whole_projections_then_rotation(cuda, dt, H, G, dk, dv, dims, layout, pad):
    """One head of q and one of k are far larger than the others, so a norm per head would show; positions up to 4999 with a
    scaled rotation; a token with a negative slot is rotated but not cached."""
    ops = _ops()
    g = torch.Generator().manual_seed(dk + H)
    T, bs, eps, scaling = 60, 8, 1e-4, U.yarn(4.0, 700, 10.0, 1.0)
    rows = torch.randn(T, (H + G) * dk + G * dv + pad, generator=g)
    rows[:, :dk] *= 9.0
    rows[:, H * dk:H * dk + dk] *= 5.0
    rows[7] *= 1e-3                                                # eps matters here
    rows = rows.to(dt)
    qw, kw = 1 + 0.4 * torch.randn(H * dk, generator=g), 1 + 0.4 * torch.randn(G * dk, generator=g)
    table = ops.rotary_table(5000, dims, 800.0, scaling, cuda) if dims else None
    pool = 12
    kc = torch.full((pool, G, bs, dk), NAN, dtype=dt, device=cuda)
    vc = torch.full((pool, G, bs, dv), NAN, dtype=dt, device=cuda)
    pos = torch.arange(T, dtype=torch.int32) * 84                    # 0 .. 4956
    slots = torch.randperm(pool * bs, generator=g)[:T]
    slots[5] = -1
    q = ops.qk_rope_cache(rows.to(cuda), H, G, dk, dv, pos.to(cuda), table, dims, slots.to(cuda), kc, vc,
                          interleaved=layout == "interleaved", q_norm=qw.to(cuda), k_norm=kw.to(cuda), eps=eps)
    r = rows.to(F64)
    qn = R.rms_norm(r[:, :H * dk], qw.to(F64), eps).view(T, H, dk)
    kn = R.rms_norm(r[:, H * dk:(H + G) * dk], kw.to(F64), eps).view(T, G, dk)
    big = lambda x: torch.zeros(4957, *x.shape[1:], dtype=F64).index_copy_(0, pos.long(), x)     # noqa: E731  (row t -> its position)
    tol = 4e-6 if dt == torch.float32 else 1e-2
    rot = _rot(dims, 800.0, scaling) if dims else None
    _close(q, R.rotate(big(qn), rot, layout)[pos.long()], tol, "queries")
    want_k = R.rotate(big(kn), rot, layout)[pos.long()]
    kf, vf = kc.permute(0, 2, 1, 3).reshape(pool * bs, G, dk).cpu(), vc.permute(0, 2, 1, 3).reshape(pool * bs, G, dv).cpu()
    kept = [t for t in range(T) if t != 5]
    _close(kf[slots[kept]], want_k[kept], tol, "keys")
    assert torch.equal(vf[slots[kept]], rows[kept, (H + G) * dk:(H + G) * dk + G * dv].view(-1, G, dv))
    free = sorted(set(range(pool * bs)) - {int(s) for s in slots[kept]})
    assert bool(torch.isnan(kf[free]).all()) and bool(torch.isnan(vf[free]).all()), "no other slot is written"


# ------------------------------------------------------------------------------------------------ sigmoid attention
def _sigmoid_case(dt, H, G, dk, dv, T, seed, amp=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(T, (H + G) * dk + G * dv, generator=g) * amp).to(dt)


def _sigmoid_step(cuda, H, G, dk, dv, bs, kc, vc, rot_dims, base, scale, window, bias, out_pad=0):
    ops = _ops()
    table = ops.rotary_table(2048, rot_dims, base, None, cuda) if rot_dims else None

    def step(x, batch, pos, slots):
        q = ops.qk_rope_cache(x, H, G, dk, dv, pos, table, rot_dims, slots, kc, vc, interleaved=True)
        wide = torch.full((x.shape[0], H * dv + out_pad), 55.0, dtype=x.dtype, device=cuda)
        ops.chunk_attention(q, kc, vc, batch, scale, window=window, weight_kind=ops.WEIGHT_SIGMOID, head_bias=bias,
                            out=wide[:, :H * dv])
        assert bool((wide[:, H * dv:] == 55.0).all())
        return wide[:, :H * dv].reshape(-1, H, dv)
    return step


def _sigmoid_oracle(rows, H, G, dk, dv, rot_dims, base, scale, window, bias):
    T, r = rows.shape[0], rows.to(F64)
    rot = _rot(rot_dims, base) if rot_dims else None
    q = R.rotate(r[:, :H * dk].view(T, H, dk), rot, "interleaved")
    k = R.rotate(r[:, H * dk:(H + G) * dk].view(T, G, dk), rot, "interleaved")
    return R.sigmoid_attention(q, k, r[:, (H + G) * dk:].view(T, G, dv), scale, window, bias.to(F64))


def _pools(cuda, dt, n, G, bs, dk, dv):
    return (torch.full((n, G, bs, dk), NAN, dtype=dt, device=cuda), torch.full((n, G, bs, dv), NAN, dtype=dt, device=cuda))


@pytest.mark.parametrize("H,G,dk,dv,bs", [(4, 1, 24, 16, 16), (3, 3, 40, 12, 8), (4, 2, 64, 32, 16), (8, 1, 128, 64, 32), (12, 1, 32, 96, 16),
                                          (2, 1, 6, 10, 8), (2, 2, 96, 128, 16)])
@pytest.mark.parametrize("window", [0, 1, 9, 16, 17, 64, 500])
@pytest.mark.parametrize("dt", DTYPES)
def test_sigmoid_attention_in_mixed_batches_over_shuffled_pages(cuda, H, G, dk, dv, bs, window, dt):
    """A sequence of 150 tokens in portions of 70, 2, 1, 1, 33, ..., beside a second one of other portions: every row equals the
    oracle over the whole sequence.  The output rows are a column range of a wider buffer."""
    T, T2, scale, base = 150, 61, dk ** -0.5, 300.0
    dims = dk // 2 // 2 * 2
    seqs = [_sigmoid_case(dt, H, G, dk, dv, T, H + dk + window), _sigmoid_case(dt, H, G, dk, dv, T2, 99)]
    bias = torch.linspace(-3.0, 1.0, H)
    n1, n2 = -(-T // bs), -(-T2 // bs)
    perm = U.pages(n1 + n2 + 5, window + dk)
    kc, vc = _pools(cuda, dt, n1 + n2 + 5, G, bs, dk, dv)
    sched = [[(1, 1), (0, 70)], [(1, 20), (0, 2)], [(0, 1), (1, 1)], [(1, 37), (0, 1)], [(0, 33)], [(0, 1), (1, 2)], [(0, 1)], [(0, 1)],
             [(0, 40)]]
    step = _sigmoid_step(cuda, H, G, dk, dv, bs, kc, vc, dims, base, scale, window, bias.to(cuda), out_pad=8)
    got = U.feed(cuda, seqs, [perm[:n1], perm[n1:n1 + n2]], bs, sched, step)
    for o, rows in zip(got, seqs):
        _close(o, _sigmoid_oracle(rows, H, G, dk, dv, dims, base, scale, window, bias), 2e-5 if dt == torch.float32 else 1.5e-2,
               f"window {window}")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv", [(2, 1, 16, 24), (4, 2, 64, 32)])
@pytest.mark.parametrize("loud,seen", [("window_in", True), ("window_out", False), ("far", True)])
@pytest.mark.parametrize("how", ["prompt", "portion", "decoded"])
def test_a_loud_key_weighs_one_inside_the_window_and_nothing_outside(cuda, dt, H, G, dk, dv, loud, seen, how):
    """Every score but one is near zero and the heads' biases are far below: all weights are ~1e-9, the loud key's ~1.  It sits on
    the last position the window still holds, on the first it has dropped (both at a page border), or 600 positions back
    without a window; the row is the last of a prompt, of a two-token portion, or a single decoded token."""
    bs, T = 16, 704
    window = 0 if loud == "far" else 64
    i = T - 1
    j = {"window_in": i - window + 1, "window_out": i - window, "far": 99}[loud]
    rows = _sigmoid_case(dt, H, G, dk, dv, T, 7, 0.1)
    rows[j, H * dk:(H + G) * dk] = 0
    rows[i, :H * dk] = 0
    for g_ in range(G):
        rows[j, H * dk + g_ * dk + dk - 1] = 6.0                    # an entry that does not turn
    for h in range(H):
        rows[i, h * dk + dk - 1] = 7.0
    bias = torch.full((H,), -20.0)
    perm = U.pages(50, 3)
    kc, vc = _pools(cuda, dt, 50, G, bs, dk, dv)
    steps = {"prompt": [T], "portion": [T - 2, 2], "decoded": [T - 1, 1]}[how]
    step = _sigmoid_step(cuda, H, G, dk, dv, bs, kc, vc, dk // 2, 1e4, 1.0, window, bias.to(cuda))
    got = U.feed(cuda, [rows], [perm[:44]], bs, [[(0, n)] for n in steps], step)[0][-1].double().cpu()
    value = rows[j, (H + G) * dk:].double().view(G, dv)
    for h in range(H):
        want = value[h // (H // G)] if seen else torch.zeros(dv, dtype=F64)
        assert float((got[h] - want).abs().max()) <= (2e-3 if dt == torch.float32 else 5e-3), f"head {h} ({loud}, {how})"


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv", [(3, 1, 16, 8), (2, 2, 64, 64)])
def test_sigmoid_weights_are_not_shares(cuda, dt, H, G, dk, dv):
    """n equal keys give n times one key's output (nothing is normalised), for prompt rows and single rows; a large score saturates
    at weight one, however large; padding rows are zero; no sink goes with these weights."""
    ops = _ops()
    bs, T = 16, 80
    rows = torch.zeros(T, (H + G) * dk + G * dv)
    rows[:, (H + G) * dk:] = 0.25
    bias = torch.linspace(-1.0, 2.0, H)
    kc, vc = _pools(cuda, dt, 6, G, bs, dk, dv)
    step = _sigmoid_step(cuda, H, G, dk, dv, bs, kc, vc, 0, 1.0, 0.5, 48, bias.to(cuda))
    got = U.feed(cuda, [rows.to(dt)], [U.pages(6, 1)[:5]], bs, [[(0, 64)]] + [[(0, 1)]] * 16, step)[0]
    n = torch.arange(1, T + 1, dtype=F64).clamp(max=48).view(T, 1, 1)
    _close(got, n * 0.25 * R.sigmoid(bias.to(F64)).view(1, H, 1).expand(T, H, dv), 1e-6 if dt == torch.float32 else 5e-3)
    rows[:, :(H + G) * dk] = 40.0                                   # scores of 12800 and more
    kc, vc = _pools(cuda, dt, 6, G, bs, dk, dv)
    step = _sigmoid_step(cuda, H, G, dk, dv, bs, kc, vc, 0, 1.0, 0.5, 48, bias.to(cuda))
    got = U.feed(cuda, [rows.to(dt)], [U.pages(6, 2)[:5]], bs, [[(0, 64)]] + [[(0, 1)]] * 16, step)[0]
    _close(got, n * 0.25 * torch.ones(T, H, dv, dtype=F64), 1e-6 if dt == torch.float32 else 5e-3)
    rows[:, :H * dk] = -40.0
    step = _sigmoid_step(cuda, H, G, dk, dv, bs, kc, vc, 0, 1.0, 0.5, 48, bias.to(cuda))
    got = U.feed(cuda, [rows.to(dt)], [U.pages(6, 2)[:5]], bs, [[(0, 64)]] + [[(0, 1)]] * 16, step)[0]
    assert float(got.abs().max()) == 0.0
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    batch = ops.SeqBatch(i32([0, 1, 2]), i32([10, -1]), i32([[U.pages(6, 2)[0]], [0]]), None, 2, 2)
    q = torch.randn(2, H, dk, device=cuda).to(dt)
    o = ops.chunk_attention(q, kc, vc, batch, 0.5, weight_kind=ops.WEIGHT_SIGMOID, head_bias=bias.to(cuda))
    assert bool((o[1] == 0).all()) and bool(torch.isfinite(o[0]).all())
    with pytest.raises(Exception, match="sink"):
        ops.chunk_attention(q, kc, vc, batch, 0.5, weight_kind=ops.WEIGHT_SIGMOID, sink=1.0)
    with pytest.raises(Exception, match="bias"):
        ops.chunk_attention(q, kc, vc, batch, 0.5, head_bias=bias.to(cuda))


# ------------------------------------------------------------------------------------------------ latent attention with sinks
class _Latent:
    """One latent layer's tensors and a step function: latent_prep in the half layout, absorbed queries, attention, W_uv."""

    def __init__(self, cuda, dt, H, dn, dr, dv, Rk, scale, window, base, bs, n_pages, seed):
        g = torch.Generator().manual_seed(seed)
        self.__dict__.update(cuda=cuda, dt=dt, H=H, dn=dn, dr=dr, dv=dv, Rk=Rk, scale=scale, window=window, base=base, bs=bs)
        self.nw = 1 + 0.2 * torch.randn(Rk, generator=g)
        self.w_uk = (torch.randn(H * dn, Rk, generator=g) * Rk ** -0.5).to(dt)
        self.w_uv = (torch.randn(H * dv, Rk, generator=g) * Rk ** -0.5).to(dt)
        self.sinks = 1.5 * torch.randn(H, generator=g)
        self.cache = torch.full((n_pages, bs, Rk + dr), NAN, dtype=dt, device=cuda)
        self.eps = 1e-5

    def rows(self, T, seed, amp=1.0):
        g = torch.Generator().manual_seed(seed)
        return (torch.randn(T, self.H * (self.dn + self.dr) + self.Rk + self.dr, generator=g) * amp).to(self.dt)

    def step(self, x, batch, pos, slots):
        ops = _ops()
        H, dn, dr, dv, Rk = self.H, self.dn, self.dr, self.dv, self.Rk
        nq, T = H * (dn + dr), x.shape[0]
        table = ops.rotary_table(2048, dr, self.base, None, self.cuda)
        qa = ops.latent_prep(x, H, dn, dr, dr, Rk, 0, nq, self.nw.to(self.cuda), self.eps, pos, table, slots, self.cache, interleaved=False)
        torch.bmm(x[:, :nq].view(T, H, dn + dr)[:, :, :dn].transpose(0, 1), self.w_uk.to(self.cuda).view(H, dn, Rk),
                  out=qa[:, :, :Rk].transpose(0, 1))
        o = ops.latent_attention(qa, self.cache, batch, Rk, self.scale, self.window, sink_logits=self.sinks.to(self.cuda))
        return torch.bmm(o.transpose(0, 1), self.w_uv.to(self.cuda).view(H, dv, Rk).transpose(1, 2)).transpose(0, 1).contiguous()

    def parts(self, rows):
        H, dn, dr, Rk = self.H, self.dn, self.dr, self.Rk
        T, r, nq = rows.shape[0], rows.to(F64), self.H * (self.dn + self.dr)
        rot = _rot(dr, self.base)
        q = r[:, :nq].view(T, H, dn + dr)
        q = torch.cat([q[..., :dn], R.rotate(q[..., dn:], rot, "half")], -1)
        c = R.rms_norm(r[:, nq:nq + Rk], self.nw.to(F64), self.eps)
        return q, c, R.rotate(r[:, nq + Rk:], rot, "half")

    def oracle(self, rows, sinks=True):
        q, c, kt = self.parts(rows)
        k, v = R.latent_keys_values(c, kt, self.w_uk.to(F64), self.w_uv.to(F64), self.H)
        return R.softmax_attention(q, k, v, self.scale, self.window, self.sinks.to(F64) if sinks else None)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,dn,dr,Rk", [(3, 16, 8, 24), (2, 8, 12, 20), (3, 6, 6, 14), (4, 32, 16, 64), (5, 4, 4, 12)])
@pytest.mark.parametrize("interleaved", [False, True])
def test_latent_write_in_both_layouts(cuda, dt, H, dn, dr, Rk, interleaved):
    ops = _ops()
    L = _Latent(cuda, dt, H, dn, dr, 8, Rk, 0.2, 0, 90.0, 8, 9, dn + Rk)
    rows, T = L.rows(61, 5), 61
    slots = torch.randperm(72, generator=torch.Generator().manual_seed(1))[:T]
    slots[3] = -1
    qa = ops.latent_prep(rows.to(cuda), H, dn, dr, dr, Rk, 0, H * (dn + dr), L.nw.to(cuda), L.eps,
                         torch.arange(T, dtype=torch.int32, device=cuda), ops.rotary_table(64, dr, 90.0, None, cuda), slots.to(cuda),
                         L.cache, interleaved=interleaved)
    layout, r, nq, tol = "interleaved" if interleaved else "half", rows.to(F64), H * (dn + dr), 3e-6 if dt == torch.float32 else 1e-2
    _close(qa[:, :, Rk:], R.rotate(r[:, :nq].view(T, H, dn + dr)[..., dn:], _rot(dr, 90.0), layout), tol, "rotated query parts")
    flat = L.cache.view(72, Rk + dr).cpu()
    kept = [t for t in range(T) if t != 3]
    _close(flat[slots[kept], :Rk], R.rms_norm(r[:, nq:nq + Rk], L.nw.to(F64), L.eps)[kept], tol, "latent")
    _close(flat[slots[kept], Rk:], R.rotate(r[:, nq + Rk:], _rot(dr, 90.0), layout)[kept], tol, "shared key part")
    free = sorted(set(range(72)) - {int(s) for s in slots[kept]})
    assert bool(torch.isnan(flat[free]).all())


LATENT_SHAPES = [(3, 16, 8, 20, 24), (6, 32, 16, 32, 64), (20, 16, 32, 16, 128), (3, 48, 48, 16, 256), (2, 16, 64, 24, 512), (70, 8, 16, 8, 64)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,dn,dr,dv,Rk", LATENT_SHAPES)
@pytest.mark.parametrize("window", [0, 1, 9, 16, 40])
def test_latent_attention_with_sinks_in_mixed_batches(cuda, dt, H, dn, dr, dv, Rk, window):
    """Whole prompts, portions down to two rows, single rows beside portions, and decode-only steps of one and two rows (whose
    keys are shared out over CTAs: the sink still counts once)."""
    L = _Latent(cuda, dt, H, dn, dr, dv, Rk, (dn + dr) ** -0.5, window, 200.0, 16, 34, H + window)
    seqs = [L.rows(230, 1), L.rows(47, 2)]
    perm = U.pages(34, H)
    sched = [[(0, 60), (1, 1)], [(1, 30), (0, 2)], [(0, 1), (1, 1)], [(1, 1), (0, 100)], [(0, 1)], [(0, 1), (1, 1)], [(0, 3), (1, 13)], [(0, 61)],
             [(0, 1)]]
    got = U.feed(cuda, seqs, [perm[:15], perm[15:18]], 16, sched, L.step)
    for o, rows in zip(got, seqs):
        _close(o, L.oracle(rows), 3e-5 if dt == torch.float32 else 3e-2, f"R={Rk} window {window}")
        assert float((L.oracle(rows, sinks=False) - L.oracle(rows)).abs().max()) > 0.05       # the sinks matter


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("Rk,H", [(24, 3), (64, 6), (128, 20), (512, 2)])
@pytest.mark.parametrize("how", ["prompt", "decoded"])
def test_sinks_far_above_and_far_below(cuda, dt, Rk, H, how):
    """A head whose sink dwarfs the scores gives nothing, one whose sink vanishes gives the ordinary softmax, one in between its share;
    700 keys, so single rows are split over CTAs."""
    L = _Latent(cuda, dt, H, 16, 16, 16, Rk, 0.2, 0, 300.0, 16, 50, 4)
    L.sinks = torch.full((H,), 60.0)
    L.sinks[0] = -60.0
    L.sinks[1] = math.log(700.0)
    rows = L.rows(700, 3)
    steps = [700] if how == "prompt" else [697, 1, 1, 1]
    got = U.feed(cuda, [rows], [U.pages(50, 2)[:44]], 16, [[(0, n)] for n in steps], L.step)[0][-3:]
    plain, want = L.oracle(rows, sinks=False)[-3:], L.oracle(rows)[-3:]
    tol = 3e-5 if dt == torch.float32 else 3e-2
    _close(got[:, 0], plain[:, 0], tol)
    _close(got[:, 1], want[:, 1], tol)
    assert float(want[:, 1].abs().max()) < 0.8 * float(plain[:, 1].abs().max())
    assert H == 2 or float(got[:, 2:].abs().max()) < 1e-6


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,Rk,dr", [(3, 24, 8), (4, 64, 16), (20, 128, 32)])
@pytest.mark.parametrize("edge", ["inside", "outside"])
@pytest.mark.parametrize("how", ["prompt", "portion", "decoded"])
def test_a_loud_latent_at_the_window_edge(cuda, dt, H, Rk, dr, edge, how):
    """The last row's query matches one key far better than the sink and all others; with the edge on a page border.  Inside: the
    output is that key's value; outside: the loud key does not show."""
    window, T = 48, 208
    L = _Latent(cuda, dt, H, 16, dr, 16, Rk, 1.0, window, 1e5, 16, 16, 3)
    rows = L.rows(T, 8, 0.2)
    i = T - 1
    j = i - window + (1 if edge == "inside" else 0)                  # 160 | 159
    nq = H * (16 + dr)
    rows[i, :nq] = 0
    rows[j, nq + Rk:] = 0
    for h in range(H):
        rows[i, h * (16 + dr) + 16 + dr - 1] = 6.0                   # the slowest pair: 1e5^(-(dr - 2) / dr) per step
    rows[j, nq + Rk + dr - 1] = 6.0
    perm = U.pages(16, 5)
    steps = {"prompt": [T], "portion": [T - 2, 2], "decoded": [T - 1, 1]}[how]
    got = U.feed(cuda, [rows], [perm[:13]], 16, [[(0, n)] for n in steps], L.step)[0]
    want = L.oracle(rows)
    _close(got, want, 3e-5 if dt == torch.float32 else 3e-2)
    _, c, _ = L.parts(rows)
    value = (c[j] @ L.w_uv.to(F64).T).view(H, 16)
    d = (got[-1].double().cpu() - value).abs().amax(-1)
    assert bool((d < 0.05).all()) if edge == "inside" else bool((d > 0.05).all())


# ------------------------------------------------------------------------------------------------ per-head prompt path
@pytest.mark.parametrize("H,dn,dr,dv,Rk", [(3, 16, 16, 32, 64), (5, 8, 24, 48, 24), (4, 128, 64, 128, 64), (2, 24, 8, 16, 40)])
@pytest.mark.parametrize("window", [0, 1, 40, 64, 150])
def test_window_attention_with_sinks_and_a_gate_per_channel(cuda, H, dn, dr, dv, Rk, window):
    """Prompt portions over per-head keys and values (bf16): sink per head, one gate column per output channel, output rows inside a
    wider buffer whose other columns stay."""
    ops = _ops()
    bf = torch.bfloat16
    L = _Latent(cuda, bf, H, dn, dr, dv, Rk, (dn + dr) ** -0.5, window, 500.0, 16, 40, H + dn)
    seqs, cuts = [L.rows(260, 1), L.rows(90, 2)], [(130, 130), (70, 20)]
    g = torch.Generator().manual_seed(window)
    gates = [(2 * torch.randn(s.shape[0], H * dv + 8, generator=g)).to(bf) for s in seqs]
    perm = U.pages(40, 9)
    tables = [perm[:17], perm[17:23]]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    nq = H * (dn + dr)
    for half in (0, 1):
        lens = [c[half] for c in cuts]
        ctx = [0 if half == 0 else c[0] for c in cuts]
        x = torch.cat([s[a:a + n] for s, a, n in zip(seqs, ctx, lens)]).to(cuda)
        gate = torch.cat([s[a:a + n] for s, a, n in zip(gates, ctx, lens)]).to(cuda)
        pos = i32([p for a, n in zip(ctx, lens) for p in range(a, a + n)])
        slots = torch.tensor([t[p // 16] * 16 + p % 16 for t, a, n in zip(tables, ctx, lens) for p in range(a, a + n)], device=cuda)
        qa = ops.latent_prep(x, H, dn, dr, dr, Rk, 0, nq, L.nw.to(cuda), L.eps, pos, ops.rotary_table(512, dr, 500.0, None, cuda), slots,
                             L.cache, interleaved=False)
        N, cu_k, k_lo = ops.latent_prompt_plan(lens, [a + n for a, n in zip(ctx, lens)], window, 10 ** 6, cuda)
        bt = torch.zeros(2, 17, dtype=torch.int32)
        for s, t in enumerate(tables):
            bt[s, :len(t)] = torch.tensor(t, dtype=torch.int32)
        lat = ops.latent_gather(L.cache, bt.to(cuda), cu_k, k_lo, 2, N)
        kn = torch.nn.functional.linear(lat[:, :Rk], L.w_uk.to(cuda)).view(N, H, dn)
        v = torch.nn.functional.linear(lat[:, :Rk], L.w_uv.to(cuda)).view(N, H, dv)
        qh = x[:, :nq].view(-1, H, dn + dr)
        wide = torch.full((x.shape[0], H * dv + 16), 33.0, dtype=bf, device=cuda)
        ops.window_attention(qh[:, :, :dn], qa[:, :, Rk:], kn, lat[:, Rk:], v, i32([0, lens[0], sum(lens)]), i32(ctx), cu_k, k_lo, 2,
                             L.scale, window, gate=gate[:, 8:], sink_logits=L.sinks.to(cuda), out=wide[:, 8:8 + H * dv])
        assert bool((wide[:, :8] == 33.0).all()) and bool((wide[:, 8 + H * dv:] == 33.0).all())
        off = 0
        for s in (0, 1):
            lo, n = ctx[s], lens[s]
            want = L.oracle(seqs[s])[lo:lo + n].reshape(n, H * dv) * R.sigmoid(gates[s][lo:lo + n, 8:].to(F64))
            _close(wide[off:off + n, 8:8 + H * dv], want, 3e-2, f"sequence {s}, portion {half}")
            off += n
