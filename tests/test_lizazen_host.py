"""Host-side pieces of the Lizazen family (no GPU): the configuration reader with its defaults and refusals, pool and state
sizes and tensor names, the rotary table, and the plain oracle against cases worked out by hand."""
import json
import math

import pytest
import torch

import lizazen_ref as R
import lizazen_util as U

F64 = torch.float64


def _config(c):
    from b200attn import lizazen
    return lizazen.config_from_dict(c)


def test_registered_and_read_from_a_directory(tmp_path):
    from b200attn.model import ARCHITECTURES, resolve_config
    assert "Lizazen" in ARCHITECTURES
    (tmp_path / "config.json").write_text(json.dumps(U.cfg_a()))
    c = resolve_config(str(tmp_path))
    assert c.family == "lizazen" and (c.vocab, c.hidden, c.layers, c.eps, c.buckets, c.mul_prev, c.mul_cur) == (97, 64, 4, 1e-5, 31, 17, 5)
    p = c.layer_specs[0].mixer
    assert (p.left.heads, p.left.kv_heads, p.left.dim, p.left.vdim, p.left.scale, p.left.chunk, p.left.rot.dims) == (4, 2, 24, 16, 0.25, 24, 12)
    assert (p.right.heads, p.right.dim, p.right.vdim, p.right.decay, p.right.rot.base) == (3, 16, 24, (0.5, 0.95, 1.0), 90.0)
    a = c.layer_specs[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.scale, a.softcap, a.window) == (4, 1, 24, 0.3, 5.0, 9)
    assert (a.rot.dims, a.rot.base, dict(a.rot.scaling)) == (12, 500.0, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 300.0})
    d = c.layer_specs[3].mixer
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.scale, d.diff, d.window, d.keep_first) == (2, 2, 8, 4, 0.5, 0.6, 5, 40)
    e, f = c.layer_specs[0].mlp, c.layer_specs[1].mlp
    assert (e.experts, e.top, e.ff, e.shared_ff) == (5, 2, 24, 40) and (f.ff, f.limit) == (40, 0.7)
    assert c.layer_specs[2].mlp is None and c.layer_specs[3].mlp.shared_ff == 0


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_tensor_names_pool_and_state_sizes(name):
    cfg = U.CONFIGS[name]()
    c = _config(cfg)
    assert c.tensors() == R.tensor_shapes(cfg)
    assert c.params == sum(math.prod(s) for s in R.tensor_shapes(cfg).values())
    per_token, state = 0, 8
    for L in cfg["layers"]:
        m = L["mixer"]
        if L["type"] == "parallel":
            r = m["right"]
            state += 4 * r["heads"] * r["dim"] * r["vdim"]
            m = m["left"]
        per_token += m["kv_heads"] * (m["dim"] * (2 if L["type"] == "attention_2" else 1) + m["vdim"])
    assert c.kv_bytes_per_token(2) == 2 * per_token and c.kv_bytes_per_token(4) == 4 * per_token
    assert c.state_bytes_per_seq() == state and c.activation_bytes(128, 4) > 0


def test_defaults():
    c = U.cfg_a()
    del c["norm"], c["embedding"]
    for k in ("mask", "rot", "softcap", "kv_heads", "vdim"):
        c["layers"][1]["mixer"].pop(k)
    for k in ("mask", "vdim", "kv_heads"):
        c["layers"][3]["mixer"].pop(k)
    del c["layers"][2]["mixer"]["rot"]["dims"]
    s = _config(c)
    assert (s.eps, s.buckets) == (1e-6, 0) and "bigram" not in s.tensors()
    m = s.layer_specs[1].mixer
    assert (m.window, m.rot.dims, m.softcap, m.kv_heads) == (0, 0, 0.0, 4)
    m = s.layer_specs[3].mixer
    assert (m.window, m.keep_first, m.vdim, m.kv_heads) == (0, 0, 8, 2)
    assert s.layer_specs[2].mixer.rot.dims == 16


@pytest.mark.parametrize("edit,match", [
    (lambda c: c["layers"][0].update(type="convolution"), "unknown mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=16), "values are the keys"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-2.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=13), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("high"), "scaling"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(low=4.0), "below high"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=-1), "mask.size"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay factors"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "left"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "router picks"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "bucket"),
])
def test_refusals(edit, match):
    c = U.cfg_a()
    edit(c)
    with pytest.raises(ValueError, match=match):
        _config(c)


@pytest.mark.parametrize("dims,base,scaling", [(12, 500.0, U.zones(4.0, 1.0, 4.0, 300)), (20, 1e3, U.zones(16.0, 0.5, 2.0, 64)),
                                               (64, 5e5, U.zones(8.0, 1.0, 4.0, 8192)), (2, 9.0, U.zones(3.0, 1.0, 8.0, 50)), (20, 77.0, None)])
def test_rotary_table_against_the_oracle(dims, base, scaling):
    from b200attn import ops
    t = ops.rotary_table(5000, dims, base, scaling, "cpu").double()
    f = R.rotary_frequencies(dims, base, scaling)
    for p in (0, 1, 77, 4999):
        want = [math.cos(p * x) for x in f] + [math.sin(p * x) for x in f]
        assert torch.allclose(t[p], torch.tensor(want, dtype=F64), atol=1e-6)


# ------------------------------------------------------------------------------------------------ the oracle by hand
def test_three_zones_by_hand():
    s = U.zones(8.0, 1.0, 4.0, 2048)
    at = lambda length: R.scaled_frequency(2 * math.pi / length, s) / (2 * math.pi / length)       # noqa: E731
    assert at(100.0) == 1.0 and at(511.9) == 1.0
    assert abs(at(2048.1) - 1 / 8) < 1e-12 and abs(at(1e6) - 1 / 8) < 1e-12
    assert abs(at(2048 / 2.5) - (0.5 / 8 + 0.5)) < 1e-12             # halfway between one and four turns
    assert abs(at(512.000001) - 1.0) < 1e-6 and abs(at(2047.999999) - 1 / 8) < 1e-6


def test_bigram_rows_by_hand():
    b = {"buckets": 7, "mul_prev": 10, "mul_cur": 3}
    assert [R.bigram_row(p, c, b) for p, c in ((None, 5), (0, 5), (5, 0), (2, 4))] == [7, 15 % 7, 50 % 7, 32 % 7]
    w = {"embed": torch.arange(6, dtype=F64).view(6, 1) * 100, "bigram": torch.arange(8, dtype=F64).view(8, 1)}
    assert R.embedding([5, 0, 0], w, b).flatten().tolist() == [507.0, 0.0 + 50 % 7, 0.0]


def test_masks_by_hand():
    assert [j for j in range(12) if R.in_window(7, j, 3)] == [5, 6, 7]
    assert [j for j in range(12) if R.in_window_or_kept(7, j, 2, 3)] == [0, 1, 2, 6, 7]
    assert [j for j in range(12) if R.in_window_or_kept(1, j, 1, 9)] == [0, 1]
    assert [j for j in range(12) if R.in_chunk(7, j, 4)] == [4, 5, 6, 7] and [j for j in range(12) if R.in_chunk(8, j, 4)] == [8]


def test_scores_caps_and_sinks_by_hand():
    assert abs(float(R.softcap(torch.tensor(1000.0, dtype=F64), 5.0)) - 5.0) < 1e-12
    assert abs(float(R.softcap(torch.tensor(0.01, dtype=F64), 5.0)) - 0.01) < 1e-7
    one = torch.ones(1, 1, dtype=torch.bool)
    z = torch.zeros(1, 1, dtype=F64)
    assert float(R.softmax_rows(z, one)) == 1.0 and abs(float(R.softmax_rows(z, one, math.log(3.0))) - 0.25) < 1e-12
    assert abs(float(R.softmax_rows(z, one, 400.0))) < 1e-100 and float(R.softmax_rows(z + 800.0, one, 0.0)) == 1.0


def test_differential_attention_by_hand():
    """One visible key per map gives a1 = a2 = v: the difference is (1 - lambda) v, its norm leaves a unit row times its sign."""
    v = torch.tensor([[[3.0, -4.0]]], dtype=F64)
    q = k = torch.ones(1, 1, 2, 2, dtype=F64)
    seen = torch.ones(1, 1, dtype=torch.bool)
    unit = v / math.sqrt(12.5)
    assert torch.allclose(R.differential_attention(q, k, v, seen, 1.0, 0.5, 0.2, 0.0), 0.8 * unit)
    assert torch.allclose(R.differential_attention(q, k, v, seen, 1.0, 3.0, 0.2, 0.0), -0.8 * unit)
    assert float(R.differential_attention(q, k, v, seen, 1.0, 1.0, 0.2, 1e-5).abs().max()) == 0.0
    n = torch.zeros(2, dtype=F64)
    assert abs(R.diff_lambda(n, n, n, n, 0.3) - 0.3) < 1e-12
    assert abs(R.diff_lambda(n + 1, n + 0.5, n, n, 0.3) - (math.e - 1 + 0.3)) < 1e-12


def test_retention_by_hand():
    q, k = torch.ones(3, 1, 1, dtype=F64), torch.tensor([1.0, 2.0, 3.0], dtype=F64).view(3, 1, 1)
    v = torch.tensor([5.0, 7.0, 11.0], dtype=F64).view(3, 1, 1)
    o, S = R.retention(q, k, v, [0.5])
    assert o.flatten().tolist() == [5.0, 16.5, 41.25] and float(S) == 41.25
    head, S1 = R.retention(q[:2], k[:2], v[:2], [0.5])
    tail, S2 = R.retention(q[2:], k[2:], v[2:], [0.5], S1)
    assert torch.equal(torch.cat([head, tail]), o) and torch.equal(S2, S)


def test_feed_forwards_by_hand():
    g, u = torch.tensor([9.0, -9.0, 0.5], dtype=F64), torch.tensor([9.0, -9.0, 0.25], dtype=F64)
    y = R.bounded_glu(g, u, 1.0)
    sg = lambda z: 1 / (1 + math.exp(-z))       # noqa: E731
    want = [sg(1.702) * 2.0, 0.0, 0.5 * sg(0.851) * 1.25]
    assert torch.allclose(y, torch.tensor(want, dtype=F64), atol=1e-12)
    ids, wts = R.route(torch.eye(2, dtype=F64), torch.tensor([[0.0, 3.0], [2.0, 1.0], [1.0, -9.0]], dtype=F64), 2)
    assert ids.tolist() == [[1, 2], [0, 1]] and torch.allclose(wts, torch.tensor([[sg(2), sg(1)], [sg(3), sg(1)]], dtype=F64))
    w = {f"m.{n}.{t}": torch.eye(2, dtype=F64) for n in ("e0", "e1", "shared") for t in ("gate", "up", "down")}
    w["m.router"] = torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F64)
    h = torch.tensor([[2.0, 1.0]], dtype=F64)
    f = {"router": {"experts": 2, "top": 1}, "expert": {"ff": 2}, "shared": {"ff": 2}}
    s = sg(2.0)
    act = lambda z: z * z * sg(z)       # noqa: E731
    assert torch.allclose(R.experts_ff(h, w, "m", f), torch.tensor([[act(2 * s) + act(2.0), act(s) + act(1.0)]], dtype=F64))


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_prefix_property(name):
    """The logits at a position do not change with what follows it."""
    cfg = U.CONFIGS[name]()
    W = R.random_model(cfg, 5)
    toks = U.tokens(26, cfg["vocab"], 1)
    whole = R.forward(cfg, W, toks)
    for n in (1, 7, 19):
        assert torch.allclose(R.forward(cfg, W, toks[:n]), whole[:n], atol=1e-9)
