"""Host-side pieces of the Gapidra family (no GPU): the configuration reader with its defaults and refusals, pool sizes and
tensor names, the rotary table, and the plain oracle against cases worked out by hand."""
import json
import math

import pytest
import torch

import gapidra_ref as R
import gapidra_util as U

F64 = torch.float64


def _config(c):
    from b200attn import gapidra
    return gapidra.config_from_dict(c)


def test_registered_and_read_from_a_directory(tmp_path):
    from b200attn.model import ARCHITECTURES, resolve_config
    assert "Gapidra" in ARCHITECTURES
    (tmp_path / "config.json").write_text(json.dumps(U.cfg_a()))
    c = resolve_config(str(tmp_path))
    assert c.family == "gapidra" and (c.vocab, c.hidden, c.layers, c.eps, c.embed_scale) == (97, 64, 4, 1e-5, 2.5)
    s = c.layer_specs[0].mixer
    assert (s.heads, s.kv_heads, s.dim, s.vdim, s.scale, s.window) == (4, 1, 24, 16, 0.3, 9)
    assert (s.rot.dims, s.rot.base, dict(s.rot.scaling)) == (12, 500.0, {"factor": 4.0, "original": 300.0, "fast": 8.0, "slow": 1.0})
    m = c.layer_specs[1].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.window, m.row, m.out) == (3, 16, 8, 20, 24, 0.2, 17, 32, 60)
    assert (m.rot.dims, m.rot.base, m.rot.scaling) == (8, 300.0, None)
    assert [L.mlp and L.mlp.ff for L in c.layer_specs] == [40, 56, None, 24]


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_tensor_names_and_pool_sizes(name):
    cfg = U.CONFIGS[name]()
    c = _config(cfg)
    assert c.tensors() == R.tensor_shapes(cfg)
    assert c.params == sum(math.prod(s) for s in R.tensor_shapes(cfg).values())
    per_token = 0
    for L in cfg["layers"]:
        m = L["mixer"]
        per_token += m["kv_rank"] + m["rot_dim"] if L["type"] == "latent_attention" else m["kv_heads"] * (m["dim"] + m["vdim"])
    assert c.kv_bytes_per_token(2) == 2 * per_token and c.kv_bytes_per_token(4) == 4 * per_token
    assert c.state_bytes_per_seq() == 0 and c.activation_bytes(128, 4) > 0


def test_defaults():
    c = U.cfg_a()
    del c["embedding"], c["norm"]
    for k in ("mask", "rot", "kv_heads", "vdim"):
        c["layers"][3]["mixer"].pop(k)
    del c["layers"][1]["mixer"]["rot"]["dims"]
    s = _config(c)
    assert (s.embed_scale, s.eps) == (1.0, 1e-6)
    m = s.layer_specs[3].mixer
    assert (m.window, m.rot.dims, m.kv_heads, m.vdim) == (0, 0, 3, 16)
    assert s.layer_specs[1].mixer.rot.dims == 8


@pytest.mark.parametrize("edit,match", [
    (lambda c: c["layers"][0].update(type="convolution"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=13), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "scaling"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=-1), "mask"),
])
def test_refusals(edit, match):
    c = U.cfg_a()
    edit(c)
    with pytest.raises(ValueError, match=match):
        _config(c)


@pytest.mark.parametrize("dims,base,scaling", [(12, 500.0, U.yarn(4.0, 300, 8.0, 1.0)), (8, 2e3, U.yarn(2.5, 128, 6.0, 1.5)),
                                               (16, 1e6, U.yarn(32.0, 4096, 32.0, 1.0)), (2, 9.0, U.yarn(3.0, 50, 2.0, 0.5)), (20, 77.0, None)])
def test_rotary_table_against_the_oracle(dims, base, scaling):
    from b200attn import ops
    t = ops.rotary_table(5000, dims, base, scaling, "cpu").double()
    f, mag = R.rotary_frequencies(dims, base, scaling), R.rotary_magnitude(scaling)
    for p in (0, 1, 77, 4999):
        want = [mag * math.cos(p * x) for x in f] + [mag * math.sin(p * x) for x in f]
        assert torch.allclose(t[p], torch.tensor(want, dtype=F64), atol=1e-6)


# ------------------------------------------------------------------------------------------------ the oracle by hand
def test_yarn_by_hand():
    s = U.yarn(4.0, 256, 8.0, 1.0)
    # pairs: turns over 256 positions of pair i: 256 f_i / 2 pi, f_i = 100^(-i / 4)
    border = lambda t: 8 * math.log(256 / (2 * math.pi * t)) / (2 * math.log(100.0))      # noqa: E731
    lo, hi = math.floor(border(8.0)), math.ceil(border(1.0))
    assert (lo, hi) == (1, 4)
    assert R.yarn_ramp(8, 100.0, s) == [0.0, 0.0, 1 / 3, 2 / 3]
    f = R.rotary_frequencies(8, 100.0, s)
    raw = [100.0 ** (-i / 4) for i in range(4)]
    assert f[:2] == raw[:2]
    assert abs(f[3] - (raw[3] / 4 * 2 / 3 + raw[3] / 3)) < 1e-15
    assert R.rotary_magnitude(s) == 0.1 * math.log(4.0) + 1.0 and R.rotary_magnitude(None) == 1.0
    # borders outside the pairs: everything kept / everything slowed (the ramp's span is never zero)
    assert R.yarn_ramp(4, 10.0, U.yarn(2.0, 10 ** 9, 2.0, 1.0)) == [0.0, 0.0]
    assert R.yarn_ramp(4, 10.0, U.yarn(2.0, 2, 2.0, 1.0))[1] == 1.0


def test_rotation_layouts_by_hand():
    x = torch.zeros(4, 6, dtype=F64)
    x[3] = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0, 6.0], dtype=F64)
    rot = {"dims": 4, "base": 100.0}
    a, b = 3 * 1.0, 3 * 0.1
    want = [1 * math.cos(a) - 3 * math.sin(a), 2 * math.cos(b) - 4 * math.sin(b), 3 * math.cos(a) + 1 * math.sin(a),
            4 * math.cos(b) + 2 * math.sin(b), 5.0, 6.0]
    assert torch.allclose(R.rotate(x, rot, "half")[3], torch.tensor(want, dtype=F64))
    want = [1 * math.cos(a) - 2 * math.sin(a), 2 * math.cos(a) + 1 * math.sin(a), 3 * math.cos(b) - 4 * math.sin(b),
            4 * math.cos(b) + 3 * math.sin(b), 5.0, 6.0]
    assert torch.allclose(R.rotate(x, rot, "interleaved")[3], torch.tensor(want, dtype=F64))
    assert torch.equal(R.rotate(x, None, "half"), x)


def test_mask_by_hand():
    see = lambda i, W: [j for j in range(i + 3) if R.visible(i, j, W)]      # noqa: E731
    assert see(5, 0) == [0, 1, 2, 3, 4, 5] and see(5, 3) == [3, 4, 5] and see(5, 1) == [5] and see(1, 3) == [0, 1]


def test_weights_by_hand():
    s = torch.tensor([[0.0, math.log(3.0)]], dtype=F64)
    both, one = torch.tensor([[True, True]]), torch.tensor([[True, False]])
    assert torch.allclose(R.sink_softmax(s, both, None), torch.tensor([[0.25, 0.75]], dtype=F64))
    assert torch.allclose(R.sink_softmax(s, both, math.log(4.0)), torch.tensor([[0.125, 0.375]], dtype=F64))     # the sink takes half
    assert torch.allclose(R.sink_softmax(s, one, 0.0), torch.tensor([[0.5, 0.0]], dtype=F64))
    # sigmoid weights: a key's weight is its own, whatever else is seen
    assert torch.allclose(R.sigmoid_weights(s, both, 0.0), torch.tensor([[0.5, 0.75]], dtype=F64))
    assert torch.allclose(R.sigmoid_weights(s, one, 0.0), torch.tensor([[0.5, 0.0]], dtype=F64))
    assert torch.allclose(R.sigmoid_weights(s, both, -math.log(3.0)), torch.tensor([[0.25, 0.5]], dtype=F64))


def test_xielu_by_hand():
    z = torch.tensor([2.0, 0.0, -1.0, -50.0], dtype=F64)
    a, b = math.log(2.0), 0.5 + math.log(1 + math.e)
    want = [4 * a + 1.0, 0.0, b * math.exp(-1.0) - 0.5, b * 49.0 - 25.0]
    assert torch.allclose(R.xielu(z, 0.0, 1.0), torch.tensor(want, dtype=F64))
    assert abs(R.softplus(-40.0) - math.exp(-40.0)) < 1e-25 and R.softplus(700.0) == 700.0


@pytest.mark.parametrize("name", ["a", "d"])
def test_both_sublayers_read_one_norm_and_the_prefix_property(name):
    """Taking a layer's output product or its down product away removes exactly that sublayer's part of the residual step; the
    logits of a position depend on the tokens before it only."""
    cfg = U.CONFIGS[name]()
    W = R.random_model(cfg, 3)
    toks = U.tokens(23, cfg["vocab"], 5)
    one = dict(cfg, layers=cfg["layers"][:1])
    trails = []
    for gone in ((), ("l0.mix.o",), ("l0.mlp.down",), ("l0.mix.o", "l0.mlp.down")):
        w = {k: (torch.zeros_like(v) if k in gone else v) for k, v in W.items()}
        trail = []
        R.forward(one, w, toks, trail)
        trails.append(trail[0])
    both, no_mix, no_ff, none = trails
    assert torch.allclose(both - none, (no_ff - none) + (no_mix - none), atol=1e-12) and float((no_ff - no_mix).abs().max()) > 0.1
    full = R.forward(cfg, W, toks)
    assert torch.allclose(R.forward(cfg, W, toks[:11]), full[:11], atol=1e-9)
