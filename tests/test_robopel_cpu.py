"""Robopel without a GPU: the plain restatement's mechanisms against hand-worked cases, that a mistake in
any of them shows in the logits of the test models, the configuration reader (round trip, refusals), and
the container / SafeTensors paths of the loader."""
import json
import math

import pytest
import torch

import robopel_plain as P
from robopel_models import MODELS, weights

D64 = dict(dtype=torch.float64)


# ------------------------------------------------------------ plain mechanisms ---
def test_output_norm_has_eps_inside_and_a_gain_around_one():
    x, y, w = torch.tensor([[1.0, 2.0]], **D64), torch.tensor([[3.0, 4.0]], **D64), torch.tensor([0.5, -1.0], **D64)
    assert torch.allclose(P.after_norm(x, y, w, 2.0), torch.tensor([[1.0 + 3 / math.sqrt(14.5) * 1.5, 2.0]], **D64))


def test_min_gru_by_hand():
    one = torch.ones(1, 1, **D64)
    h, zero = torch.tensor([[2.0], [-3.0]], **D64), torch.zeros(1, **D64)
    sg = lambda v: 1 / (1 + math.exp(-v))   # noqa: E731
    got = P.min_gru(h, 0.5 * one, zero + 0.1, one, zero + 0.2, one, one)
    z1, z2 = sg(1.1), sg(-1.4)
    s1 = z1 * 2.7                                   # u = 2.2: the line
    s2 = (1 - z2) * s1 + z2 * sg(-2.8)              # u = -2.8: the curve
    assert got[:, 0].tolist() == pytest.approx([s1 * 2 * sg(2), s2 * -3 * sg(-3)])


def test_frequencies_keep_short_waves_and_slow_long_ones():
    sc = {"factor": 10.0, "low": 1.0, "high": 4.0, "original": 100}
    plain = P.frequencies(8, 1000.0)
    got = P.frequencies(8, 1000.0, sc)
    wave = [2 * math.pi / f for f in plain]
    assert wave[0] < 25 and 25 < wave[1] < 100 and wave[2] > 100
    s = (100 / wave[1] - 1) / 3
    assert got == pytest.approx([plain[0], (1 - s) * plain[1] / 10 + s * plain[1], plain[2] / 10, plain[3] / 10])


def test_rotation_pairs_neighbours_and_leaves_the_rest():
    x = torch.tensor([[[1.0, 0.0, 5.0]], [[1.0, 2.0, 5.0]]], **D64)
    got = P.rotate(x, [0.3], first=4)
    a, b = 1.2, 1.5
    assert got[0, 0].tolist() == pytest.approx([math.cos(a), math.sin(a), 5.0])
    assert got[1, 0].tolist() == pytest.approx([math.cos(b) - 2 * math.sin(b), 2 * math.cos(b) + math.sin(b), 5.0])


def test_window_and_blocks_by_hand():
    """Window 3, blocks of 2: row 6 sees tokens 4..6 and the blocks that end at 3 or before; row 5 has lost
    token 2 and does not see its block yet."""
    t, b = P.visible_tokens(8, 3), P.visible_blocks(8, 3, 2)
    assert t[6].nonzero()[:, 0].tolist() == [4, 5, 6] and t[0].nonzero()[:, 0].tolist() == [0]
    assert [b[i].nonzero()[:, 0].tolist() for i in range(8)] == [[], [], [], [], [0], [0], [0, 1], [0, 1]]


def test_attention_by_hand():
    """One head of size one; row 3 with window 2 and blocks of 2 sees tokens 2, 3 and the mean of 0, 1."""
    q, k, v = (torch.tensor(x, **D64).reshape(4, 1, 1) for x in ([0, 0, 0, 2.0], [1.0, 3.0, -1.0, 0.5], [10.0, 20.0, 30.0, 40.0]))
    cap = lambda s: 1.5 * math.tanh(s / 1.5)   # noqa: E731
    w = [math.exp(cap(2 * 0.7 * x)) for x in (2.0, -1.0, 0.5)]
    got = P.sink_attention(q, k, v, 0.7, 1.5, 2, 2, torch.tensor([0.25], **D64))[3, 0, 0].item()
    assert got == pytest.approx((w[0] * 15 + w[1] * 30 + w[2] * 40) / (sum(w) + math.exp(0.25)))
    assert P.sink_attention(q, k, v, 0.7, None, 2, 0, None)[0, 0, 0].item() == pytest.approx(10.0)


def test_poly_norm_by_hand():
    z = torch.tensor([[1.0, -2.0]], **D64)
    n = [math.sqrt((1 + 2.0 ** (2 * p)) / 2 + 0.1) for p in (1, 2, 3)]
    got = P.poly_norm(z, torch.tensor([2.0, 3.0, 5.0, 7.0], **D64), 0.1)[0].tolist()
    assert got == pytest.approx([2 / n[0] + 3 / n[1] + 5 / n[2] + 7, -4 / n[0] + 12 / n[1] - 40 / n[2] + 7])


def test_mixture_chooses_corrected_and_weighs_uncorrected():
    h, router = torch.tensor([[1.0, -1.0]], **D64), torch.tensor([[1.0, 0.0], [0.5, 0.0], [0.0, 0.0]], **D64)
    s = torch.softmax(torch.tensor([1.0, 0.5, 0.0], **D64), 0)
    up, down = torch.tensor([[3.0, 1.0]], **D64), torch.tensor([[1.0], [2.0]], **D64)
    corr = torch.tensor([-5.0, 0.0, 0.5], **D64)     # the identity first, then expert 1; never expert 0
    got = P.mixture(h, router, corr, 2, [(9 * up, down), (up, down)])
    assert torch.allclose(got[0], s[2] * h[0] + s[1] * torch.tensor([4.0, 8.0], **D64))
    assert P.choice_margin(h, router, corr, 2).item() == pytest.approx((s[1] - (s[0] - 5)).item())


# ------------------------------------------ mistakes show in the test models ---
def _model(name, **patch):
    m = P.Plain(MODELS[name], weights(name))
    c = json.loads(json.dumps(m.c))
    m.c = c
    return m


def _mask(edit):
    def f(m):
        for ly in m.c["layers"]:
            if ly["type"] == "attention":
                edit(ly["mixer"])
    return f


def _weights(suffix, value):
    def f(m):
        for n in m.w:
            if n.endswith(suffix):
                m.w[n] = value(m.w[n])
    return f


MISTAKES = {
    "window one more": _mask(lambda x: x["mask"].update(size=x["mask"]["size"] + 1)),
    "window one less": _mask(lambda x: x["mask"].update(size=x["mask"]["size"] - 1)),
    "blocks left out": _mask(lambda x: x["mask"].update(pool=None)),
    "block size": _mask(lambda x: x["mask"].update(pool=x["mask"]["pool"] + 1)),
    "no cap": _mask(lambda x: x.update(softcap=None)),
    "no rotation": _mask(lambda x: x.pop("rot")),
    "no scaling of waves": _mask(lambda x: x["rot"].pop("scaling", None)),
    "no sink": _weights("mix.sink", lambda w: w - 100),
    "no query norm weight": _weights("q.norm", lambda w: w * 0 + 1),
    "no key norm weight": _weights("k.norm", lambda w: w * 0 + 1),
    "recurrence forgets": _weights("z.b", lambda w: w + 6),
    "candidate's bias": _weights("x.b", lambda w: w * 0),
    "no correction": _weights("correction", lambda w: w * 0),
    "activation's constant": _weights("act", lambda w: w * torch.tensor([1.0, 1, 1, 0], dtype=w.dtype)),
    "activation's cube": _weights("act", lambda w: w * torch.tensor([1.0, 1, 0, 1], dtype=w.dtype)),
    "activation's square": _weights("act", lambda w: w * torch.tensor([1.0, 0, 1, 1], dtype=w.dtype)),
    "norm weight around one": _weights("norm1", lambda w: w - 1),
}


@pytest.mark.parametrize("what", sorted(MISTAKES))
def test_a_mistake_shows(what):
    """In at least one model, well above the tolerance of the bf16 tests."""
    worst = 0.0
    for name in ("shared", "wide"):
        m = _model(name)
        ids = torch.randint(0, m.c["vocab"], (130,), generator=torch.Generator().manual_seed(4)).tolist()
        want = m.forward(ids)
        MISTAKES[what](m)
        worst = max(worst, (((m.forward(ids) - want) ** 2).mean(-1).sqrt().max() / want.std()).item())
    assert worst > 0.2, worst


# -------------------------------------------------------------- configuration ---
@pytest.fixture(scope="module")
def rt():
    from ainfer_b200 import runtime
    runtime.load()
    return runtime


def _write(tmp_path, c):
    p = tmp_path / "config.json"
    p.write_text(json.dumps(c, indent=2))
    return str(p)


@pytest.mark.parametrize("name", sorted(MODELS))
def test_config_round_trip(rt, tmp_path, name):
    assert json.loads(rt.preset_config_json("config:" + _write(tmp_path, MODELS[name]))) == MODELS[name]


def _at(*path, **kw):
    def f(c):
        for k in path:
            c = c[k]
        c.update(kw)
    return f


@pytest.mark.parametrize("edit", [
    _at(architecture="Nothing"), _at(layers=[]), _at(width=0), _at(vocab=0), _at(norm={}),
    _at("layers", 0, type="convolution"), _at("layers", 0, "mixer", kv_heads=3), _at("layers", 0, "mixer", dim=0),
    _at("layers", 0, "mixer", dim=600), _at("layers", 0, "mixer", vdim=0), _at("layers", 0, "mixer", scale=None),
    _at("layers", 0, "mixer", softcap=-1.0), _at("layers", 0, "mixer", "mask", size=-1), _at("layers", 0, "mixer", "rot", dims=5),
    _at("layers", 0, "mixer", "rot", dims=64), _at("layers", 0, "mixer", "rot", "scaling", factor=0), _at("layers", 0, "mixer", "rot", "scaling", high=1.0),
    _at("layers", 2, "mixer", kv_from=2), _at("layers", 2, "mixer", kv_from=1), _at("layers", 2, "mixer", kv_from=-1), _at("layers", 4, "mixer", kv_from=2),
    _at("layers", 2, "mixer", dim=24), _at("layers", 1, "mixer", width=0), _at("layers", 1, "mlp", kind="gated"), _at("layers", 1, "mlp", ff=0),
    _at("layers", 0, "mlp", "router", top=7), _at("layers", 0, "mlp", "router", experts=0), _at("layers", 0, "mlp", "router", experts=2000),
    _at("layers", 0, "mlp", "expert", ff=0),
])
def test_config_refusals(rt, tmp_path, edit):
    c = json.loads(json.dumps(MODELS["shared"]))
    edit(c)
    assert rt.preset_config_json("config:" + _write(tmp_path, c)) is None


def test_synthetic_file_and_conversion(rt, tmp_path):
    c = MODELS["shared"]
    out = str(tmp_path / "m.binfer")
    rt.synth_write(out, "config:" + _write(tmp_path, c), seed=3)
    assert rt.validate(out, 2) == (0, "")
    w = weights("shared")
    P.write_model(str(tmp_path / "model"), c, w)
    rt.from_safetensors(str(tmp_path / "model"), json.dumps(c), str(tmp_path / "n.binfer"))
    assert rt.validate(str(tmp_path / "n.binfer"), 2) == (0, "")
    raw = open(tmp_path / "n.binfer", "rb").read()
    for n in ("l0.mix.q", "l1.mix.z.b", "l3.mlp.e5.down", "head"):
        assert w[n].contiguous().view(torch.int16).numpy().tobytes() in raw
    for drop, keep, why in (("l0.mix.o", w["l0.mix.o"][:-1], "shape of l0.mix.o"), ("l3.mlp.e5.up", None, "missing l3.mlp.e5.up")):
        bad = {k: v for k, v in w.items() if k != drop}
        if keep is not None:
            bad[drop] = keep
        P.write_model(str(tmp_path / "bad"), c, bad)
        with pytest.raises(rt.RuntimeError_, match=why):
            rt.from_safetensors(str(tmp_path / "bad"), json.dumps(c), str(tmp_path / "x.binfer"))


@pytest.mark.parametrize("name", ["robopel-tiny", "robopel-small"])
def test_named_shapes(rt, name):
    c = json.loads(rt.preset_config_json(name))
    assert c["architecture"] == "Robopel" and {ly["type"] for ly in c["layers"]} == {"attention", "mingru"}
    assert any("kv_from" in ly["mixer"] for ly in c["layers"])
