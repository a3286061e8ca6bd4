"""Sinepel without a GPU: the plain restatement's mechanisms against hand-worked cases, the
configuration reader (round trip, refusals), and the container / SafeTensors paths of the loader."""
import json
import math

import pytest
import torch

import sinepel_plain as P


# ------------------------------------------------------------ plain mechanisms ---
def test_norm_puts_eps_inside_the_root():
    x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
    assert torch.allclose(P.rms(x, 2.0), x / math.sqrt(12.5 + 2.0))


def test_streams_mix_is_indexed_from_to():
    x = torch.tensor([[[1.0], [10.0]]])
    mix, out, y = torch.tensor([[2.0, 3.0], [5.0, 7.0]]), torch.tensor([0.5, -1.0]), torch.tensor([[4.0]])
    got = P.streams_write(x, mix, out, y)[0, :, 0]
    assert got.tolist() == [2 + 50 + 2.0, 3 + 70 - 4.0]


def test_shift_uses_the_unshifted_predecessor():
    h = torch.tensor([[1.0], [3.0], [7.0]])
    assert P.token_shift(h, torch.tensor([0.25]))[:, 0].tolist() == [0.75, 2.5, 6.0]


def test_conv_last_tap_meets_the_current_token():
    y = P.short_conv(torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[100.0, 10.0, 1.0]]))
    assert y[:, 0].tolist() == [1.0, 12.0, 124.0]
    assert P.short_conv(torch.tensor([[5.0], [6.0]]), torch.tensor([[3.0]]))[:, 0].tolist() == [15.0, 18.0]


def test_chunks_count_from_position_zero():
    m = P.visible(7, 3)
    assert [m[i].nonzero()[:, 0].tolist() for i in range(7)] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]


def test_attention_values_are_keys_and_distance_lowers_scores():
    q, k = torch.ones(2, 1, 1), torch.tensor([[[2.0]], [[3.0]]])
    temp, r1, r2 = torch.tensor([1.5]), torch.tensor([0.7]), torch.tensor([2.0])
    s0, s1 = 2 * 0.5 * 1.5 - 0.7 * math.log(3.0), 3 * 0.5 * 1.5
    w = math.exp(s0) / (math.exp(s0) + math.exp(s1))
    got = P.shared_kv_attention(q, k, 0.5, temp, r1, r2, 8)
    assert got[0, 0, 0].item() == pytest.approx(2.0) and got[1, 0, 0].item() == pytest.approx(2 * w + 3 * (1 - w), rel=1e-6)


def test_a_layer_reads_only_its_chunk_through_attention():
    """Two sequences that differ in one token differ later only through the shift and the taps once the
    chunk is over: with neither, positions of the next chunk agree."""
    ly = P.make_layer(conv=1, chunk=4)
    c = P.make_config(layers=[ly])
    w = P.make_weights(c, 3)
    w["l0.shift"].zero_()
    m = P.Plain(c, w)
    a, b = [5, 6, 7, 8, 9, 10], [5, 60, 7, 8, 9, 10]
    la, lb = m.forward(a), m.forward(b)
    assert not torch.allclose(la[3], lb[3]) and torch.equal(la[4:], lb[4:])


# -------------------------------------------------------------- configuration ---
@pytest.fixture(scope="module")
def rt():
    from ainfer_b200 import runtime
    runtime.load()
    return runtime


def _cfg(tmp_path, edit=None):
    c = P.make_config(layers=[P.make_layer(), P.make_layer(heads=6, kv_heads=3, dim=20, conv=1, chunk=7, ff=None)])
    if edit:
        edit(c)
    p = tmp_path / "config.json"
    p.write_text(json.dumps(c, indent=2))
    return c, str(p)


def test_config_round_trip(rt, tmp_path):
    c, path = _cfg(tmp_path)
    assert json.loads(rt.preset_config_json("config:" + path)) == c


@pytest.mark.parametrize("edit", [
    lambda c: c.update(architecture="Nothing"),
    lambda c: c["layers"][0].update(type="recurrence"),
    lambda c: c["layers"][0]["mixer"].update(vdim=8),
    lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"].update(dim=0),
    lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mlp"].update(kind="experts"),
    lambda c: c.update(streams=99),
    lambda c: c.update(layers=[]),
    lambda c: c.pop("width"),
    lambda c: c.pop("max_positions"),
    lambda c: c.pop("norm"),
])
def test_config_refusals(rt, tmp_path, edit):
    _, path = _cfg(tmp_path, edit)
    assert rt.preset_config_json("config:" + path) is None


def test_synthetic_file_and_conversion(rt, tmp_path):
    """A synthetic container of the shape validates; a SafeTensors folder of the same shape converts to
    one whose payload is the source's bytes; a tensor of another shape or a missing one is refused."""
    c, path = _cfg(tmp_path)
    out = str(tmp_path / "m.binfer")
    rt.synth_write(out, "config:" + path, seed=3)
    assert rt.validate(out, 2) == (0, "")
    w = P.make_weights(c, 1)
    P.write_model(str(tmp_path / "model"), c, w)
    rt.from_safetensors(str(tmp_path / "model"), json.dumps(c), str(tmp_path / "n.binfer"))
    assert rt.validate(str(tmp_path / "n.binfer"), 2) == (0, "")
    raw = open(tmp_path / "n.binfer", "rb").read()
    for n in ("l0.mix.q", "l1.mix.k.conv", "head"):
        assert w[n].contiguous().view(torch.int16).numpy().tobytes() in raw
    bad = dict(w)
    bad["l0.mix.o"] = bad["l0.mix.o"][:-1]
    P.write_model(str(tmp_path / "bad"), c, bad)
    with pytest.raises(rt.RuntimeError_, match="shape of l0.mix.o"):
        rt.from_safetensors(str(tmp_path / "bad"), json.dumps(c), str(tmp_path / "x.binfer"))
    bad = {k: v for k, v in w.items() if k != "l1.shift"}
    P.write_model(str(tmp_path / "bad2"), c, bad)
    with pytest.raises(rt.RuntimeError_, match="missing l1.shift"):
        rt.from_safetensors(str(tmp_path / "bad2"), json.dumps(c), str(tmp_path / "x.binfer"))


@pytest.mark.parametrize("name", ["sinepel-tiny", "sinepel-small"])
def test_named_shapes(rt, name):
    c = json.loads(rt.preset_config_json(name))
    assert c["architecture"] == "Sinepel" and len(c["layers"]) >= 3
    assert all(ly["mixer"]["heads"] % ly["mixer"]["kv_heads"] == 0 for ly in c["layers"])


def test_plain_reader_and_writer_agree(tmp_path):
    c = P.make_config(layers=[P.make_layer()])
    w = P.make_weights(c, 2)
    P.write_model(str(tmp_path), c, w)
    c2, w2 = P.read_model(str(tmp_path))
    assert c2 == c and all(torch.equal(w[k], w2[k]) for k in w)
