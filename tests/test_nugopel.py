"""Nugopel without a GPU: config.json is read into a typed configuration and
back, the model description names the tensors, parts, caches and run list that
the plain implementation's weights ask for, bad configurations are refused, and
the plain implementation itself has the properties the engine is held to (a
position depends on its prefix alone; latent, gate, rotation, scaled
frequencies, window, the one in the denominator and the router behave as their
equations say on inputs made to show it)."""
import json
import math

import numpy as np
import pytest

import plain_nugopel as plain
import tiny_nugopel as tiny
from alofa_b200.config.registry import get_architecture, read_model_config
from alofa_b200.config.spec import PartSpec
from alofa_b200.errors import AlofaError
from alofa_b200.parts.base import PagedKV, PagedRows, Runtime, build_part
from alofa_b200.parts.model import Model, expected_tensors


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("nugopel")
    return {name: tiny.write(base / name, name, seed=i) for i, name in enumerate(tiny.CONFIGS)}


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_config_is_read_and_written_back(folders, name):
    arch, cfg = read_model_config(folders[name])
    assert arch.name == "Nugopel"
    assert arch.to_json(cfg) == json.loads(json.dumps(tiny.CONFIGS[name]))


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_the_description_names_the_tensors_parts_and_caches(folders, name):
    import torch

    raw = tiny.CONFIGS[name]
    arch, cfg = read_model_config(folders[name])
    spec = arch.build_spec(cfg)
    assert {n: tuple(t.shape) for n, t in expected_tensors(spec).items()} == tiny.tensor_shapes(raw)
    assert all(layer.block.kind == "sandwich_residual" and layer.block.params["mixer_norm"].params["weight_offset"] == 1.0 for layer in spec.layers)
    model = Model(spec, Runtime(torch.device("cpu"), torch.float32))
    plan = model.cache_plan()
    for i, layer in enumerate(raw["layers"]):
        m = layer["mixer"]
        if layer["type"] == "attention":
            assert plan[i] == PagedKV(m["kv_heads"], m["dim"], m["mask"]["size"] if "mask" in m else None, m["vdim"])
            assert model.layers[i].mixer.sink_score == 0.0
        elif "kv_from" in m:
            assert i not in plan and model.run[i] == (i, m["kv_from"]) and not model.layers[i].mixer.own_latent
        else:
            assert plan[i] == PagedRows(m["kv_rank"]) and model.run[i] == (i, i)
    assert all(n is not None for n in model.next_norms) and model.next_norms[-1] is model.final_norm
    assert spec.head.params["tied_to"] is None


@pytest.mark.parametrize("broken", [
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"].pop("kv_rank"),
    lambda c: c["layers"][0]["mixer"].update(heads=0),
    lambda c: c["layers"][0]["mixer"].update(kv_from=0),  # itself
    lambda c: c["layers"][2]["mixer"].update(kv_from=1),  # not a latent attention
    lambda c: c["layers"][2]["mixer"].update(kv_from=4),  # a later layer
    lambda c: c["layers"][4]["mixer"].update(kv_from=2),  # no latent of its own
    lambda c: c["layers"][4]["mixer"].update(kv_rank=32),  # another rank
    lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][1]["mixer"].pop("rot"),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=22),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("low"),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5),
    lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][1]["mixer"]["mask"].pop("size"),
    lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0),
    lambda c: c["layers"][0]["mlp"].pop("expert"),
    lambda c: c.update(layers=[]),
    lambda c: c.pop("norm"),
    lambda c: c.pop("width"),
])
def test_bad_configs_are_refused(broken):
    raw = json.loads(json.dumps(tiny.CONFIGS["A"]))
    broken(raw)
    with pytest.raises(AlofaError) as err:
        get_architecture("Nugopel").read_config(raw, "test")
    assert err.value.code == "parse"


def test_random_model_folder(tmp_path):
    """The package's seeded random mode writes a folder of this architecture that the plain reader takes."""
    from alofa_b200.weights.random_init import write_random_model

    arch = get_architecture("Nugopel")
    folder = write_random_model(tmp_path / "m", "Nugopel", arch.read_config(tiny.CONFIGS["A"], "test"), seed=3)
    w, cfg = plain.load(folder)
    assert {n: v.shape for n, v in w.items()} == tiny.tensor_shapes(tiny.CONFIGS["A"])
    assert abs(w["l0.norm1"].mean()) < 0.1 and abs(w["l0.mix.dkv.norm"].mean() - 1.0) < 0.1
    assert np.isfinite(plain.forward(w, cfg, tiny.tokens("A", 9))).all()


def test_parts_refuse_what_they_cannot_do():
    import torch

    rt = Runtime(torch.device("cpu"), torch.float32)
    base = {"hidden_size": 16, "heads": 2, "dim": 8, "vdim": 8, "scale": 1.0, "eps": 1e-5}
    with pytest.raises(AlofaError):
        build_part("mixer", PartSpec("latent_attention", {**base, "kv_rank": 8, "rot_dim": 4}), rt)  # a rotated part without an encoding
    with pytest.raises(AlofaError):
        build_part("mixer", PartSpec("latent_attention", {**base, "kv_rank": 8, "gate": "row"}), rt)
    with pytest.raises(AlofaError):  # halves where heads are normed one by one
        build_part("mixer", PartSpec("normed_attention", {**base, "kv_heads": 2, "position": PartSpec("rotary_interleaved", {"dims": 4, "base": 10.0, "layout": "halves"})}), rt)
    reader = build_part("mixer", PartSpec("latent_attention", {**base, "kv_rank": 8, "own_latent": False}), rt)
    with pytest.raises(AlofaError):
        reader.forward(None, torch.zeros(1, 16), None, None, writes=True)


@pytest.mark.parametrize("rot", [{"base": 100.0, "dims": 16, "scaling": {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 60.0}},
                                 {"base": 5e5, "dims": 128, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192.0}},
                                 {"base": 50.0, "dims": 8, "scaling": {"factor": 2.0, "low": 2.0, "high": 2.0, "original": 40.0}}, {"base": 30.0, "dims": 2}])
def test_scaled_frequencies(rot):
    """The part's frequencies equal plain's; kept, stretched and mixed ones all occur where the scaling has room for them."""
    import torch

    scaling = {"kind": "wavelength", **rot["scaling"]} if "scaling" in rot else None
    part = build_part("position", PartSpec("rotary_interleaved", {"dims": rot["dims"], "base": rot["base"], "layout": "halves", "scaling": scaling}), Runtime(torch.device("cpu"), torch.float32))
    np.testing.assert_allclose(part.make_frequencies(), plain.frequencies(rot), rtol=1e-12)
    assert part.magnitude == 1.0
    f = plain.frequencies({k: rot[k] for k in ("base", "dims")})
    if scaling and scaling["high"] > scaling["low"]:
        r = plain.frequencies(rot) / f
        kept, stretched = r == 1.0, np.abs(r - 1.0 / scaling["factor"]) < 1e-12
        assert kept.any() and stretched.any() and (~kept & ~stretched).any()


# ---- the plain implementation's own properties -------------------------------------------------------------------
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_plain_positions_depend_on_their_prefix_alone(folders, name):
    w, cfg = plain.load(folders[name])
    ids = tiny.tokens(name, 45)
    np.testing.assert_allclose(plain.forward(w, cfg, ids[:27]), plain.forward(w, cfg, ids)[:27], rtol=1e-9, atol=1e-9)


def test_plain_scaled_frequencies_by_hand():
    # wavelengths 2 pi, 20 pi and 200 pi against borders of 25 and 100
    rot = {"base": 1000.0, "dims": 6, "scaling": {"factor": 5.0, "low": 1.0, "high": 4.0, "original": 100.0}}
    s = (100.0 / (20 * math.pi) - 1.0) / 3.0
    np.testing.assert_allclose(plain.frequencies(rot), [1.0, (1 - s) * 0.1 / 5 + s * 0.1, 0.01 / 5])


def test_plain_rotation_pairs_halves_and_depends_on_distance():
    rot = {"base": 10.0, "dims": 4}
    x = np.zeros((4, 1, 6))
    x[:, 0] = [1.0, 0.0, 0.0, 0.0, 7.0, 8.0]
    y = plain.rotate(x, rot)
    np.testing.assert_allclose(y[2, 0], [math.cos(2.0), 0.0, math.sin(2.0), 0.0, 7.0, 8.0])  # number 0 goes with number 2
    rng = np.random.default_rng(0)
    a, b = np.tile(rng.standard_normal((1, 1, 6)), (9, 1, 1)), np.tile(rng.standard_normal((1, 1, 6)), (9, 1, 1))
    dots = plain.rotate(a, rot)[:, 0] @ plain.rotate(b, rot)[:, 0].T
    assert dots[5, 3] == pytest.approx(dots[8, 6]) and dots[5, 3] != pytest.approx(dots[5, 2])


def test_plain_window_and_the_one_in_the_denominator():
    m = plain.causal_mask(9, 3)
    assert m[7].tolist() == [False] * 5 + [True] * 3 + [False] and m[1].tolist() == [True, True] + [False] * 7
    assert (plain.causal_mask(5, 1) == np.eye(5, dtype=bool)).all() and (plain.causal_mask(6) == np.tri(6, dtype=bool)).all()
    p = plain.softmax(np.array([[0.0, math.log(3.0), 50.0]]), np.array([[True, True, False]]), one_more=True)
    np.testing.assert_allclose(p[0], [1 / 5, 3 / 5, 0.0])
    np.testing.assert_allclose(plain.softmax(np.array([[0.0, math.log(3.0)]]), np.ones((1, 2), bool))[0], [1 / 4, 3 / 4])
    low = plain.softmax(np.full((1, 2), -40.0), np.ones((1, 2), bool), one_more=True)
    np.testing.assert_allclose(low[0], np.exp(-40.0), rtol=1e-9)  # nothing overflows, the keys share what is left


def test_plain_norms_span_all_heads_and_offsets_are_added():
    x = np.array([[100.0, 0.0, 1.0, 1.0]])
    n = plain.rms_norm(x, np.ones(4), 0.0)
    assert n[0, 0] == pytest.approx(2.0, rel=1e-3) and n[0, 2] < 0.03
    np.testing.assert_allclose(plain.offset_norm(x, np.array([0.5, 0.0, -1.0, 0.0]), 0.0), n * [1.5, 1.0, 0.0, 1.0])


def test_plain_latent_attention_gates_channels_and_reads_any_latent():
    rng = np.random.default_rng(1)
    m = {"heads": 2, "dim": 3, "vdim": 2, "kv_rank": 4, "scale": 0.7}
    w = {"a.q": rng.standard_normal((6, 5)), "a.uk": rng.standard_normal((6, 4)), "a.uv": rng.standard_normal((4, 4)), "a.g": rng.standard_normal((4, 5)), "a.o": np.eye(4),
         "a.dkv": rng.standard_normal((4, 5)), "a.dkv.norm": np.ones(4)}
    h = rng.standard_normal((1, 5))
    c = plain.latent(w, "a.", h, 1e-6)
    np.testing.assert_allclose((c * c).mean(), 1.0, rtol=1e-4)
    for other in (c, 3.0 * c + 1.0):  # one token sees itself alone: its value, channel by channel
        np.testing.assert_allclose(plain.latent_attention(w, "a.", m, h, other), (other @ w["a.uv"].T) * plain.sigmoid(h @ w["a.g"].T))


def test_plain_experts_and_router():
    w = {"m.up": np.array([[1.0], [-1.0]]), "m.down": np.array([[1.0, 10.0]])}
    assert plain.expert(w, "m.", np.array([[3.0]]))[0, 0] == 9.0 and plain.expert(w, "m.", np.array([[-2.0]]))[0, 0] == 40.0
    w = {"m.router": np.diag([0.3, 2.0, -1.0, 1.0])}
    chosen, weights, margin = plain.route(w, "m.", {"experts": 4, "top": 2}, np.ones((1, 4)))
    assert chosen[0].tolist() == [1, 3] and margin[0] == pytest.approx(0.7)
    np.testing.assert_allclose(weights[0], [1 / (1 + math.exp(-1.0)), 1 / (1 + math.exp(1.0))])  # over the chosen alone
