"""Pekerax without a GPU: config.json is read into a typed configuration and
back, the model description names the tensors, parts and caches that the plain
implementation's weights ask for, bad configurations are refused, the cache
manager and the scheduler keep a request's first pages beside a window, and the
plain implementation itself has the properties the engine is held to (a
position depends on its prefix alone; window, kept tokens, bias, sink, mixed
values, the delta rule, the clamped gate and the router behave as their
equations say on inputs made to show it)."""
import json
import math

import numpy as np
import pytest

import plain_pekerax as plain
import tiny_pekerax as tiny
from alofa_b200.cache import CacheManager, GroupSpec
from alofa_b200.config.registry import get_architecture, read_model_config
from alofa_b200.engine.scheduler import SchedConfig, SchedInput, Scheduler, format_config, parse_config
from alofa_b200.errors import AlofaError
from alofa_b200.parts.base import PagedKV, Runtime, SlotState
from alofa_b200.parts.model import Model, expected_tensors


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("pekerax")
    return {name: tiny.write(base / name, name, seed=i) for i, name in enumerate(tiny.CONFIGS)}


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_config_is_read_and_written_back(folders, name):
    arch, cfg = read_model_config(folders[name])
    assert arch.name == "Pekerax"
    assert arch.to_json(cfg) == json.loads(json.dumps(tiny.CONFIGS[name]))


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_the_description_names_the_tensors_parts_and_caches(folders, name):
    import torch

    raw = tiny.CONFIGS[name]
    arch, cfg = read_model_config(folders[name])
    spec = arch.build_spec(cfg)
    assert {n: tuple(t.shape) for n, t in expected_tensors(spec).items()} == tiny.tensor_shapes(raw)
    assert all(layer.block.kind == "prenorm_residual" and layer.block.params["mixer_norm"].kind == "layernorm" for layer in spec.layers)
    model = Model(spec, Runtime(torch.device("cpu"), torch.float32))
    plan, seen = model.cache_plan(), False
    for i, layer in enumerate(raw["layers"]):
        m = layer["mixer"]
        if layer["type"] == "attention":
            mask = m.get("mask") or {}
            assert plan[i] == PagedKV(m["kv_heads"], m["dim"], mask.get("size"), m["vdim"], None, mask.get("keep_first", 0))
            assert model.layers[i].mixer.value_mix == ((("later" if seen else "first") if m["v_mix"] else None))
            seen = seen or m["v_mix"]
        else:
            assert plan[i] == SlotState((m["heads"] * m["dim"] * m["vdim"] + (m["conv"] - 1) * (2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"]),))
    mixing = [l["mixer"] for l in raw["layers"] if l["mixer"].get("v_mix")]
    assert model.shared_value_width == mixing[0]["kv_heads"] * mixing[0]["vdim"]
    assert spec.head.params["tied_to"] == "embed" and spec.embedding.params["scale"] == raw["embedding"]["scale"]


@pytest.mark.parametrize("broken", [
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"]["mask"].pop("size"),
    lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1),
    lambda c: c["layers"][0]["mixer"].update(v_mix=1),
    lambda c: c["layers"][0]["mixer"].update(vdim=20),  # another number of values than the later layers that mix theirs
    lambda c: c["layers"][0]["mlp"].update(kind="routed"),
    lambda c: c["layers"][0]["mlp"].update(limit=0.0),
    lambda c: c["layers"][1]["mixer"].update(conv=0),
    lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=0),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=3),  # one group of two experts holds two
    lambda c: c.update(layers=[]),
    lambda c: c.update(embedding=3.0),
    lambda c: c.pop("norm"),
    lambda c: c.pop("width"),
])
def test_bad_configs_are_refused(broken):
    raw = json.loads(json.dumps(tiny.CONFIGS["A"]))
    broken(raw)
    with pytest.raises(AlofaError) as err:
        get_architecture("Pekerax").read_config(raw, "test")
    assert err.value.code == "parse"


def test_random_model_folder(tmp_path):
    """The package's seeded random mode writes a folder of this architecture that the plain reader takes."""
    from alofa_b200.weights.random_init import write_random_model

    arch = get_architecture("Pekerax")
    folder = write_random_model(tmp_path / "m", "Pekerax", arch.read_config(tiny.CONFIGS["A"], "test"), seed=3)
    w, cfg = plain.load(folder)
    assert {n: v.shape for n, v in w.items()} == tiny.tensor_shapes(tiny.CONFIGS["A"])
    assert np.isfinite(plain.forward(w, cfg, tiny.tokens("A", 9))).all()


# ---- pages kept beside a window ---------------------------------------------------------------------------------
@pytest.mark.parametrize("window,keep", [(24, 1), (24, 16), (24, 17), (8, 40), (1, 3), (50, 100)])
def test_kept_pages_stay_while_the_window_gives_pages_back(window, keep):
    cm = CacheManager([GroupSpec(16, 64, window, keep), GroupSpec(16, 64, window)], max_requests=2, max_tokens=1024)
    s, length = cm.admit(1), 0
    kept = -(-keep // 16)
    rng = np.random.default_rng(0)
    while length < 700:
        n = int(rng.integers(1, 40))
        cm.reserve(s, length + n)
        table = cm.block_table(s, 0)
        for p in range(length, length + n):  # every key a query of this portion sees has a page
            assert all(table[j // 16] >= 0 for j in range(p + 1) if p - j < window or j < keep)
        length += n
        cm.advance(s, length)
        table, passed = cm.block_table(s, 0), max(0, length - window + 1) // 16
        assert all(p >= 0 for p in table[:kept]) and all(p < 0 for p in table[kept:passed]) and all(p >= 0 for p in table[max(kept, passed):])
        assert all(p < 0 for p in cm.block_table(s, 1)[:passed])
        assert cm.defects() == 0
    first = cm.block_table(s, 0)[0]
    cm.release(s)
    assert cm.free_pages() == [64, 64] and cm.defects() == 0
    assert first >= 0


def test_kept_keys_need_a_window():
    with pytest.raises(AlofaError):
        CacheManager([GroupSpec(16, 8, None, 4)], max_requests=1, max_tokens=64)


def test_scheduler_books_the_kept_pages():
    """Two requests of 160 tokens over a window of 24 with 40 kept tokens hold three kept pages and up to four more each:
    the books never promise pages the kept ones take."""
    cfg = SchedConfig(token_budget=64, max_chunk=16, max_batch=2, max_tokens=256, watermark_permille=1000, groups=[(16, 24, 14, 40)])
    assert parse_config(format_config(cfg)) == cfg
    plain_cfg = SchedConfig(groups=[(16, 24, 14)])
    assert parse_config(format_config(plain_cfg)).groups == [(16, 24, 14)]
    cm = CacheManager([GroupSpec(16, 14, 24, 40)], max_requests=2, max_tokens=256)
    sched, slots, done = Scheduler(cfg), {}, []
    arrivals = [(1, 120, 40), (2, 120, 40)]
    for _ in range(400):
        act = sched.step(SchedInput(arrivals=arrivals, free_pages=cm.free_pages()))
        for (rid, *_), status in zip(list(arrivals), act.arrival_status):
            if status == 1:
                slots[rid] = cm.admit(rid)
        arrivals = [a for a, status in zip(arrivals, act.arrival_status) if status != 1]
        for rid, start, end in act.prefill:
            cm.reserve(slots[rid], end)  # raises when the books were wrong
            cm.advance(slots[rid], end)
        for rid in act.decode:
            n = cm.computed_len(slots[rid]) + 1
            cm.reserve(slots[rid], n)
            cm.advance(slots[rid], n)
        for rid in act.finished:
            cm.release(slots.pop(rid))
            done.append(rid)
        assert cm.defects() == 0
        if len(done) == 2:
            break
    assert sorted(done) == [1, 2] and cm.free_pages() == [14]


# ---- the plain implementation's own properties -------------------------------------------------------------------
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_plain_positions_depend_on_their_prefix_alone(folders, name):
    w, cfg = plain.load(folders[name])
    ids = tiny.tokens(name, 45)
    np.testing.assert_allclose(plain.forward(w, cfg, ids[:27]), plain.forward(w, cfg, ids)[:27], rtol=1e-9, atol=1e-9)


def test_plain_window_and_kept_tokens():
    m = plain.window_mask(12, 4, 2)
    assert m[3, :4].all() and m[9].tolist() == [True, True] + [False] * 4 + [True] * 4 + [False] * 2
    assert (plain.window_mask(6) == np.tri(6, dtype=bool)).all() and (plain.window_mask(6, 100, 3) == np.tri(6, dtype=bool)).all()
    assert (plain.window_mask(5, 1, 0) == np.eye(5, dtype=bool)).all()


def test_plain_bias_and_sink():
    np.testing.assert_allclose(plain.slopes(2), [1 / 16, 1 / 256])
    np.testing.assert_allclose(plain.slopes(3)[2], 1 / 256)
    # equal scores: weights fall off by exp(-slope) a step back, and the sink takes its share without adding a value
    T, v = 5, np.arange(5.0)[:, None, None]
    out = plain.biased_attention(np.zeros((T, 1, 1)), np.zeros((T, 1, 1)), v, 1.0, plain.window_mask(T), np.array([0.7]))
    slope = 2.0 ** -8
    e = np.exp(-slope * (4 - np.arange(5.0)))
    assert out[4, 0, 0] == pytest.approx((e * np.arange(5.0)).sum() / (e.sum() + math.exp(0.7)))
    # not the same as adding slope * j to the scores: the sink would weigh less and less
    moved = np.exp(slope * np.arange(5.0))
    assert out[4, 0, 0] != pytest.approx((moved * np.arange(5.0)).sum() / (moved.sum() + math.exp(0.7)))


def test_plain_norms_span_all_heads_and_values_are_mixed():
    rng = np.random.default_rng(0)
    m = {"heads": 2, "kv_heads": 2, "dim": 3, "vdim": 2, "scale": 1.0}
    width = 6 + 6 + 4 + 2
    eye = np.eye(width)
    w = {"a.q": eye[:6], "a.k": eye[6:12], "a.v": eye[12:16], "a.g": eye[16:], "a.o": np.eye(4), "a.q.norm": np.ones(6), "a.k.norm": np.ones(6), "a.sink": np.full(2, -1e9), "a.vmix": np.array(0.25)}
    h = rng.standard_normal((1, width))
    first = rng.standard_normal((1, 4))
    out, own = plain.attention(w, "a.", m, h, 1e-6, first)
    np.testing.assert_allclose(own, h[:, 12:16])
    gate = np.repeat(plain.sigmoid(h[:, 16:]), 2, axis=1)
    np.testing.assert_allclose(out, (0.75 * h[:, 12:16] + 0.25 * first) * gate)  # one token sees itself alone
    # a large first head takes most of the root mean square: the second head's query is small beside it
    h[0, :3] = 100.0
    q = plain.rms_norm(h[:, :6], np.ones(6), 1e-6)
    assert np.abs(q[0, 3:]).max() < 0.1 and np.abs(q[0, :3]).max() == pytest.approx(math.sqrt(2.0), rel=1e-3)


def test_plain_layer_norm():
    x = np.array([[1.0, 3.0, 5.0, 7.0]])
    np.testing.assert_allclose(plain.layer_norm(x, np.array([1.0, 2.0, 1.0, 1.0]), np.array([0.0, 0.0, 0.5, 0.0]), 0.0), [[-3 / math.sqrt(5), -2 / math.sqrt(5), 1 / math.sqrt(5) + 0.5, 3 / math.sqrt(5)]])


def test_plain_delta_rule_by_hand():
    rng = np.random.default_rng(1)
    q, k = plain.unit(rng.standard_normal((3, 1, 4))), plain.unit(rng.standard_normal((3, 1, 4)))
    v, beta, g = rng.standard_normal((3, 2, 2)), rng.uniform(0.2, 1, (3, 2)), rng.uniform(0.5, 1, (3, 2))
    out = plain.delta_recurrence(q, k, v, beta, g)
    np.testing.assert_allclose(out[0, 1], beta[0, 1] * v[0, 1] * (k[0, 0] @ q[0, 0]))  # the read-out sees the token's own write
    S = np.outer(k[0, 0], beta[0, 1] * v[0, 1]) * g[1, 1]
    S = S + np.outer(k[1, 0], beta[1, 1] * (v[1, 1] - S.T @ k[1, 0]))
    np.testing.assert_allclose(out[1, 1], S.T @ q[1, 0])
    # beta = 1, no decay and the same key again: the old value is replaced, not added to
    same = plain.delta_recurrence(np.repeat(k[:1], 2, 0), np.repeat(k[:1], 2, 0), v[:2], np.ones((2, 2)), np.ones((2, 2)))
    np.testing.assert_allclose(same[1], v[1], rtol=1e-5, atol=1e-5)


def test_plain_clamped_gate():
    w = {"m.gate": np.array([[1.0]]), "m.up": np.array([[1.0]]), "m.down": np.array([[1.0]])}
    for h, g, u in ((0.5, 0.5, 0.5), (9.0, 1.25, 1.25), (-9.0, -9.0, -1.25)):  # g is held from above only
        want = g / (1 + math.exp(-1.702 * g)) * (u + 1)
        assert plain.clamped_gated(w, "m.", np.array([[h]]), 1.25)[0, 0] == pytest.approx(want)


def test_plain_router_takes_the_best_groups_by_their_best():
    z = np.log(np.array([0.05, 0.3, 0.2, 0.19, 0.25, 0.01]))
    w = {"m.router": np.diag(z)}
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    # groups (0, 1), (2, 3), (4, 5): the first holds the largest score, although the second's two add up to more
    chosen, weights, margin = plain.route(w, "m.", r, np.ones((1, 6)))
    assert chosen[0].tolist() == [1, 0]
    np.testing.assert_allclose(weights[0], [0.3 / 0.35, 0.05 / 0.35])
    assert margin[0] == pytest.approx(1 - 0.25 / 0.3)
    assert plain.route(w, "m.", {"experts": 6, "top": 2}, np.ones((1, 6)))[0][0].tolist() == [1, 4]
