"""Gokapel: configuration, registry, tensor list, schedule and caches, and the plain implementation's mechanisms
against closed forms (all on the CPU)."""
import copy
import math

import pytest
import torch

import plain_gokapel as pg
from gokapel_cases import CASES, make_weights, tokens


def _spec(cfg):
    from tq_kv_b200.config import spec_from_config_dict
    return spec_from_config_dict(cfg)


def test_the_architecture_is_registered_and_a_configuration_round_trips():
    from tq_kv_b200.config import registered_architectures
    assert "Gokapel" in registered_architectures()
    kinds = {"channel_delta": "channel_delta_mixer", "parallel": "side_by_side"}
    for name, cfg in CASES.items():
        arch, typed, spec = _spec(cfg)
        back = typed.to_dict()
        assert arch.name == "Gokapel" and all(back[k] == cfg[k] for k in cfg), name
        own = [i for i, l in enumerate(cfg["layers"]) if l.get("weights_of") is None]
        assert [l.mixer.kind for l in spec.layers] == [kinds[cfg["layers"][i]["type"]] for i in own]
        assert all(l.block == "residual_streams" for l in spec.layers) and spec.residual_streams == cfg["streams"]
        assert [e.layer for e in spec.schedule] == [own.index(l.get("weights_of", i)) for i, l in enumerate(cfg["layers"])]
        assert all(e.cache_of is None for e in spec.schedule)
        assert spec.head.params["tied_to"] == "embed" and spec.embedding.params["scale"] == cfg["embedding"]["scale"]


@pytest.mark.parametrize("path,key", [((), "vocab"), ((), "width"), ((), "layers"), ((), "streams"), ((), "residual_mult"),
                                      (("embedding",), "scale"), (("norm",), "eps"),
                                      (("layers", 1, "mixer"), "conv"), (("layers", 1, "mixer"), "vdim"),
                                      (("layers", 0, "mixer"), "left"), (("layers", 0, "mixer"), "right_scale"),
                                      (("layers", 0, "mixer", "left"), "rot"), (("layers", 0, "mixer", "left", "rot"), "base"),
                                      (("layers", 0, "mixer", "left"), "scale"), (("layers", 0, "mixer", "right"), "width"),
                                      (("layers", 0, "mlp", "router"), "top"), (("layers", 0, "mlp", "router", "groups"), "keep"),
                                      (("layers", 0, "mlp", "expert"), "ff"), (("layers", 0, "mlp", "shared"), "ff"),
                                      (("layers", 1, "mlp"), "ff"), (("layers", 1), "type")])
def test_a_missing_key_is_named(path, key):
    from tq_kv_b200.config import ConfigError
    cfg = copy.deepcopy(CASES["a"])
    d = cfg
    for p in path:
        d = d[p]
    del d[key]
    with pytest.raises(ConfigError, match=key):
        _spec(cfg)


def test_sizes_that_contradict_each_other_are_refused():
    from tq_kv_b200.config import ConfigError

    def broken(change):
        cfg = copy.deepcopy(CASES["a"])
        change(cfg)
        with pytest.raises(ConfigError):
            _spec(cfg)

    broken(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4))         # 6 heads on 4 key heads
    broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=22))     # more rotated entries than the head has
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=9))      # an odd count
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4))  # 6 experts in 4 groups
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4))   # 4 of 3 groups
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=5))              # 5 of the 4 experts of two groups
    broken(lambda c: c["layers"][2].update(weights_of=9))
    broken(lambda c: c["layers"][2].update(weights_of=2))                        # itself
    broken(lambda c: c["layers"][2].update(weights_of=3))                        # a layer without tensors of its own
    broken(lambda c: c["layers"][2].update(weights_of=1))                        # a layer of another kind
    broken(lambda c: c["layers"][2]["mixer"].update(left_scale=0.1))             # not like the layer it names
    broken(lambda c: c["layers"][0].update(type="gru"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda c: c["norm"].update(eps=0.0))
    broken(lambda c: c.update(streams=0))


def test_the_model_asks_for_exactly_the_tensors_of_the_design_and_the_caches_its_mixers_need():
    from tq_kv_b200.engine import DecoderModel
    for name, cfg in CASES.items():
        w = make_weights(cfg, 3)
        model = DecoderModel(_spec(cfg)[2])
        specs = model.weight_specs()
        assert sorted(specs) == sorted(w), name
        for n, s in specs.items():
            assert len(s.shape) == w[n].dim() and all(a in (-1, b) for a, b in zip(s.shape, w[n].shape)), (name, n)
        kv, state = model.cache_requests()
        both = [i for i, l in enumerate(cfg["layers"]) if l["type"] == "parallel"]
        assert sorted(kv) == both and sorted(state) == list(range(len(cfg["layers"]))), name
        for i, l in enumerate(cfg["layers"]):
            m = l["mixer"]
            if i in both:
                assert kv[i].window == (m["left"].get("mask") or {}).get("size") and kv[i].n_kv_heads == m["left"]["kv_heads"]
                assert state[i].shape == (m["right"]["width"],)
            else:
                conv = (m["conv"] - 1) * (2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"])
                assert state[i].shape == (m["heads"] * m["dim"] * m["vdim"] + conv,)
            assert state[i].dtype == torch.float32


def test_random_weights_need_the_inner_widths_and_then_have_the_design_s_tensors(tmp_path):
    from tq_kv_b200.weights import write_model_folder
    with pytest.raises(ValueError, match="only a checkpoint gives"):
        write_model_folder(CASES["c"], str(tmp_path / "x"), 11)
    cfg = copy.deepcopy(CASES["c"])
    for l in cfg["layers"]:
        if l["type"] == "channel_delta":
            l["mixer"].update(decay_rank=10, gate_rank=14)
    path = write_model_folder(cfg, str(tmp_path / "m"), 11)
    back, w = pg.read_folder(path)
    want = make_weights(CASES["c"], 1)
    assert {n: tuple(t.shape) for n, t in w.items()} == {n: tuple(t.shape) for n, t in want.items()}
    assert back["layers"] == cfg["layers"] and back["architecture"] == "Gokapel"
    logits = pg.decoder(back, w, tokens(20, back["vocab"], 2))
    assert logits.shape == (20, back["vocab"]) and torch.isfinite(logits).all()


# ---- the plain implementation's mechanisms against closed forms -----------------------------------------------------
def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_the_convolution_and_the_unit_vectors():
    x, taps = _rand(9, 3, seed=1), _rand(3, 4, seed=2)
    y = pg.short_conv(x, taps)
    for t in range(9):
        for c in range(3):
            z = sum(float(taps[c, 3 - j] * x[t - j, c]) for j in range(4) if t >= j)
            assert abs(float(y[t, c]) - z / (1.0 + math.exp(-z))) < 1e-12
    u = pg.unit(torch.tensor([[3.0, 4.0], [0.0, 0.0]], dtype=torch.float64))
    assert abs(float(u[0].norm()) - 1.0) < 1e-7 and torch.equal(u[1], torch.zeros(2, dtype=torch.float64))


def test_the_delta_rule_replaces_what_the_state_holds_along_a_key():
    """With no decay and beta = 1 the state answers a key with the value written last; a decay per key channel fades
    that channel's row; a later read of an orthogonal key is untouched."""
    d, e = 4, 3
    eye = torch.eye(d, dtype=torch.float64)
    k = torch.stack([eye[0], eye[1], eye[0], eye[1]]).reshape(4, 1, d)
    v = _rand(4, 1, e, seed=3)
    one = torch.ones(4, 1, dtype=torch.float64)
    out = pg.delta_scan(k, k, v, torch.ones(4, 1, d, dtype=torch.float64), one)
    assert torch.allclose(out[:, 0], v[:, 0], atol=1e-12)                    # every read sees its own write
    q = eye[0].expand(4, 1, d)
    assert torch.allclose(pg.delta_scan(q, k, v, torch.ones(4, 1, d, dtype=torch.float64), one)[:, 0], v[[0, 0, 2, 2], 0], atol=1e-12)
    g = torch.ones(4, 1, d, dtype=torch.float64)
    g[1, 0, 0] = 0.25                                                        # at token 1 channel 0 fades
    out = pg.delta_scan(q, k, v, g, one)
    assert torch.allclose(out[1, 0], 0.25 * v[0, 0], atol=1e-12) and torch.allclose(out[2, 0], v[2, 0], atol=1e-12)
    # in general: S_t = (I - beta k k^T) diag(g) S_{t-1} + beta k v^T, and two heads share a key head
    T = 6
    q, k = pg.unit(_rand(T, 1, d, seed=4)), pg.unit(_rand(T, 1, d, seed=5))
    v, g, beta = _rand(T, 2, e, seed=6), torch.sigmoid(_rand(T, 2, d, seed=7)), torch.sigmoid(_rand(T, 2, seed=8))
    out = pg.delta_scan(q, k, v, g, beta)
    for h in range(2):
        S = torch.zeros(d, e, dtype=torch.float64)
        for t in range(T):
            kk = k[t, 0].reshape(d, 1)
            S = (torch.eye(d, dtype=torch.float64) - beta[t, h] * kk @ kk.T) @ torch.diag(g[t, h]) @ S + beta[t, h] * kk @ v[t, h].reshape(1, e)
            assert torch.allclose(out[t, h], S.T @ q[t, 0], atol=1e-12)


def test_the_gru_as_a_weighted_sum_over_the_past():
    z, c = torch.sigmoid(_rand(7, 3, seed=9)), _rand(7, 3, seed=10)
    out = pg.gru_scan(z, c)
    for t in range(7):
        want = sum(torch.prod(1.0 - z[s + 1:t + 1], dim=0) * z[s] * c[s] for s in range(t + 1))
        assert torch.allclose(out[t], want, atol=1e-12)


def test_rotation_turns_neighbours_and_depends_on_the_distance_only():
    q, k = _rand(1, 1, 24, seed=11), _rand(1, 1, 24, seed=12)
    dots = []
    for pq, pk in ((5, 2), (105, 102), (1003, 1000)):
        a, b = pg.rotate(q, torch.tensor([pq]), 16, 1e4), pg.rotate(k, torch.tensor([pk]), 16, 1e4)
        assert torch.equal(a[..., 16:], q[..., 16:])
        dots.append(float((a * b).sum()))
    assert max(dots) - min(dots) < 1e-9
    x = torch.zeros(1, 1, 16, dtype=torch.float64)
    x[..., 2] = 1.0
    y = pg.rotate(x, torch.tensor([3]), 16, 1e4)[0, 0]
    t = 3.0 * 1e4 ** (-2.0 / 16.0)
    assert float(y[2]) == pytest.approx(math.cos(t)) and float(y[3]) == pytest.approx(math.sin(t))


def test_the_chunks_and_the_sink():
    assert pg.visible(7, 3).tolist() == [[j <= i and i // 3 == j // 3 for j in range(7)] for i in range(7)]
    assert pg.visible(4, None).tolist() == [[j <= i for j in range(4)] for i in range(4)]
    assert pg.visible(4, 1).tolist() == torch.eye(4, dtype=torch.bool).tolist()
    q, k, v = _rand(5, 2, 8, seed=13), _rand(5, 1, 8, seed=14), _rand(5, 1, 8, seed=15)
    sinks = torch.tensor([0.7, -40.0], dtype=torch.float64)
    out = pg.softmax_heads(q, k, v, 0.5, pg.visible(5, None), sinks)
    for t in range(5):
        for h in range(2):
            p = torch.exp(0.5 * k[:t + 1, 0] @ q[t, h])
            want = (p @ v[:t + 1, 0]) / (p.sum() + torch.exp(sinks[h]))
            assert torch.allclose(out[t, h], want, atol=1e-12)


def test_the_router_s_groups_correction_and_weights():
    z = torch.log(torch.tensor([[0.30, 0.05, 0.20, 0.15, 0.25, 0.05]], dtype=torch.float64))     # softmax gives these back
    none = torch.zeros(6, dtype=torch.float64)
    idx, wts, _ = pg.route(z, none, 2, 1, 1)
    assert idx.tolist() == [[0, 4]] and torch.allclose(wts, torch.tensor([[0.30, 0.25]], dtype=torch.float64))
    idx, wts, margin = pg.route(z, none, 2, 3, 1)                  # groups (0, 1), (2, 3), (4, 5): the first is best
    assert idx.tolist() == [[0, 1]] and torch.allclose(wts, torch.tensor([[0.30, 0.05]], dtype=torch.float64))
    assert float(margin) == pytest.approx(0.05)                    # 0.30 against the second group's 0.25
    # a correction moves the choice, not the weights; choice scores may all be negative
    corr = torch.tensor([-1.0, -1.0, -0.5, -0.6, -1.0, -1.0], dtype=torch.float64)
    idx, wts, _ = pg.route(z, corr, 2, 3, 1)
    assert idx.tolist() == [[2, 3]] and torch.allclose(wts, torch.tensor([[0.20, 0.15]], dtype=torch.float64))
    idx, _, _ = pg.route(z, corr, 3, 3, 2)
    assert idx.tolist() == [[2, 3, 0]]


def test_a_sublayer_reads_scales_gates_and_writes_the_streams():
    cfg = CASES["a"]
    w = {n: t.double() for n, t in make_weights(cfg, 6).items()}
    toks = tokens(30, cfg["vocab"], 7)
    layers = []
    pg.decoder(cfg, w, toks, layers_out=layers)
    x = [w["embed"][torch.tensor(toks)] * 3.0] * 3
    for q, f in ((1, lambda h: pg.parallel(h, w, "l0.mix.", cfg["layers"][0]["mixer"], torch.arange(30), 1e-6)),
                 (2, lambda h: pg.routed_ff(h, w, "l0.mlp.", cfg["layers"][0]["mlp"]))):
        u = sum(w[f"l0.hc{q}.in"][s] * x[s] for s in range(3))
        h = torch.tanh(w[f"l0.norm{q}.alpha"] * u) * w[f"l0.norm{q}"] + w[f"l0.norm{q}.b"]
        y = f(h) * w[f"l0.ls{q}"] / (1.0 + torch.exp(-(h @ w[f"l0.rg{q}"].T + w[f"l0.rg{q}.b"])))
        x = [sum(w[f"l0.hc{q}.mix"][s, t] * x[s] for s in range(3)) + 0.8 * w[f"l0.hc{q}.out"][t] * y for t in range(3)]
    assert torch.allclose(layers[0], sum(x), atol=1e-10)
    z = torch.linspace(-2, 2, 5, dtype=torch.float64)
    assert torch.equal(pg.square_relu(z), torch.tensor([0.0, 0.0, 0.0, 1.0, 4.0], dtype=torch.float64))
    assert torch.allclose(pg.softplus(z), torch.nn.functional.softplus(z), atol=1e-12)
