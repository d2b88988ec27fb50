"""Safurax: configuration, registry, tensor list, schedule and caches, and the plain implementation's mechanisms
against closed forms (all on the CPU)."""
import copy
import math

import pytest
import torch

import plain_safurax as ps
from safurax_cases import CASES, make_weights, tokens


def _spec(cfg):
    from tq_kv_b200.config import spec_from_config_dict
    return spec_from_config_dict(cfg)


def test_the_architecture_is_registered_and_a_configuration_round_trips():
    from tq_kv_b200.config import named_shape, registered_architectures
    assert "Safurax" in registered_architectures()
    kinds = {"latent_attention": "latent_attention", "latent_attention_2": "latent_attention", "attention": "softmax_attention"}
    for name, cfg in [*CASES.items(), ("named shape", named_shape("safurax-tiny"))]:
        arch, typed, spec = _spec(cfg)
        back = typed.to_dict()
        assert arch.name == "Safurax" and all(back[k] == cfg[k] for k in cfg), name
        assert all(l.block == "prenorm_residual" and l.mixer_norm.kind == "layer_norm" for l in spec.layers)
        assert [l.mixer.kind for l in spec.layers] == [kinds[x["type"]] for x in cfg["layers"]]
        assert [l.feed_forward is None for l in spec.layers] == [x["mlp"] is None for x in cfg["layers"]]
        assert [e.layer for e in spec.schedule] == list(range(len(cfg["layers"])))
        assert [e.cache_of for e in spec.schedule] == [x["mixer"].get("kv_from") for x in cfg["layers"]]
        assert spec.embedding.params["scale"] == cfg["embedding"]["scale"] and spec.final_norm.kind == "layer_norm"


@pytest.mark.parametrize("path,key", [((), "vocab"), ((), "width"), ((), "layers"), (("norm",), "eps"), ((), "embedding"),
                                      (("embedding",), "scale"),
                                      (("layers", 0, "mixer"), "rot_dim"), (("layers", 0, "mixer"), "rot"),
                                      (("layers", 0, "mixer", "mask"), "size"), (("layers", 0, "mixer"), "kv_rank"),
                                      (("layers", 1, "mixer"), "diff"), (("layers", 1, "mixer", "rot"), "base"),
                                      (("layers", 1, "mixer", "rot", "scaling"), "factor"),
                                      (("layers", 1, "mixer"), "kv_heads"), (("layers", 1, "mixer"), "scale"),
                                      (("layers", 2, "mixer"), "q_rank"), (("layers", 2, "mixer"), "vdim"),
                                      (("layers", 0, "mlp", "router"), "top"), (("layers", 0, "mlp", "router"), "experts"),
                                      (("layers", 0, "mlp", "expert"), "ff"), (("layers", 0, "mlp", "shared"), "ff"),
                                      (("layers", 1, "mlp"), "ff"), (("layers", 2), "type")])
def test_a_missing_key_is_named(path, key):
    from tq_kv_b200.config import ConfigError
    cfg = copy.deepcopy(CASES["a"])
    d = cfg
    for p in path:
        d = d[p]
    del d[key]
    if key == "size":                                       # a mask without a size is no window
        assert _spec(cfg)[2].layers[0].mixer.params["window"] is None
        return
    with pytest.raises(ConfigError, match=key):
        _spec(cfg)


def test_sizes_that_contradict_each_other_are_refused():
    from tq_kv_b200.config import ConfigError

    def broken(change):
        cfg = copy.deepcopy(CASES["a"])
        change(cfg)
        with pytest.raises(ConfigError):
            _spec(cfg)

    broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))                 # 6 heads on 4 key heads
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=22))             # more rotated entries than the map has
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=9))              # an odd count
    broken(lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10))             # beyond the rotated part
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=3))                  # itself
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=2))                  # a latent of the other kind
    broken(lambda c: c["layers"][3]["mixer"].update(kv_rank=40))                 # other rows than layer 0 caches
    broken(lambda c: c["layers"][3]["mixer"]["rot"].update(base=10000.0))        # another rotation
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))              # 7 of 6 experts
    broken(lambda c: c["layers"][0].update(type="latent"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda c: c["norm"].update(eps=0.0))
    cfg = copy.deepcopy(CASES["a"])
    cfg["layers"].insert(0, copy.deepcopy(cfg["layers"][3]))                     # reads a layer that comes later (itself)
    with pytest.raises(ConfigError):
        _spec(cfg)


def test_the_model_asks_for_exactly_the_tensors_of_the_design_and_the_caches_its_mixers_need():
    from tq_kv_b200.engine import DecoderModel
    for name, cfg in CASES.items():
        w = make_weights(cfg, 3)
        model = DecoderModel(_spec(cfg)[2])
        specs = model.weight_specs()
        assert sorted(specs) == sorted(w), name
        for n, s in specs.items():
            assert tuple(s.shape) == tuple(w[n].shape), (name, n)
        assert model.padded_rows_ok and model.graph_capturable
        kv, state = model.cache_requests()
        own = [i for i, l in enumerate(cfg["layers"]) if l["mixer"].get("kv_from") is None]
        assert sorted(kv) == own and not state, name
        for i in own:
            m = cfg["layers"][i]["mixer"]
            if cfg["layers"][i]["type"] == "attention":     # rows that hold both maps, and the values once
                assert kv[i].n_kv_heads == m["kv_heads"] and kv[i].head_dim >= 2 * m["dim"] and kv[i].window is None
                assert (kv[i].value_dim or kv[i].head_dim) >= m["vdim"]
                continue
            assert kv[i].n_kv_heads == 1 and kv[i].head_dim >= m["kv_rank"] + m.get("rot_dim", 0)
            ws = [(m.get("mask") or {}).get("size")] + [(l["mixer"].get("mask") or {}).get("size")
                                                        for l in cfg["layers"] if l["mixer"].get("kv_from") == i]
            assert kv[i].window == (None if None in ws else max(ws)), (name, i)


def test_a_difference_of_maps_refuses_what_it_cannot_combine_with():
    from tq_kv_b200.config import ConfigError
    from tq_kv_b200.parts import make_part
    from tq_kv_b200.config import PartSpec
    base = {"hidden_size": 64, "num_heads": 2, "num_kv_heads": 1, "key_dim": 16, "value_dim": 32, "scale": 0.25,
            "difference": {"offset": 0.3, "eps": 1e-5}}
    make_part(PartSpec("softmax_attention", base))
    for extra in ({"sink": "learned"}, {"output_gate": True}, {"values": "keys", "value_dim": 16}, {"slope_exponent": 8.0},
                  {"result_scale": 2.0}, {"shared_kv": True}):
        with pytest.raises(ConfigError):
            make_part(PartSpec("softmax_attention", {**base, **extra}))


def test_random_weights_of_a_configuration_have_the_design_s_tensors(tmp_path):
    from tq_kv_b200.weights import write_model_folder
    path = write_model_folder(CASES["c"], str(tmp_path / "m"), 11)
    cfg, w = ps.read_folder(path)
    assert sorted(w) == sorted(make_weights(CASES["c"], 1))
    assert cfg["layers"] == CASES["c"]["layers"] and cfg["architecture"] == "Safurax"
    logits = ps.decoder(cfg, w, tokens(20, cfg["vocab"], 2))
    assert logits.shape == (20, cfg["vocab"]) and torch.isfinite(logits).all()


def test_the_rates_of_the_product_s_tables_are_divided_by_the_factor():
    from tq_kv_b200.config import PartSpec
    from tq_kv_b200.parts import Runtime, make_part
    part = make_part(PartSpec("rotary_tables", {"rotary_dim": 8, "theta": 1e4, "layout": "halves", "rate_divisor": 4.0}))
    rt = Runtime(torch.device("cpu"), torch.float32, 300)
    shared: dict = {}
    part.prepare(rt, shared)
    for p in (0, 1, 17, 299):
        for i in range(4):
            a = p * 1e4 ** (-2 * i / 8) / 4.0
            assert float(part.cos[p, i]) == pytest.approx(math.cos(a), abs=1e-6) and float(part.sin[p, i]) == pytest.approx(math.sin(a), abs=1e-6)
    other = make_part(PartSpec("rotary_tables", {"rotary_dim": 8, "theta": 1e4, "layout": "halves"}))
    other.prepare(rt, shared)                               # the shared tables are told apart
    assert not torch.equal(other.cos, part.cos)


# ---- the plain implementation's mechanisms against closed forms -----------------------------------------------------
def test_the_layer_norm_ignores_shifts_and_scales():
    g = torch.Generator().manual_seed(1)
    x, w = torch.randn(3, 10, generator=g, dtype=torch.float64), torch.randn(10, generator=g, dtype=torch.float64)
    y = ps.layer_norm(x, w, 1e-12)
    assert torch.allclose(ps.layer_norm(5.0 * x + 7.0, w, 1e-12), y, atol=1e-9)
    assert torch.allclose(y, torch.nn.functional.layer_norm(x, (10,), w, None, 1e-12), atol=1e-12)
    assert float((y / w).mean().abs()) < 1e-12


def test_rotation_depends_on_the_distance_only_and_a_factor_stretches_it():
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 1, 24, generator=g, dtype=torch.float64), torch.randn(1, 1, 24, generator=g, dtype=torch.float64)
    for factor in (1.0, 8.0):
        dots = []
        for pq, pk in ((5, 2), (105, 102), (1003, 1000)):
            a, b = ps.rotate(q, torch.tensor([pq]), 16, 1e4, factor), ps.rotate(k, torch.tensor([pk]), 16, 1e4, factor)
            assert torch.allclose(a[..., 16:], q[..., 16:]) and float(a.norm()) == pytest.approx(float(q.norm()))
            dots.append(float((a * b).sum()))
        assert max(dots) - min(dots) < 1e-9
    assert torch.allclose(ps.rotate(q, torch.tensor([40]), 16, 1e4, 8.0), ps.rotate(q, torch.tensor([5]), 16, 1e4), atol=1e-12)


def test_the_window_and_the_sink():
    assert ps.visible(6, 3).tolist() == [[j <= i and i - j < 3 for j in range(6)] for i in range(6)]
    assert ps.visible(4).tolist() == [[j <= i for j in range(4)] for i in range(4)]
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(5, 8, generator=g, dtype=torch.float64) for _ in range(3))
    s = torch.tensor(1.3, dtype=torch.float64)
    sunk = ps.softmax_head(q, k, v, 0.5, ps.visible(5), s)
    for i in range(5):                                      # by hand: the sink counts once and carries nothing
        e = torch.exp((k[:i + 1] @ q[i]) * 0.5)
        assert torch.allclose(sunk[i], (e / (e.sum() + math.exp(1.3))) @ v[:i + 1], atol=1e-12)


def test_the_difference_of_maps_by_hand():
    g = torch.Generator().manual_seed(4)
    W, T, H, G, d, e = 12, 7, 4, 2, 6, 5
    c = {"heads": H, "kv_heads": G, "dim": d, "vdim": e, "scale": 0.4, "diff": 0.3,
         "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0}}}
    shapes = {"q": (H * 2 * d, W), "k": (G * 2 * d, W), "v": (G * e, W), "g": (H, W), "q.norm": (d,), "k.norm": (d,),
              "lq1": (d,), "lk1": (d,), "lq2": (d,), "lk2": (d,)}
    w = {"m." + n: torch.randn(*s, generator=g, dtype=torch.float64) * 0.5 for n, s in shapes.items()}
    w["m.o"] = torch.eye(H * e, dtype=torch.float64)
    x = torch.randn(T, W, generator=g, dtype=torch.float64)
    got = ps.differential_attention(x, w, "m.", c, torch.arange(T), 1e-6).reshape(T, H, e)
    lam = math.exp(float(w["m.lq1"] @ w["m.lk1"])) - math.exp(float(w["m.lq2"] @ w["m.lk2"])) + 0.3
    assert float(ps.difference_factor(w, "m.", 0.3)) == pytest.approx(lam)

    def vector(mat, row, t, weight):
        y = mat[row * d:(row + 1) * d] @ x[t]
        y = y / torch.sqrt((y * y).mean() + 1e-6) * weight
        out = y.clone()
        for i in range(2):
            a = t * 100.0 ** (-2 * i / 4) / 2.0
            out[i] = y[i] * math.cos(a) - y[i + 2] * math.sin(a)
            out[i + 2] = y[i + 2] * math.cos(a) + y[i] * math.sin(a)
        return out

    for t in (0, 3, 6):
        for h in range(H):
            kv = h // 2
            maps = []
            for m in (0, 1):
                q = vector(w["m.q"], 2 * h + m, t, w["m.q.norm"])
                s = torch.stack([0.4 * q @ vector(w["m.k"], 2 * kv + m, j, w["m.k.norm"]) for j in range(t + 1)])
                maps.append(torch.softmax(s, 0) @ (x[:t + 1] @ w["m.v"][kv * e:(kv + 1) * e].T))
            o = maps[0] - lam * maps[1]
            o = o / torch.sqrt((o * o).mean() + 1e-6) * 0.7 * torch.sigmoid(w["m.g"][h] @ x[t])
            assert torch.allclose(got[t, h], o, atol=1e-10), (t, h)


def test_the_chosen_experts_softmax_and_the_gated_shared_expert():
    cfg = {"kind": "moe", "expert": {"ff": 6}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 4}}
    g = torch.Generator().manual_seed(5)
    W = 8
    w = {"p.router": torch.randn(5, W, generator=g, dtype=torch.float64), "p.router.b": torch.randn(5, generator=g, dtype=torch.float64),
         "p.shared.sg": torch.randn(1, W, generator=g, dtype=torch.float64)}
    for n in [f"e{i}." for i in range(5)] + ["shared."]:
        f = 4 if n == "shared." else 6
        w["p." + n + "gate"], w["p." + n + "up"] = (torch.randn(f, W, generator=g, dtype=torch.float64) for _ in range(2))
        w["p." + n + "down"] = torch.randn(W, f, generator=g, dtype=torch.float64)
    x = torch.randn(3, W, generator=g, dtype=torch.float64)
    got = ps.routed_ff(x, w, "p.", cfg)
    for t in range(3):
        z = w["p.router"] @ x[t] + w["p.router.b"]
        a, b = sorted(range(5), key=lambda i: -float(z[i]))[:2]
        p = 1.0 / (1.0 + math.exp(float(z[b] - z[a])))
        want = p * ps.gated_ff(x[t:t + 1], w, f"p.e{a}.")[0] + (1.0 - p) * ps.gated_ff(x[t:t + 1], w, f"p.e{b}.")[0]
        want = want + ps.gated_ff(x[t:t + 1], w, "p.shared.")[0] / (1.0 + math.exp(-float(w["p.shared.sg"][0] @ x[t])))
        assert torch.allclose(got[t], want, atol=1e-12)


def test_a_layer_norms_what_its_sublayers_read_and_shared_latents_are_the_other_layer_s():
    cfg = copy.deepcopy(CASES["a"])
    w = make_weights(cfg, 6)
    toks = tokens(40, cfg["vocab"], 7)
    layers = []
    ps.decoder(cfg, w, toks, layers_out=layers)
    wd = {k: v.double() for k, v in w.items()}
    pos = torch.arange(40)
    x0 = wd["embed"][torch.tensor(toks)] * 2.0
    n = ps.layer_norm(x0, wd["l0.norm1"], 1e-6)
    kept = ps.latent_of(n, wd, "l0.mix.", cfg["layers"][0]["mixer"], pos, 1e-6)
    x1 = x0 + ps.latent_attention_2(n, wd, "l0.mix.", cfg["layers"][0]["mixer"], pos, 1e-6, kept)
    x1 = x1 + ps.feed_forward(ps.layer_norm(x1, wd["l0.norm2"], 1e-6), wd, "l0.mlp.", cfg["layers"][0]["mlp"])
    assert torch.allclose(layers[0], x1, atol=1e-10)
    # layer 3 reads layer 0's latents (made from layer 0's input), with its own queries, window, sink and gate
    n = ps.layer_norm(layers[2], wd["l3.norm1"], 1e-6)
    x3 = layers[2] + ps.latent_attention_2(n, wd, "l3.mix.", cfg["layers"][3]["mixer"], pos, 1e-6, kept)
    x3 = x3 + ps.feed_forward(ps.layer_norm(x3, wd["l3.norm2"], 1e-6), wd, "l3.mlp.", cfg["layers"][3]["mlp"])
    assert torch.allclose(layers[3], x3, atol=1e-10)
