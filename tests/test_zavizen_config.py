"""The Zavizen configuration on the CPU: keys, the parts it names, tensor names and shapes, looped layers, what each layer
asks of the cache manager, refusals, the residual streams' bookkeeping, and the plain implementation's own consistency."""

import copy
import math

import pytest
import torch

import plain_zavizen as plain
import zavizen_cases as Z


def test_the_specification_names_every_tensor_the_plain_implementation_reads():
    from llm_pipeline_b200.config import resolve_config
    from llm_pipeline_b200.models import build_model

    for name, cfg in Z.CONFIGS.items():
        config = resolve_config(cfg)
        model = build_model(config)
        expected = {n: tuple(s.shape) for n, s in model.expected_params().items() if not s.optional}
        W = Z.weights_for(cfg, 0)
        assert expected == {n: tuple(t.shape) for n, t in W.items()}, name
        plain.forward(cfg, W, [1, 2, 3])                                         # and the oracle needs no other
        assert config.to_json() == cfg, name
        assert resolve_config(config.to_json()).model_spec() == config.model_spec()
        assert config.parameter_counts()["total_parameters"] == sum(t.numel() for t in W.values())
        # a layer without a feed-forward may find the second sublayer's small tensors in a checkpoint, and reads none of them
        spare = {n for n, s in model.expected_params().items() if s.optional}
        assert spare == {f"l{i}.{n}" for i, layer in enumerate(cfg["layers"]) if layer["mlp"] is None
                         for n in ("norm2", "ls2", "hc2.in", "hc2.out", "hc2.mix")}


def test_looped_layers_and_what_they_ask_of_the_cache_manager():
    from llm_pipeline_b200.cache.spec import HeadRowPagesSpec, StateSpec
    from llm_pipeline_b200.config import resolve_config
    from llm_pipeline_b200.models import build_model

    model = build_model(resolve_config(Z.CONFIGS["mixed"]))
    assert [e.layer for e in model.schedule] == [0, 1, 2, 1, 2, 3] == plain.layer_order(Z.CONFIGS["mixed"])
    assert [e.cache for e in model.schedule] == list(range(6))                   # every pass has a cache and a state of its own
    specs = model.cache_specs()
    assert specs[0] == (HeadRowPagesSpec(2, 40), StateSpec((2 * 3 * 16 * 20,)))
    assert specs[1] == specs[3] == (None, StateSpec((2 * 3 * (4 * 16 + 2 * 2 * 24) + 2 * 4 * 24 * 16,)))
    assert specs[2] == specs[4] == (HeadRowPagesSpec(1, 64), StateSpec((2 * 2 * 24 * 16,)))
    assert specs[5][0] is None
    assert model.pieces() == [(0, 6, True)]                                      # a decode step is one captured graph
    assert model.settled_shape(7) == (7, 3, 64)
    for loop, order in (((0, 4, 1), [0, 1, 2, 3]), ((3, 4, 3), [0, 1, 2, 3, 3, 3]), ((2, 2, 5), [0, 1, 2, 3])):
        cfg = {**Z.CONFIGS["mixed"], "loop": dict(zip(("start", "stop", "times"), loop))}
        assert resolve_config(cfg).layer_order() == order == plain.layer_order(cfg)
    # rotations of equal size, base and factor are one table; others are their own
    spec = resolve_config(Z.CONFIGS["mixed"]).model_spec()
    assert len(spec.positions) == 4 and spec.layers[2].mixer.args["left"]["args"]["rotary_dim"] == 32


@pytest.mark.parametrize("damage, message", [
    (lambda c: c["layers"][0].update(type="lstm"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "lacks"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "lacks"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("decay"), "lacks"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "cannot share"),
    (lambda c: c["layers"][0]["mixer"]["right"]["decay"].pop(), "one constant per head"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["right"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].pop("base"), "rot.base"),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "positive factor"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "cannot share"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mlp"].update(kind="conv"), "unknown mlp kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "needs ff"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "expert.ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "cannot use 9 of 8"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "equal groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=1), "do not hold 3"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "needs shared.ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].pop("times"), "loop lacks"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("norm"), "required keys"),
    (lambda c: c.update(layers=[]), "required keys|no layers"),
])
def test_refusals(damage, message):
    from llm_pipeline_b200.config import resolve_config

    cfg = copy.deepcopy(Z.CONFIGS["mixed"])
    damage(cfg)
    with pytest.raises(ValueError, match=message):
        resolve_config(cfg)


def test_linear_scaling_divides_the_frequencies():
    from llm_pipeline_b200.parts.position import RotaryPositions

    plain_f = RotaryPositions("", 8, 100.0)._inv_freq_cpu
    scaled = RotaryPositions("", 8, 100.0, frequency_scaling={"kind": "linear", "factor": 4.0})._inv_freq_cpu
    assert torch.allclose(scaled * 4.0, plain_f, rtol=1e-6)
    with pytest.raises(ValueError, match="positive factor"):
        RotaryPositions("", 8, 100.0, frequency_scaling={"kind": "linear", "factor": 0.0})


def test_the_streams_keep_one_update_pending():
    from llm_pipeline_b200.parts import Addend, HyperStream
    from llm_pipeline_b200.parts.hyper_connections import HyperConnection

    stream = HyperStream(torch.arange(6.0).view(2, 3), 4)
    assert stream.settle().shape == (2, 4, 3) and torch.equal(stream.residual[:, 3], torch.arange(6.0).view(2, 3))
    connection = HyperConnection("c", 4, 3)
    stream.update([Addend(torch.zeros(2, 3))], connection)
    with pytest.raises(RuntimeError, match="pending"):
        stream.update([Addend(torch.zeros(2, 3))], connection)
    with pytest.raises(RuntimeError, match="hyper-connections"):
        stream.add(torch.zeros(2, 3))
    with pytest.raises(ValueError, match="streams"):
        HyperConnection("c", 17, 3)


def test_the_plain_implementation_is_causal_and_its_mechanisms_have_their_closed_forms():
    F = torch.float64
    cfg = Z.CONFIGS["mixed"]
    W = Z.weights_for(cfg, 1)
    tokens = [t % cfg["vocab"] for t in range(3, 60)]
    whole = plain.forward(cfg, W, tokens)
    assert (plain.forward(cfg, W, tokens[:17]) - whole[:17]).abs().max() < 1e-9
    # retention with a decay of one and keys that are the queries sums (q . k) v; a state handed on gives the same rows
    gen = torch.Generator().manual_seed(1)
    q, k = (torch.randn(9, 2, 5, generator=gen, dtype=F) for _ in range(2))
    v = torch.randn(9, 2, 3, generator=gen, dtype=F)
    a = torch.tensor([1.0, 0.5], dtype=F)
    o, _ = plain.retention_scan(q, k, v, a)
    want = sum(a[:, None] ** (8 - j) * (q[8] * k[j]).sum(-1, keepdim=True) * v[j] for j in range(9))
    assert torch.allclose(o[8], want)
    head, S = plain.retention_scan(q[:4], k[:4], v[:4], a)
    tail, _ = plain.retention_scan(q[4:], k[4:], v[4:], a, S)
    assert torch.allclose(torch.cat([head, tail]), o)
    # the rotation keeps lengths, leaves the entries past its size alone and turns pair (1, 5) by its scaled frequency
    x = torch.randn(6, 2, 12, generator=gen, dtype=F)
    r = plain.rotate(x, Z.rot(8, 100.0, 2.0))
    assert torch.equal(r[..., 8:], x[..., 8:]) and (r.norm(dim=-1) - x.norm(dim=-1)).abs().max() < 1e-12 and torch.equal(r[0], x[0])
    one = torch.zeros(8, 1, 8, dtype=F)
    one[7, 0, 1] = 1.0
    turned, angle = plain.rotate(one, Z.rot(8, 100.0, 2.0))[7, 0], 7 * 100.0 ** (-2.0 / 8) / 2.0
    assert abs(float(turned[1]) - math.cos(angle)) < 1e-12 and abs(float(turned[5]) - math.sin(angle)) < 1e-12
    # the router: scores over all experts, the best group alone, weights that sum to the scale
    logits = torch.tensor([[3.0, -4.0, 2.0, 2.5, 1.0, 2.9]], dtype=F)
    chosen, w = plain.route(logits, torch.eye(6, dtype=F), {"experts": 6, "top": 2, "scale": 1.5, "groups": {"count": 3, "keep": 1}})
    s = torch.softmax(logits[0], 0)
    assert chosen.tolist() == [[0, 1]] and torch.allclose(w[0], 1.5 * s[:2] / s[:2].sum())
    chosen, _ = plain.route(logits, torch.eye(6, dtype=F), {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}})
    assert chosen.tolist() == [[0, 5]]
    chosen, _ = plain.route(logits, torch.eye(6, dtype=F), {"experts": 6, "top": 3})
    assert chosen.tolist() == [[0, 5, 3]]
    # hyper-connections with one stream, mix and out of one and no scale are a plain residual
    y = torch.randn(4, 3, generator=gen, dtype=F)
    one = {"l.hc1.in": torch.ones(1, dtype=F), "l.hc1.out": torch.ones(1, dtype=F), "l.hc1.mix": torch.ones(1, 1, dtype=F),
           "l.ls1": torch.ones(3, dtype=F), "l.norm1": torch.zeros(3, dtype=F)}
    x = torch.randn(1, 4, 3, generator=gen, dtype=F)
    assert torch.allclose(plain.sublayer(x, one, "l", 1, 1e-5, lambda h: y)[0], x[0] + y)
    two = {**one, "l.hc1.in": torch.tensor([1.0, 2.0], dtype=F), "l.hc1.out": torch.tensor([0.5, -1.0], dtype=F),
           "l.hc1.mix": torch.tensor([[0.0, 3.0], [5.0, 0.0]], dtype=F)}
    xs, seen = torch.randn(2, 4, 3, generator=gen, dtype=F), []
    out = plain.sublayer(xs, two, "l", 1, 1e-5, lambda h: seen.append(h) or y)
    assert torch.allclose(seen[0], plain.rms(xs[0] + 2 * xs[1], 1e-5))
    assert torch.allclose(out[0], 5 * xs[1] + 0.5 * y) and torch.allclose(out[1], 3 * xs[0] - y)         # mix is [from, to]


def test_a_random_model_folder_can_be_written_and_read_back(tmp_path):
    from llm_pipeline_b200.config import load_config
    from llm_pipeline_b200.models import build_model
    from llm_pipeline_b200.weights import write_random_model
    from llm_pipeline_b200.weights.source import SafetensorsSource, check_names_and_shapes

    folder = write_random_model(Z.CONFIGS["mixed"], 3, str(tmp_path))
    config = load_config(folder)
    assert config.architecture == "Zavizen" and config.loop == {"start": 1, "stop": 3, "times": 2}
    source = SafetensorsSource(folder)
    check_names_and_shapes(build_model(config).expected_params(), source)
    assert abs(float(source.get("l0.norm1").float().mean())) < 0.3                # stored around zero
    assert abs(float(source.get("l0.mix.left.out").float().mean()) - 1.0) < 0.3   # and around one
    source.close()
