"""The Zasudra configuration on the CPU: keys, the parts it names, tensor names and shapes, what each layer and the
embedding ask of the cache manager (pages, chunks, state, rows read from another layer), refusals, and the plain
implementation's own consistency."""

import copy
import math

import pytest
import torch

import plain_zasudra as plain
import zasudra_cases as Z


def test_the_specification_names_every_tensor_the_plain_implementation_reads():
    from llm_pipeline_b200.config import resolve_config
    from llm_pipeline_b200.models import build_model
    from llm_pipeline_b200.weights.source import shape_matches

    for name, cfg in Z.CONFIGS.items():
        config = resolve_config(cfg)
        model = build_model(config)
        expected = {n: tuple(s.shape) for n, s in model.expected_params().items() if not s.optional}
        W = Z.weights_for(cfg, 0)
        assert set(expected) == set(W), name
        assert all(shape_matches(tuple(t.shape), expected[n]) for n, t in W.items()), name
        # only the inner size of the decays' projection is left to the tensors
        assert {n.rsplit(".", 1)[1] for n, s in expected.items() if None in s} <= {"w1", "w2"}
        plain.forward(cfg, W, [1, 2, 3])                                         # and the oracle needs no other
        assert config.to_json()["layers"] == cfg["layers"] and config.to_json().get("embedding") == cfg.get("embedding")
        assert resolve_config(config.to_json()).model_spec() == config.model_spec()
        assert config.parameter_counts()["total_parameters"] > 0
        # a layer without experts may still find its second norm in a checkpoint, and does not read it
        spare = {n for n, s in model.expected_params().items() if s.optional}
        assert spare == {f"l{i}.norm2" for i, layer in enumerate(cfg["layers"]) if layer["mlp"] is None}


def test_what_the_layers_and_the_embedding_ask_of_the_cache_manager():
    from llm_pipeline_b200.cache import CacheManager
    from llm_pipeline_b200.cache.spec import HeadRowPagesSpec
    from llm_pipeline_b200.config import resolve_config
    from llm_pipeline_b200.models import build_model
    from llm_pipeline_b200.ops.kernels import wkv_state_entries

    cfg = Z.CONFIGS["mixed"]
    model = build_model(resolve_config(cfg))
    specs = model.cache_specs()
    assert len(specs) == 7                                                       # six layers and the embedding's last token
    assert specs[0] == (HeadRowPagesSpec(2, 32, chunk=24), None)                 # [k | v] rows, v the projected keys
    assert specs[1][0] is None and specs[1][1].dtype == torch.float32
    assert specs[1][1].shape == (2 * 64 + 2 * wkv_state_entries(3, 20),)
    assert wkv_state_entries(3, 20) >= 3 * 20 * 20
    assert specs[2] == (HeadRowPagesSpec(3, 40), None)
    assert specs[3] == (None, None)                                              # reads the third layer's rows
    assert [e.pages_from for e in model.spec.schedule] == [None, None, None, 2, None, None]
    assert specs[6][0] is None and specs[6][1].shape == (2,) and specs[6][1].dtype == torch.int32
    assert not any(n.startswith("l3.mix.k") or n.startswith("l3.mix.v") for n in model.expected_params())
    assert "l0.mix.v" not in model.expected_params() and "l2.mix.v" in model.expected_params()
    # a chunked group gives pages back when the next token begins a chunk; the causal group keeps all of its pages
    cache = CacheManager(specs, page_size=4, num_pages=64, max_requests=2, max_request_tokens=128)
    by_chunk = {group.spec.chunk: g for g, group in enumerate(cache.groups)}
    assert set(by_chunk) == {24, 10, None}
    cache.admit("a")
    assert cache.reserve("a", 47)
    cache.commit("a", 47)                                                        # the next token is 47, of the chunk from 24 on
    assert cache.block_table("a", by_chunk[24])[:6] == [-1] * 6 and min(cache.block_table("a", by_chunk[24])[6:]) >= 0
    assert cache.block_table("a", by_chunk[10])[:10] == [-1] * 10 and min(cache.block_table("a", by_chunk[10])[10:]) >= 0   # from 40 on
    assert cache.reserve("a", 48)
    cache.commit("a", 48)                                                        # token 48 begins a chunk of 24: all pages before it go
    assert cache.block_table("a", by_chunk[24]) == [-1] * 12
    assert min(cache.block_table("a", by_chunk[None])) >= 0
    cache.check()
    cache.free("a")
    cache.check()
    # a model without a bigram table carries nothing for its embedding
    assert len(build_model(resolve_config(Z.CONFIGS["wkv_only"])).cache_specs()) == 2


def test_the_first_key_a_token_sees():
    from llm_pipeline_b200.cache.spec import HeadRowPagesSpec
    chunk = HeadRowPagesSpec(1, 8, chunk=5)
    assert [chunk.first_key(p) for p in (0, 4, 5, 9, 10)] == [0, 0, 5, 5, 10] and chunk.bounded
    window = HeadRowPagesSpec(1, 8, window=3)
    assert [window.first_key(p) for p in (0, 2, 3, 9)] == [0, 0, 1, 7] and window.bounded
    assert HeadRowPagesSpec(1, 8).first_key(99) == 0 and not HeadRowPagesSpec(1, 8).bounded
    assert chunk.group_key() != HeadRowPagesSpec(1, 8).group_key() != window.group_key()


@pytest.mark.parametrize("damage, message", [
    (lambda c: c["layers"][0].update(type="lstm"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].pop("dim"), "lacks"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "lacks"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "cannot share"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=8), "vdim must equal dim"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=-2), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "rot.base"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_heads=6), "must equal"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown mlp kind"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "expert.ff"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "cannot use 6 of 5"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "bigram lacks"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c.pop("norm"), "required keys"),
    (lambda c: c.update(layers=[]), "required keys|no layers"),
])
def test_refusals(damage, message):
    from llm_pipeline_b200.config import resolve_config

    cfg = copy.deepcopy(Z.CONFIGS["mixed"])
    damage(cfg)
    with pytest.raises(ValueError, match=message):
        resolve_config(cfg)


def test_defaults_where_the_configuration_is_silent():
    from llm_pipeline_b200.config import resolve_config

    cfg = copy.deepcopy(Z.CONFIGS["mixed"])
    for key in ("residual_mult", "logit_scale", "embedding"):
        cfg.pop(key)
    cfg["layers"][0]["mixer"].pop("mask")
    cfg["layers"][0]["mixer"]["rot"].pop("dims")
    spec = resolve_config(cfg).model_spec()
    assert spec.embedding.kind == "token_embedding" and spec.final_norm.args["gain"] == 1.0
    assert all(norm.args["gain"] == 1.0 for layer in spec.layers for norm in layer.norms.values())
    assert spec.layers[0].mixer.args["chunk"] is None and spec.layers[0].mixer.args["rotary_dim"] == 16
    assert spec.layers[1].feed_forward.args["top"] == 3 and spec.layers[3].feed_forward is None


def test_the_plain_implementation_is_causal_and_its_mechanisms_have_their_closed_forms():
    cfg = Z.CONFIGS["mixed"]
    W = Z.weights_for(cfg, 1)
    tokens = [t % cfg["vocab"] for t in range(3, 70)]
    whole = plain.forward(cfg, W, tokens)
    assert (plain.forward(cfg, W, tokens[:17]) - whole[:17]).abs().max() < 1e-9
    assert plain.bigram_rows([4, 9, 4], 7, 3, 10) == [10, (4 * 7 + 9 * 3) % 10, (9 * 7 + 4 * 3) % 10]
    # a chunk: the token that begins one sees itself alone; the one before it sees the whole chunk before
    mask = plain.seen(9, 4)
    assert mask[4].nonzero().flatten().tolist() == [4] and mask[3].nonzero().flatten().tolist() == [0, 1, 2, 3]
    assert mask[8].nonzero().flatten().tolist() == [8] and plain.seen(9, None)[8].all()
    # with a zero score and a sink of zero, one key takes half; two keys take a third each
    q, k, v = torch.zeros(3, 2, 4, dtype=torch.float64), torch.zeros(3, 1, 4, dtype=torch.float64), torch.ones(3, 1, 5, dtype=torch.float64)
    out = plain.attend(q, k, v, 1.0, None, torch.zeros(2, dtype=torch.float64))
    assert torch.allclose(out[:, 0, 0], torch.tensor([1 / 2, 2 / 3, 3 / 4], dtype=torch.float64))
    # the rotation keeps lengths, leaves the entries past its size alone and turns pair (2, 3) by its frequency
    x = torch.randn(6, 2, 12, dtype=torch.float64)
    r = plain.rotate_interleaved(x, 8, 100.0)
    assert torch.equal(r[..., 8:], x[..., 8:]) and (r.norm(dim=-1) - x.norm(dim=-1)).abs().max() < 1e-12 and torch.equal(r[0], x[0])
    one = torch.zeros(8, 1, 8, dtype=torch.float64)
    one[7, 0, 2] = 1.0
    turned, a = plain.rotate_interleaved(one, 8, 100.0)[7, 0], 7 * 100.0 ** (-2.0 / 8)
    assert abs(float(turned[2]) - math.cos(a)) < 1e-12 and abs(float(turned[3]) - math.sin(a)) < 1e-12
    # the recurrence with decays of one and no bonus sums the earlier tokens; a state handed on gives the same rows
    rr, kk, vv, ww = (torch.rand(7, 2, 3, dtype=torch.float64) for _ in range(4))
    o, _ = plain.wkv_scan(rr, kk, vv, torch.ones_like(ww), torch.zeros(2, 3, dtype=torch.float64))
    for t in range(7):
        want = sum((torch.einsum("hc,hc->h", rr[t], kk[s])[:, None] * vv[s] for s in range(t)), torch.zeros(2, 3, dtype=torch.float64))
        assert torch.allclose(o[t], want)
    u = torch.rand(2, 3, dtype=torch.float64)
    full, _ = plain.wkv_scan(rr, kk, vv, ww, u)
    head, S = plain.wkv_scan(rr[:4], kk[:4], vv[:4], ww[:4], u)
    tail, _ = plain.wkv_scan(rr[4:], kk[4:], vv[4:], ww[4:], u, S)
    assert torch.allclose(torch.cat([head, tail]), full)
    # the router: the largest logits in order, their softmax alone
    chosen, weights = plain.route(torch.tensor([[1.0, 0.0]], dtype=torch.float64), torch.tensor([[1.0, 5.0], [3.0, 0.0], [2.0, 0.0]], dtype=torch.float64),
                                  torch.tensor([0.5, 0.0, 2.0], dtype=torch.float64), 2)
    assert chosen.tolist() == [[2, 1]] and torch.allclose(weights[0], torch.softmax(torch.tensor([4.0, 3.0], dtype=torch.float64), 0))


def test_a_random_model_folder_can_be_written_and_read_back(tmp_path):
    from llm_pipeline_b200.config import load_config
    from llm_pipeline_b200.models import build_model
    from llm_pipeline_b200.weights import write_random_model
    from llm_pipeline_b200.weights.source import SafetensorsSource, check_names_and_shapes

    folder = write_random_model(Z.CONFIGS["mixed"], 3, str(tmp_path))
    config = load_config(folder)
    assert config.architecture == "Zasudra"
    source = SafetensorsSource(folder)
    check_names_and_shapes(build_model(config).expected_params(), source)
    assert abs(float(source.get("l0.norm1").float().mean()) - 1.0) < 0.3          # around one, not noise around zero
    assert source.shape("bigram") == (54, 64) and "l3.mix.k" not in source.names()
    source.close()
