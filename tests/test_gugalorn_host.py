"""CPU: host-side parts of the Gugalorn path — the plain restatement against itself (whole prompt, token by token,
portions) and its mechanisms by hand, the product's shape and frequency tables against the tests' own, the registry and a
model folder's reader."""
import json
import math

import numpy as np
import pytest
import torch

from oracle import gugalorn as og
from tests import gugalorn_case as gc


def toks(n, vocab, seed):
    return [int(x) for x in np.random.default_rng(seed).integers(0, vocab, size=n)]


@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
def test_oracle_whole_equals_token_by_token_and_portions(name):
    cfg = gc.CONFIGS[name]
    m = og.Gugalorn(cfg, gc.weights(cfg, 1))
    tokens = toks(34, cfg["vocab"], 3)
    whole = m.forward(tokens, m.new_state())
    for cuts in ([1] * 34, [7, 2, 1, 15, 9], [2] * 17):
        st, rows, at = m.new_state(), [], 0
        for n in cuts:
            rows.append(m.forward(tokens[at:at + n], st))
            at += n
        assert float((torch.cat(rows) - whole).abs().max()) < 1e-9


def test_filter_by_hand():
    st = {}
    x = torch.arange(1.0, 6.0, dtype=torch.float64)[:, None]
    c = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64)          # the last column is the current row's
    y = torch.cat([og.filter_causal(x[:2], c, st, "k"), og.filter_causal(x[2:3], c, st, "k"),
                   og.filter_causal(x[3:], c, st, "k")])
    assert y[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]
    assert st["k"][:, 0].tolist() == [4.0, 5.0]
    one = {}
    assert og.filter_causal(x, torch.tensor([[3.0]], dtype=torch.float64), one, "k")[:, 0].tolist() == [3.0, 6.0, 9.0, 12.0, 15.0]
    assert one["k"].shape == (0, 1)


def test_attention_with_one_in_the_denominator_by_hand():
    K = torch.zeros(3, 1, 2, dtype=torch.float64)
    V = torch.tensor([[[1.0]], [[2.0]], [[4.0]]], dtype=torch.float64)
    q = torch.ones(3, 2, 2, dtype=torch.float64)
    o = og.attend_with_one(q, K, V, torch.arange(3), 1.0)                # scores 0: a key weighs 1 / (n + 1)
    assert torch.allclose(o[:, 0, 0], torch.tensor([1 / 2, 3 / 3, 7 / 4], dtype=torch.float64))
    assert torch.equal(o[:, 0], o[:, 1])                                 # two query heads on one key/value head
    low = og.attend_with_one(q, K - 300.0, V, torch.arange(3), 1.0)      # no key matters: the sink takes everything
    assert float(low.abs().max()) < 1e-100
    high = og.attend_with_one(q, K + 300.0, V, torch.arange(3), 1.0)     # the sink does not matter: a plain average
    assert torch.allclose(high[:, 0, 0], torch.tensor([1.0, 1.5, 7 / 3], dtype=torch.float64))


def test_turn_and_projection_norm_by_hand():
    x = torch.randn(5, 2, 6, dtype=torch.float64)
    r = og.turn(x, torch.arange(5), 100.0, 4)
    for a in range(2):
        assert torch.allclose(r[..., a] ** 2 + r[..., a + 2] ** 2, x[..., a] ** 2 + x[..., a + 2] ** 2)
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.allclose(r[0], x[0])
    u = og.turn(torch.tensor([[[1.0, 0.0]]], dtype=torch.float64), torch.tensor([3]), 7.0, 2)
    assert torch.allclose(u[0, 0], torch.tensor([math.cos(3.0), math.sin(3.0)], dtype=torch.float64))
    # one root mean square for all heads: a head of small numbers stays small
    y = og.norm(torch.tensor([[3.0, 4.0, 0.0, 0.0]], dtype=torch.float64), torch.ones(4, dtype=torch.float64), 0.0)
    assert torch.allclose(y, torch.tensor([[1.2, 1.6, 0.0, 0.0]], dtype=torch.float64))


def test_recurrences_by_hand():
    # forget gate: what is forgotten is written; f = 1 keeps everything, f = 0 replaces everything
    S = torch.zeros(1, 2, 1, dtype=torch.float64)
    f = torch.tensor([[[0.0, 0.5]], [[1.0, 0.5]], [[0.0, 1.0]]], dtype=torch.float64)
    v = torch.tensor([[[8.0]], [[4.0]], [[2.0]]], dtype=torch.float64)
    o = og.forget_write_scan(torch.ones_like(f), f, v, S)
    assert S[0, :, 0].tolist() == [2.0, 4.0] and o[:, 0, 0].tolist() == [12.0, 12.0, 6.0]
    # state space: decay exp(-exp(A) dt), write dt B x^T, D x past the state; head h reads group h // (H / G)
    S = torch.zeros(2, 1, 1, dtype=torch.float64)
    x = torch.ones(2, 2, 1, dtype=torch.float64)
    B = torch.tensor([[[1.0], [10.0]]] * 2, dtype=torch.float64)
    dt = torch.tensor([[1.0, 2.0]] * 2, dtype=torch.float64)
    A = torch.log(torch.tensor([math.log(2.0), math.log(2.0)], dtype=torch.float64))
    y = og.ssd_scan(x, B, torch.ones(2, 2, 1, dtype=torch.float64), dt, A, torch.tensor([0.0, 5.0], dtype=torch.float64), S)
    assert torch.allclose(y[:, 0, 0], torch.tensor([1.0, 1.5], dtype=torch.float64))
    assert torch.allclose(y[:, 1, 0], torch.tensor([25.0, 30.0], dtype=torch.float64))
    # gated first, normalised after, part by part
    u = og.gated_part_norm(torch.tensor([[1.0, 1.0, 100.0, 100.0]], dtype=torch.float64),
                           torch.tensor([[5.0, 5.0, 1.0, 1.0]], dtype=torch.float64), torch.ones(4, dtype=torch.float64), 2, 0.0)
    assert torch.allclose(u, torch.ones(1, 4, dtype=torch.float64))


def test_product_shape_and_frequency_tables():
    from scalellm_b200 import gugalorn
    for name, cfg in gc.CONFIGS.items():
        assert gugalorn.tensor_shapes(cfg) == gc.shapes(cfg), name
        made = gugalorn.random_tensors(cfg, 1)
        assert {k: tuple(v.shape) for k, v in made.items()} == gc.shapes(cfg), name
    f = gugalorn.rotary_frequencies(500.0, 6)
    assert f.dtype == torch.float32 and torch.allclose(f.double(), torch.tensor([1.0, 500.0 ** (-1 / 3), 500.0 ** (-2 / 3)], dtype=torch.float64))
    for bad in ({"type": "other", "mixer": {}, "mlp": None}, dict(gc.CONFIGS["mix"]["layers"][0], mlp={"kind": "moe"})):
        with pytest.raises(ValueError):
            gugalorn.tensor_shapes(dict(gc.CONFIGS["mix"], layers=[bad]))


def test_registry_and_model_folder(tmp_path):
    from scalellm_b200 import checkpoint, gugalorn, registry
    cfg = gc.CONFIGS["odd"]
    assert registry.model_class(cfg) is gugalorn.GugalornDecoder
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    w = gc.weights(cfg, 2)
    checkpoint.write_safetensors(str(tmp_path / "model.safetensors"), w)
    back = checkpoint.read_safetensors(str(tmp_path / "model.safetensors"))
    assert checkpoint.read_config(str(tmp_path)) == cfg and set(back) == set(w)
    assert all(torch.equal(back[k], w[k]) for k in w)
    assert all(torch.equal(v, og.read_safetensors(str(tmp_path / "model.safetensors"))[k]) for k, v in back.items())
