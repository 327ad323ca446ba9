"""CPU: host-side parts of the Palulorn path — the plain restatement against itself (whole prompt, token by token,
portions) and its mechanisms by hand, the product's shape, run and frequency tables against the tests' own, the registry
and a model folder's reader."""
import json
import math

import numpy as np
import pytest
import torch

from oracle import palulorn as op
from tests import palulorn_case as pc

F64 = torch.float64


def toks(n, vocab, seed):
    return [int(x) for x in np.random.default_rng(seed).integers(0, vocab, size=n)]


@pytest.mark.parametrize("name", sorted(pc.CONFIGS))
def test_oracle_whole_equals_token_by_token_and_portions(name):
    cfg = pc.CONFIGS[name]
    m = op.Palulorn(cfg, pc.weights(cfg, 1))
    tokens = toks(34, cfg["vocab"], 3)
    whole = m.forward(tokens, m.new_state())
    for cuts in ([1] * 34, [7, 2, 1, 15, 9], [2] * 17):
        st, rows, at = m.new_state(), [], 0
        for n in cuts:
            rows.append(m.forward(tokens[at:at + n], st))
            at += n
        assert float((torch.cat(rows) - whole).abs().max()) < 1e-9


def test_filter_by_hand():
    x, st = torch.arange(1.0, 6.0, dtype=F64)[:, None], {}
    c = torch.tensor([[100.0, 10.0, 1.0]], dtype=F64)                    # the last column is the current row's
    y = torch.cat([op.short_filter(x[:2], c, st, "k"), op.short_filter(x[2:3], c, st, "k"), op.short_filter(x[3:], c, st, "k")])
    assert y[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0] and st["k"][:, 0].tolist() == [4.0, 5.0]


def test_window_sink_and_temperature_by_hand():
    K = torch.zeros(4, 1, 2, dtype=F64)
    V = torch.tensor([1.0, 2.0, 4.0, 8.0], dtype=F64)[:, None, None]
    q = torch.ones(4, 2, 2, dtype=F64)
    pos = torch.arange(4)
    o = op.attend(q, K, V, pos, 1.0, window=2)                           # the row itself and the one before it
    assert torch.allclose(o[:, 0, 0], torch.tensor([1.0, 1.5, 3.0, 6.0], dtype=F64))
    o = op.attend(q, K, V, pos, 1.0, sink=torch.tensor([0.0, math.log(3.0)], dtype=F64))
    assert torch.allclose(o[:, 0, 0], torch.tensor([1 / 2, 3 / 3, 7 / 4, 15 / 5], dtype=F64))
    assert torch.allclose(o[:, 1, 0], torch.tensor([1 / 4, 3 / 5, 7 / 6, 15 / 7], dtype=F64))
    # the step comes at the token that completes a stretch: position every - 1
    t = op.temperature(torch.tensor([0, 3, 4, 8, 9]), 0.5, 5)
    assert torch.allclose(t, torch.tensor([1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)], dtype=F64))


def test_turn_by_hand():
    x = torch.randn(5, 2, 6, dtype=F64)
    r = op.turn(x, torch.arange(5), 100.0, 4, 2.0)
    for a in range(2):
        assert torch.allclose(r[..., a] ** 2 + r[..., a + 2] ** 2, x[..., a] ** 2 + x[..., a + 2] ** 2)
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.allclose(r[0], x[0])
    u = op.turn(torch.tensor([[[1.0, 0.0]]], dtype=F64), torch.tensor([6]), 7.0, 2, 2.0)
    assert torch.allclose(u[0, 0], torch.tensor([math.cos(3.0), math.sin(3.0)], dtype=F64))


def test_matrix_memory_by_hand():
    one = lambda *v: torch.tensor(v, dtype=F64)
    S, n, m = torch.zeros(1, 1, 1, dtype=F64), torch.zeros(1, 1, dtype=F64), torch.zeros(1, dtype=F64)
    k = v = torch.ones(2, 1, 1, dtype=F64)
    # i below the running maximum 0: written small, and the denominator is exp(-m) = 1
    o = op.matrix_memory(one(2.0)[None, :, None], k[:1], v[:1] * 3, one(-1.0)[None], one(-0.5)[None], S, n, m)
    # m' = max(-0.5 + 0, -1) = -0.5: n = exp(-0.5), the denominator max(2 n, exp(0.5))
    assert abs(float(m) + 0.5) < 1e-12 and abs(float(n) - math.exp(-0.5)) < 1e-12
    assert abs(float(o) - 6 * math.exp(-0.5) / (max(2 * math.exp(-0.5), math.exp(0.5)) + 1e-6)) < 1e-9
    # a loud gate takes the memory over: the read-out is the new value
    o = op.matrix_memory(one(2.0)[None, :, None], k[:1], v[:1] * 7, one(30.0)[None], one(-0.5)[None], S, n, m)
    assert abs(float(o) - 7.0) < 1e-4 and float(m) == 30.0


def test_gated_scan_and_block_map_by_hand():
    S = torch.zeros(1, dtype=F64)
    lam = torch.tensor([math.log(math.expm1(math.log(2.0) / 8.0))], dtype=F64)       # a = 1/2 at r = 1
    o = op.gated_scan(torch.ones(2, 1, dtype=F64), torch.ones(2, 1, dtype=F64), torch.ones(2, 1, dtype=F64), lam, S)
    w = math.sqrt(0.75)
    assert torch.allclose(o[:, 0], torch.tensor([w, 1.5 * w], dtype=F64))            # the first token gets no special weight
    M = torch.tensor([[[1.0, 2.0], [0.0, 1.0]], [[3.0, 0.0], [0.0, 0.0]]], dtype=F64)
    y = op.block_map(torch.tensor([[1.0, 10.0, 100.0, 1000.0]], dtype=F64), M, torch.tensor([[0.0, 1.0], [0.0, 5.0]], dtype=F64))
    assert y.tolist() == [[21.0, 11.0, 300.0, 5.0]]


def test_route_by_hand():
    logit = lambda *p: torch.log(torch.tensor([p], dtype=F64) / (1 - torch.tensor([p], dtype=F64)))
    # the first group holds the largest score, the second the larger sum of two
    z = logit(0.9, 0.1, 0.05, 0.7, 0.6, 0.2)
    ids, w = op.route(z, 2, 2, 1, 3.0)
    assert sorted(ids[0].tolist()) == [3, 4] and torch.allclose(w.sum(), torch.tensor(3.0, dtype=F64))
    assert torch.allclose(w.max(), torch.tensor(3.0 * 0.7 / 1.3, dtype=F64))
    ids, _ = op.route(z, 2, 1, 1, 1.0)
    assert sorted(ids[0].tolist()) == [0, 3]


def test_runs_of_a_looped_model():
    from scalellm_b200 import palulorn
    assert palulorn.layer_runs(pc.CONFIGS["mix"]) == [(0, -1), (1, 0), (2, -1), (1, 1), (2, -1), (1, 2), (2, -1), (3, -1)]
    assert palulorn.layer_runs(pc.CONFIGS["odd"]) == [(i, -1) for i in range(5)]
    assert palulorn.layer_runs(pc.CONFIGS["loop"]) == [(0, 0), (1, -1), (0, 1), (1, -1)]
    for name, cfg in pc.CONFIGS.items():
        assert [(i, t if s else -1) for i, t, s in op.layer_runs(cfg)] == palulorn.layer_runs(cfg), name
    for bad in ((0, 5, 1), (2, 2, 1), (0, 1, 0)):
        with pytest.raises(ValueError):
            palulorn.layer_runs(dict(pc.CONFIGS["mix"], loop=dict(zip(("start", "stop", "times"), bad))))


def test_product_shape_and_frequency_tables():
    from scalellm_b200 import palulorn
    for name, cfg in pc.CONFIGS.items():
        assert palulorn.tensor_shapes(cfg) == pc.shapes(cfg), name
        made = palulorn.random_tensors(cfg, 1)
        assert {k: tuple(v.shape) for k, v in made.items()} == pc.shapes(cfg), name
    f, dims = palulorn.rotary_table({"base": 500.0, "dims": 6, "scaling": {"factor": 4.0}})
    want = torch.tensor([1.0, 500.0 ** (-1 / 3), 500.0 ** (-2 / 3)], dtype=F64) / 4.0
    assert dims == 6 and f.dtype == torch.float32 and torch.allclose(f.double(), want)
    assert palulorn.rotary_table(None) == (None, 0) and palulorn.rotary_table({"base": 10.0, "dims": 0}) == (None, 0)
    layer = pc.CONFIGS["mix"]["layers"][1]
    uneven = dict(layer, mixer=dict(layer["mixer"], left=dict(layer["mixer"]["left"], vdim=8)))
    for bad in ({"type": "other", "mixer": {}, "mlp": None}, dict(layer, mlp={"kind": "dense", "ff": 8}), uneven,
                dict(pc.rglru(10, 3), mlp=None)):
        with pytest.raises(ValueError):
            palulorn.tensor_shapes(dict(pc.CONFIGS["mix"], layers=[bad]))


def test_padded_input_rows():
    from scalellm_b200.layers import input_rows_multiple, stack_rows
    a, b = torch.ones(3, 4), torch.full((2, 4), 2.0)
    s = stack_rows([a, b], 8)
    assert s.shape == (8, 4) and torch.equal(s[:5], torch.cat([a, b])) and float(s[5:].abs().max()) == 0.0
    assert stack_rows([a, b]).shape == (5, 4)
    assert input_rows_multiple(100) == 8 and input_rows_multiple(4000) == 128


def test_registry_and_model_folder(tmp_path):
    from scalellm_b200 import checkpoint, palulorn, registry
    cfg = pc.CONFIGS["odd"]
    assert registry.model_class(cfg) is palulorn.PalulornDecoder
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    w = pc.weights(cfg, 2)
    checkpoint.write_safetensors(str(tmp_path / "model.safetensors"), w)
    back = checkpoint.read_safetensors(str(tmp_path / "model.safetensors"))
    assert checkpoint.read_config(str(tmp_path)) == cfg and set(back) == set(w)
    assert all(torch.equal(back[k], w[k]) for k in w)
    assert all(torch.equal(v, op.read_safetensors(str(tmp_path / "model.safetensors"))[k]) for k, v in back.items())
