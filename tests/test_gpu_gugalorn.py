"""GPU: the Gugalorn decoder through the serving engine against the plain CPU restatement (oracle/gugalorn.py, float64):
every mechanism alone, whole prompts, token-by-token decoding, portions, mixed batches, reuse of blocks and state slots,
keys far away and at cache-block borders, the sink, the first tokens, filter and matrix states carried over steps,
generation through the scheduler."""
import json

import numpy as np
import pytest
import torch

from oracle import gugalorn as og
from tests import gugalorn_case as gc

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0) if torch.cuda.is_available() else None
TOL = {torch.float32: 1e-4, torch.bfloat16: 6e-2}
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5


def build(cfg, dtype, seed=0, max_seqs=4):
    from scalellm_b200 import registry
    w = gc.weights(cfg, seed)
    model = registry.create_model(cfg, dtype, DEV, max_seqs=max_seqs)
    model.load_weights({k: v.to(DEV) for k, v in w.items()})
    return model, og.Gugalorn(cfg, w)


def engine_for(model, max_tokens=512, block_size=4, max_seqs=4, use_graphs=False):
    from scalellm_b200.engine import Engine
    return Engine(model, max_tokens, block_size=block_size, max_seqs=max_seqs, use_graphs=use_graphs)


def oracle_logits(oracle, tokens):
    return oracle.forward(tokens, oracle.new_state())


def run_schedule(eng, tokens, cuts, rid="r"):
    """Feed `tokens` in portions of the given sizes (the rest one by one); logits of every position."""
    from scalellm_b200.engine import StepEntry
    out, at = [], 0
    sizes = list(cuts)
    while at < len(tokens):
        n = min(sizes.pop(0) if sizes else 1, len(tokens) - at)
        out.append(eng.step([StepEntry(rid, tokens[at:at + n], list(range(n)))]).float().cpu())
        at += n
    eng.finish(rid)
    return torch.cat(out, 0)


def toks(n, vocab, seed):
    return [int(x) for x in np.random.default_rng(seed).integers(0, vocab, size=n)]


def _params(n_tokens_per_seq, cached, block_size=4, n_blocks=256, pool_seed=3, slots=None):
    from scalellm_b200.decode_step import BlockPool, StepBuffers, build_step_batch
    pool = BlockPool(n_blocks, block_size, seed=pool_seed)
    seqs = []
    for n, c in zip(n_tokens_per_seq, cached):
        s = pool.open_sequence()
        pool.reserve(s, n + c)
        seqs.append(s)
    hb = build_step_batch(pool, seqs, [[0] * n for n in n_tokens_per_seq], list(cached), slots)
    bufs = StepBuffers(DEV, sum(n_tokens_per_seq) + 8, len(seqs) + 1, n_blocks + 8)
    return bufs.upload(hb), hb


def _slots(hb, seq_index, n, block_size):
    lo = int(hb.cu_block_lens[seq_index])
    return [int(hb.block_tables[lo + j // block_size]) + j % block_size for j in range(n)]


def assert_rows(e, dtype, what=""):
    """float32: every row within the tolerance.  bfloat16: where a small part of a row has a root mean square near zero
    its norm magnifies the rounding of the projections before it, so now and then a token is off by more (the plain
    restatement with its norms' results rounded to 16 bits has such rows too): there the typical row is held to the
    tolerance and at most a twentieth may exceed it.  Faults of logic show in float32, which runs the same schedules."""
    if dtype == torch.float32:
        assert float(e.max()) < TOL[dtype], f"{what}: {float(e.max())}"
        return
    over = int((e > TOL[dtype]).sum())
    assert float(e.median()) < TOL[dtype] / 3 and over <= max(2, e.numel() // 20), \
        f"{what}: median {float(e.median())}, {over} of {e.numel()} rows over"


def assert_logits(got, want, dtype, what=""):
    assert_rows(gc.row_errors(got, want), dtype, what)


def close(got, want, dtype, what="", tol=None):
    tol = tol or (2e-5 if dtype == torch.float32 else 2e-2)
    err = float((got.double().cpu() - want.double()).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), f"{what}: {err}"


# Two sequences in two of three state slots, fed in portions of 1, 2, fewer and more tokens than a filter has taps, and
# more than a chunk of rows; the slots hold stale numbers of an old owner.
PLANS = {0: [1, 2, 1, 7, 3, 40, 1, 1, 12], 1: [21, 1, 1, 2, 2, 5, 37, 1, 7]}
SLOT_OF = {0: 2, 1: 0}


def over_portions(data, run):
    """data[s]: a tuple of [tokens, ...] tensors; run(step, rows, positions, params) -> [rows, n] for the two sequences'
    rows of one step.  Returns the concatenated results per sequence."""
    at, got = {0: 0, 1: 0}, {0: [], 1: []}
    for step in range(len(PLANS[0])):
        ns = [PLANS[s][step] for s in (0, 1)]
        (tok, pos, par), _ = _params(ns, [at[0], at[1]], slots=[SLOT_OF[0], SLOT_OF[1]])
        rows = [torch.cat([data[s][i][at[s]:at[s] + ns[s]] for s in (0, 1)]).to(DEV) for i in range(len(data[0]))]
        o = run(step, rows, pos, par)
        got[0].append(o[:ns[0]].cpu())
        got[1].append(o[ns[0]:].cpu())
        at[0] += ns[0]
        at[1] += ns[1]
    return {s: torch.cat(got[s]) for s in got}


def total(s):
    return sum(PLANS[s])


# ------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("W", [1, 42, 200, 1030])
@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_sum_and_norm(W, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(W)
    x, y = torch.randn(5, W, generator=g) * 3.0, torch.randn(5, W, generator=g).to(dtype)
    w = 0.5 + torch.rand(W, generator=g)
    wide = torch.cat([y, y], dim=1).to(DEV)
    xd = x.to(DEV)
    out, h = kernels.prenorm(xd, wide[:, W:], w.to(DEV), EPS, dtype)      # a strided column block
    want = x.double() + y.double()
    close(out, want, torch.float32)
    close(h, og.norm(want, w.double(), EPS), dtype)
    assert torch.equal(xd.cpu(), x) and h.dtype == dtype
    same, h = kernels.prenorm(xd, None, w.to(DEV), EPS, dtype)
    assert same is xd
    close(h, og.norm(x.double(), w.double(), EPS), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,taps", [(40, 4), (64, 1), (33, 3), (1030, 2), (24, 7)])
def test_norm_and_input_filter_over_portions(W, taps, dtype):
    """The sum, its norm and the filter with its state: a lost or stale row of the state shows at the start of a portion."""
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(W + taps)
    filt, w = torch.randn(W, taps, generator=g), 0.5 + torch.rand(W, generator=g)
    data = {s: (torch.randn(total(s), W, generator=g) * 2.0, torch.randn(total(s), W, generator=g).to(dtype)) for s in PLANS}
    state = torch.full((3, taps - 1, W), 5.0, device=DEV)
    fd, wd = filt.t().contiguous().to(DEV), w.to(DEV)

    def run(step, rows, pos, par):
        y = rows[1] if step % 3 else None
        x = rows[0] if y is not None else rows[0] + rows[1].float()
        out, h = kernels.prenorm(x, y, wd, EPS, dtype, fd, state, par.q_cu_seq_lens, pos, par.state_slots,
                                 par.num_sequences, par.q_max_seq_len)
        assert torch.equal(out.cpu(), (rows[0] + rows[1].float()).cpu())
        return h
    got = over_portions(data, run)
    for s in PLANS:
        n = og.norm(data[s][0].double() + data[s][1].double(), w.double(), EPS)
        close(got[s], n + og.filter_causal(n, filt.double(), {}, "k"), dtype, s)
    assert bool((state[1] == 5.0).all())


@pytest.mark.parametrize("rows", [1, 7, 70])
def test_norm_and_filter_take_split_k_partials(rows):
    """The same launch fed by a product's partials equals the product followed by the launch."""
    from scalellm_b200 import kernels
    from scalellm_b200.layers import Linear
    g = torch.Generator().manual_seed(rows)
    W, K, taps = 256, 384, 4
    lin = Linear((torch.randn(W, K, generator=g) / 20).to(torch.bfloat16).to(DEV))
    a = torch.randn(rows, K, generator=g).to(torch.bfloat16).to(DEV)
    x, w = torch.randn(rows, W, generator=g).to(DEV), (0.5 + torch.rand(W, generator=g)).to(DEV)
    filt = torch.randn(taps, W, generator=g).to(DEV)
    assert lin.supports_partials(rows)
    (tok, pos, par), _ = _params([rows], [9], slots=[0])
    for f in (None, filt):
        res = []
        for y in (lin(a), lin.forward_partials(a)):
            st = torch.ones(1, taps - 1, W, device=DEV)
            args = () if f is None else (f, st, par.q_cu_seq_lens, pos, par.state_slots, 1, rows)
            res.append(kernels.prenorm(x, y, w, EPS, torch.bfloat16, *args) + (st,))
        close(res[1][0], res[0][0].cpu(), torch.float32, tol=1e-6)
        close(res[1][1], res[0][1].cpu(), torch.bfloat16)
        close(res[1][2], res[0][2].cpu(), torch.float32, tol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ch,taps,bias", [(40, 4, True), (37, 3, True), (512, 2, False), (20, 1, True), (24, 9, True), (700, 6, False)])
def test_short_filter_with_silu_over_portions(ch, taps, bias, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(ch + taps)
    filt = torch.randn(ch, taps, generator=g)
    b = torch.randn(ch, generator=g) if bias else None
    data = {s: (torch.randn(total(s), ch + 4, generator=g).to(dtype),) for s in PLANS}
    state = torch.full((3, taps - 1, ch), 5.0, device=DEV)
    fd, bd = filt.t().contiguous().to(DEV), None if b is None else b.to(DEV)
    for silu in (True, False):
        got = over_portions(data, lambda step, rows, pos, par: kernels.causal_filter(
            rows[0][:, 4:], fd, bd, state, par.q_cu_seq_lens, pos, par.state_slots, 2, par.q_max_seq_len, silu))
        for s in PLANS:
            y = og.filter_causal(data[s][0][:, 4:].double(), filt.double(), {}, "k") + (b.double() if bias else 0.0)
            close(got[s], og.silu(y) if silu else y, dtype, s)
    assert taps == 1 or bool((state[1] == 5.0).all())


FORGET = [(3, 20, 12), (1, 9, 15), (2, 64, 64), (2, 128, 128), (1, 150, 136), (4, 16, 7), (1, 33, 300), (1, 300, 40)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,N,V", FORGET)
@pytest.mark.parametrize("form", ["", "simt"])
def test_forget_gate_recurrence_over_portions(H, N, V, dtype, form, monkeypatch):
    """Gates from nearly all forgotten to nearly all kept, lower bounds at 0 and near 1; scaled into a column block."""
    from scalellm_b200 import kernels
    monkeypatch.setenv("B200_SCAN_IMPL", form)                   # portions on the tensor cores where they fit, or never
    g = torch.Generator().manual_seed(H * N + V)
    fb, low = torch.randn(H * N, generator=g) * 3.0, torch.rand(H * N, generator=g) ** 0.3
    low[::5] = 0.0
    fb[::35] = -60.0                                             # with a lower bound of 0: nothing is kept at all
    nw = 0.5 + torch.rand(V, generator=g)
    n, nv = H * N, H * V
    data = {s: (torch.randn(total(s), 2 * n + nv, generator=g).mul(2.0).to(dtype),) for s in PLANS}
    state = torch.full((3, H, N, V), 5.0, device=DEV)
    d = [t.to(DEV) for t in (fb, low, nw)]

    def run(step, rows, pos, par):
        p = rows[0]
        out = torch.zeros(p.shape[0], nv + 8, dtype=dtype, device=DEV)
        kernels.forget_scan(p[:, :n], p[:, n:2 * n], p[:, 2 * n:], *d, state, par.q_cu_seq_lens, pos, par.state_slots, 2,
                            par.q_max_seq_len, EPS, 0.7, out[:, 8:])
        assert float(out[:, :8].abs().max()) == 0.0
        return out[:, 8:]
    got = over_portions(data, run)
    for s in PLANS:
        p = data[s][0].double()
        T = p.shape[0]
        f = low.double() + (1.0 - low.double()) * torch.sigmoid(p[:, n:2 * n] + fb.double())
        S = torch.zeros(H, N, V, dtype=torch.float64)
        o = og.forget_write_scan(og.silu(p[:, :n]).reshape(T, H, N), f.reshape(T, H, N), p[:, 2 * n:].reshape(T, H, V), S)
        close(got[s], 0.7 * og.norm(o, nw.double(), EPS).reshape(T, nv), dtype, s, tol=1e-4 if dtype == torch.float32 else 2e-2)
        close(state[SLOT_OF[s]], S, torch.float32, f"state {s}", tol=1e-5)
    assert bool((state[1] == 5.0).all())


SSD = [(6, 3, 24, 10), (1, 1, 18, 13), (4, 2, 64, 32), (2, 1, 128, 64), (2, 2, 130, 140), (4, 4, 16, 64), (8, 2, 128, 64), (2, 1, 32, 300)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,V", SSD)
@pytest.mark.parametrize("form", ["", "simt"])
def test_state_space_recurrence_over_portions(H, G, N, V, dtype, form, monkeypatch):
    from scalellm_b200 import kernels
    monkeypatch.setenv("B200_SCAN_IMPL", form)
    g = torch.Generator().manual_seed(H * N + V)
    ch = H * V + 2 * G * N
    a_log, dtb, D = torch.log(0.05 + 8.0 * torch.rand(H, generator=g)), -4.0 + 5.0 * torch.rand(H, generator=g), torch.randn(H, generator=g)
    data = {s: (torch.randn(total(s), ch, generator=g).to(dtype), torch.randn(total(s), H + 3, generator=g).mul(2.0).to(dtype))
            for s in PLANS}
    state = torch.full((3, H, N, V), 5.0, device=DEV)
    d = [t.to(DEV) for t in (dtb, a_log, D)]
    got = over_portions(data, lambda step, rows, pos, par: kernels.ssd_scan(
        rows[0][:, :H * V], rows[0][:, H * V:H * V + G * N], rows[0][:, H * V + G * N:], rows[1][:, 3:], *d, state,
        par.q_cu_seq_lens, pos, par.state_slots, 2, par.q_max_seq_len, G))
    for s in PLANS:
        p, T = data[s][0].double(), total(s)
        dt = torch.nn.functional.softplus(data[s][1][:, 3:].double() + dtb.double())
        S = torch.zeros(H, N, V, dtype=torch.float64)
        y = og.ssd_scan(p[:, :H * V].reshape(T, H, V), p[:, H * V:H * V + G * N].reshape(T, G, N),
                        p[:, H * V + G * N:].reshape(T, G, N), dt, a_log.double(), D.double(), S)
        # the walk is fp32 whatever the inputs' type is
        close(got[s], y.reshape(T, H * V), torch.float32, s, tol=5e-5)
        close(state[SLOT_OF[s]], S, torch.float32, f"state {s}", tol=5e-5)
    assert bool((state[1] == 5.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,parts", [(60, 4), (15, 3), (13, 13), (256, 1), (1024, 8), (1000, 20), (6, 1)])
def test_gate_then_norm_in_parts(n, parts, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(n + parts)
    y, w = torch.randn(5, n, generator=g) * 3.0, 0.5 + torch.rand(n, generator=g)
    y[:, : n // parts] *= 50.0                                   # a loud part must not quiet the others
    z = torch.randn(5, n + 4, generator=g).to(dtype)
    got = kernels.gated_part_norm(y.to(DEV), z.to(DEV)[:, 4:], w.to(DEV), parts, EPS)
    close(got, og.gated_part_norm(y.double(), z[:, 4:].double(), w.double(), parts, EPS), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,rot", [(4, 2, 16, 24, 8), (3, 3, 10, 7, 2), (6, 2, 12, 20, 12), (2, 1, 64, 130, 4), (5, 1, 6, 5, 6)])
def test_attention_inputs_norm_turn_and_cache_rows(H, G, dim, vdim, rot, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(H * dim)
    bs = 4
    (tok, pos, par), hb = _params([5, 1], [3, 9], block_size=bs)
    rows, nq, nk = 6, H * dim, G * dim
    proj = torch.randn(rows, nq + nk + G * vdim, generator=g)
    proj[:, :dim] *= 10.0                                        # one loud head: the others share its root mean square
    proj = proj.to(dtype)
    qw, kw = 0.5 + torch.rand(nq, generator=g), 0.5 + torch.rand(nk, generator=g)
    f = torch.tensor([100.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
    kc = torch.full((256 * bs, G, dim), 7.0, dtype=dtype, device=DEV)
    vc = torch.full((256 * bs, G, vdim), 7.0, dtype=dtype, device=DEV)
    pd = proj.to(DEV)
    q = kernels.sink_attn_prepare_turned(pd[:, :nq], pd[:, nq:nq + nk], pd[:, nq + nk:], qw.to(DEV), kw.to(DEV), f.to(DEV),
                                         kc, vc, pos, par.new_cache_slots, H, G, dim, vdim, rot, EPS)
    p64, positions = proj.double(), torch.tensor([3, 4, 5, 6, 7, 9])
    close(q, og.turn(og.norm(p64[:, :nq], qw.double(), EPS).reshape(rows, H, dim), positions, 100.0, rot), torch.float32, "queries")
    written = _slots(hb, 0, 8, bs)[3:] + [_slots(hb, 1, 10, bs)[9]]
    close(kc[written], og.turn(og.norm(p64[:, nq:nq + nk], kw.double(), EPS).reshape(rows, G, dim), positions, 100.0, rot), dtype, "keys")
    assert torch.equal(vc[written].cpu(), proj[:, nq + nk:].reshape(rows, G, vdim))
    mask = torch.ones(kc.shape[0], dtype=torch.bool)
    mask[written] = False
    assert bool((kc.cpu()[mask] == 7.0).all()) and bool((vc.cpu()[mask] == 7.0).all())


def _attend_case(dtype, H, G, dim, vdim, block_size, cached, n_new, loud, quiet=-12.0, seed=0, n_splits=0, prefill=True,
                 gated=True):
    """A hand-made cache of one sequence: every key scores about `quiet` (far below the sink) but the one at position
    `loud`, which scores about +6: a row that sees it carries its value, a row that does not carries almost nothing."""
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(seed)
    n = cached + n_new
    (tok, pos, par), hb = _params([n_new], [cached], block_size=block_size)
    K, V = torch.randn(n, G, dim, generator=g) * 0.05, torch.randn(n, G, vdim, generator=g)
    q = torch.randn(n_new, H, dim, generator=g) * 0.05
    q[:, :, 0] = 4.0
    K[:, :, 0] = quiet / 4.0
    if loud is not None:
        K[loud, :, 0] = 1.5
    K, V = K.to(dtype), V.to(dtype)
    gate = torch.randn(n_new, H * vdim + 8, generator=g).to(dtype)
    kc = torch.zeros((256 * block_size, G, dim), dtype=dtype, device=DEV)
    vc = torch.zeros((256 * block_size, G, vdim), dtype=dtype, device=DEV)
    sl = _slots(hb, 0, n, block_size)
    kc[sl], vc[sl] = K.to(DEV), V.to(DEV)
    out = torch.zeros(n_new, H * vdim + 8, dtype=dtype, device=DEV)
    kernels.sink_attn(q.to(DEV), kc, vc, None, None, torch.zeros(H, device=DEV), par.q_cu_seq_lens, par.kv_cu_seq_lens,
                      par.block_tables, par.cu_block_lens, par.token_seq, block_size, 1.0, 1 if prefill else 0, n_new, n,
                      n_splits, gate=gate.to(DEV)[:, 8:] if gated else None, out_mul=0.6, out=out[:, 8:])
    assert float(out[:, :8].abs().max()) == 0.0
    want = og.attend_with_one(q.double(), K.double(), V.double(), torch.arange(cached, n), 1.0).reshape(n_new, -1)
    return out[:, 8:], 0.6 * want * (torch.sigmoid(gate[:, 8:].double()) if gated else 1.0)


HEADS = [(4, 2, 16, 24), (3, 3, 10, 7), (8, 1, 32, 32), (6, 2, 48, 96), (2, 2, 64, 130), (16, 4, 64, 64), (4, 1, 128, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
def test_attention_far_keys_sink_and_cache_block_borders(H, G, dim, vdim, dtype):
    for bs in (1, 4, 16):
        for cached, loud in ((0, 0), (1, 0), (15, 3), (16, 15), (17, 16), (63, 0), (64, 63), (65, 64), (255, 1), (240, 128)):
            for n_splits in ((0,) if bs != 4 else (0, 1, 3)):
                got, want = _attend_case(dtype, H, G, dim, vdim, bs, cached, 1, loud, seed=cached, n_splits=n_splits)
                close(got, want, dtype, f"cached {cached} loud {loud} blocks of {bs}")
                assert float(want.abs().max()) > 0.15
    # nothing but quiet keys: the sink takes all the weight (without it the result would be an average of values)
    for n_new in (1, 20):
        got, want = _attend_case(dtype, H, G, dim, vdim, 4, 100, n_new, None, seed=3)
        close(got, want, dtype)
        assert float(want.abs().max()) < 0.02 and float(got.float().abs().max()) < 0.02


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
def test_attention_in_portions_loud_key_before_inside_and_after(H, G, dim, vdim, dtype):
    for cached, n_new, loud in ((0, 2, 0), (0, 40, 17), (30, 4, 2), (14, 13, 20), (100, 70, 3), (60, 10, 69), (33, 33, 64)):
        for prefill in (True, False):
            got, want = _attend_case(dtype, H, G, dim, vdim, 4, cached, n_new, loud, seed=cached + n_new, prefill=prefill)
            close(got, want, dtype, f"cached {cached} new {n_new} loud {loud}")
        sees = torch.arange(cached, cached + n_new) >= loud
        size = want.abs().amax(dim=1)
        assert bool((size[sees] > 0.1).all()) and bool((size[~sees] < 0.02).all())
    got, want = _attend_case(dtype, H, G, dim, vdim, 4, 20, 9, 5, seed=1, gated=False)
    close(got, want, dtype, "no gate")


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_rows_of_single_tokens_and_portions_in_the_recurrences(dtype):
    """A step with one long portion and many single tokens, each sequence against itself alone."""
    from scalellm_b200 import kernels
    H, N, V = 2, 24, 16
    n, nv = H * N, H * V
    g = torch.Generator().manual_seed(4)
    lens = [1, 45, 1, 2, 1]
    proj = torch.randn(sum(lens), 2 * n + nv, generator=g).to(dtype).to(DEV)
    fb, low, nw = torch.randn(n, generator=g).to(DEV), torch.rand(n, generator=g).to(DEV), torch.ones(V, device=DEV)
    st0 = torch.randn(5, H, N, V, generator=g).to(DEV)
    (tok, pos, par), _ = _params(lens, [3, 0, 7, 1, 0], slots=[4, 2, 0, 1, 3])
    st = st0.clone()
    both = kernels.forget_scan(proj[:, :n], proj[:, n:2 * n], proj[:, 2 * n:], fb, low, nw, st, par.q_cu_seq_lens, pos,
                               par.state_slots, 5, 45, EPS)
    at = 0
    for i, (m, c, sl) in enumerate(zip(lens, [3, 0, 7, 1, 0], [4, 2, 0, 1, 3])):
        (tok, pos, par), _ = _params([m], [c], slots=[sl])
        s1, p = st0.clone(), proj[at:at + m].contiguous()
        one = kernels.forget_scan(p[:, :n], p[:, n:2 * n], p[:, 2 * n:], fb, low, nw, s1, par.q_cu_seq_lens, pos,
                                  par.state_slots, 1, m, EPS)
        close(both[at:at + m], one.cpu(), dtype, i)       # (alone a single token takes another form of the walk)
        close(st[sl], s1[sl].cpu(), torch.float32, i, tol=2e-5 if dtype == torch.float32 else 1e-4)
        at += m


# ------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
def test_whole_prompt_layers_and_logits(name, dtype):
    from scalellm_b200.decode_step import build_step_batch
    cfg = gc.CONFIGS[name]
    model, oracle = build(cfg, dtype)
    eng = engine_for(model)
    tokens = toks(75, cfg["vocab"], 1)
    lo = []
    want = oracle.forward(tokens, oracle.new_state(), lo)
    s = eng.open("x")
    eng.pool.reserve(s.seq, len(tokens))
    tok, pos, par = eng.bufs.upload(build_step_batch(eng.pool, [s.seq], [tokens], [0], [s.slot]))
    got_layers = []
    got = model.forward(tok, pos, par, layer_out=got_layers)
    assert len(got_layers) == len(lo) == len(cfg["layers"])
    for a, b in zip(got_layers, lo):
        assert_rows((a.cpu().double() - b).abs().amax(dim=1) / float(b.abs().max()), dtype)
    assert_logits(got, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
def test_prefill_decode_and_portions_agree_with_the_oracle(name, dtype):
    cfg = gc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=1)
    tokens = toks(90, cfg["vocab"], 2)
    want = oracle_logits(oracle, tokens)
    for cuts in ([90], [58], [1] * 3, [2, 2, 5, 2, 31, 1, 2, 17, 2], [7] * 13, [33, 4, 4, 4, 40], [2] * 45):
        assert_logits(run_schedule(engine_for(model, block_size=4), tokens, cuts), want, dtype, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiles", "mix"])
def test_long_portions_over_many_tiles_and_chunks(name, dtype):
    """Portions cut at places that are no multiple of a key tile, a cache block or a chunk of a scan."""
    cfg = gc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=6)
    tokens = toks(333, cfg["vocab"], 7)
    want = oracle_logits(oracle, tokens)
    for cuts in ([333], [150, 2, 181], [129, 130, 71], [63, 1, 1, 64, 100], [64, 128, 65, 2]):
        assert_logits(run_schedule(engine_for(model, max_tokens=400, block_size=16), tokens, cuts), want, dtype, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "tiles", "wide"])
def test_mixed_batches_with_reused_blocks_and_slots(name, dtype):
    """Five unequal requests through a pool and state slots for three: portions beside single tokens, requests that
    pause, blocks and slots handed on without being cleared."""
    from scalellm_b200.engine import StepEntry
    cfg = gc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=2, max_seqs=3)
    lens = {"a": 61, "b": 9, "c": 40, "d": 1, "e": 33}
    T = {k: toks(n, cfg["vocab"], 10 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: oracle_logits(oracle, v) for k, v in T.items()}
    eng = engine_for(model, max_tokens=128, block_size=4, max_seqs=3)
    plan = [[("a", 17), ("b", 2)], [("a", 2), ("b", 1), ("c", 5)], [("b", 6), ("c", 1)], [("a", 30), ("c", 30)],
            [("a", 1), ("c", 2)], [("a", 1), ("c", 2), ("d", 1)], [("a", 10), ("e", 2)], [("e", 29)], [("e", 1)], [("e", 1)]]
    at, got = {k: 0 for k in T}, {k: [] for k in T}
    for step in plan:
        out = eng.step([StepEntry(k, T[k][at[k]:at[k] + n], list(range(n))) for k, n in step]).float().cpu()
        r = 0
        for k, n in step:
            got[k].append(out[r:r + n])
            r += n
            at[k] += n
            if at[k] == lens[k]:
                eng.finish(k)
    for k in T:
        assert at[k] == lens[k]
        assert_logits(torch.cat(got[k]), want[k], dtype, k)
    for k in ("a", "e"):       # each request alone gives the same rows as in the batch, beyond rounding
        alone = run_schedule(engine_for(model, max_tokens=128, block_size=4, max_seqs=3), T[k], [lens[k]], rid=k)
        assert_logits(torch.cat(got[k]), alone, dtype)
    assert eng.pool.n_free_blocks() == 32 and len(eng.slots.free) == 3 and not eng.seqs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "odd"])
def test_long_decoding_over_small_blocks(name, dtype):
    cfg = gc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=3)
    tokens = toks(200, cfg["vocab"], 4)
    want = oracle_logits(oracle, tokens)
    assert_logits(run_schedule(engine_for(model, max_tokens=208, block_size=2), tokens, [3]), want, dtype)


@pytest.mark.parametrize("name", ["mix", "tiles"])
def test_graph_replay_of_single_token_steps(name):
    cfg = gc.CONFIGS[name]
    model, oracle = build(cfg, torch.bfloat16, seed=4)
    tokens = toks(40, cfg["vocab"], 5)
    eng = engine_for(model, block_size=4, use_graphs=True)
    got = run_schedule(eng, tokens, [6])
    assert eng._graphs, "no graph was captured"
    assert_logits(got, oracle_logits(oracle, tokens), torch.bfloat16)


@pytest.mark.parametrize("name", ["mix", "tiles"])
def test_greedy_generation_through_the_scheduler(name):
    """More requests than places; the ids must be those of greedy decoding with the oracle wherever its two best
    logits are not a near tie."""
    from scalellm_b200.engine import SamplingParams
    cfg = gc.CONFIGS[name]
    model, oracle = build(cfg, torch.float32, seed=5, max_seqs=2)
    eng = engine_for(model, max_tokens=96, block_size=4, max_seqs=2)
    prompts = [toks(n, cfg["vocab"], 20 + n) for n in (5, 17, 1, 9)]
    outs = eng.generate(prompts, [SamplingParams(max_new_tokens=6) for _ in prompts], max_step_tokens=8)
    for p, o in zip(prompts, outs):
        assert len(o) == 6
        st = oracle.new_state()
        lg = oracle.forward(p, st)[-1]
        for tok in o:
            top = torch.topk(lg, 2).values
            if float(top[0] - top[1]) > 1e-3:
                assert int(lg.argmax()) == tok
            lg = oracle.forward([tok], st)[-1]


def test_model_folder_through_the_registry(tmp_path):
    """config.json + model.safetensors -> registry -> engine: the way the commands load a model."""
    from scalellm_b200 import checkpoint, registry
    cfg = gc.CONFIGS["odd"]
    w = gc.weights(cfg, 8)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    checkpoint.write_safetensors(str(tmp_path / "model.safetensors"), w)
    model = registry.load_model(str(tmp_path), torch.float32, DEV, max_seqs=2)
    tokens = toks(30, cfg["vocab"], 9)
    got = run_schedule(engine_for(model, max_tokens=64, block_size=16, max_seqs=2), tokens, [11, 2])
    assert_logits(got, oracle_logits(og.Gugalorn(cfg, w), tokens), torch.float32)
    with pytest.raises(ValueError):
        model.load_weights(dict(w, **{"l0.mix.o": w["l0.mix.o"][:, 1:]}))
    with pytest.raises(KeyError):
        model.load_weights({k: v for k, v in w.items() if k != "final.norm"})
