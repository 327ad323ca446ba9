"""GPU: the Palulorn decoder through the serving engine against the plain CPU restatement (oracle/palulorn.py, float64):
every mechanism alone, whole prompts, token-by-token decoding, portions, mixed batches, reuse of blocks and state slots,
keys far away, at cache-block borders and at the edges of a window, the sink, the first tokens, states carried over steps
and over the passes of a loop, generation through the scheduler."""
import json
import math

import numpy as np
import pytest
import torch

from oracle import palulorn as op
from tests import palulorn_case as pc

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0) if torch.cuda.is_available() else None
TOL = {torch.float32: 1e-4, torch.bfloat16: 8e-2}
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5


@pytest.fixture(autouse=True)
def _one_thread():
    """The restatement works on small matrices one token at a time: more threads only wait for each other."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def build(cfg, dtype, seed=0, max_seqs=4):
    """In bf16 the experts of a layer are nearly alike, so that a choice which rounding turns over changes little (other
    tests tell experts apart: the model in float32, the router, the expert products and the layer in both formats)."""
    from scalellm_b200 import registry
    w = pc.weights(cfg, seed, alike=0.0 if dtype == torch.float32 else 0.998)
    model = registry.create_model(cfg, dtype, DEV, max_seqs=max_seqs)
    model.load_weights({k: v.to(DEV) for k, v in w.items()})
    return model, op.Palulorn(cfg, w)


def engine_for(model, max_tokens=512, block_size=4, max_seqs=4, use_graphs=False):
    from scalellm_b200.engine import Engine
    return Engine(model, max_tokens, block_size=block_size, max_seqs=max_seqs, use_graphs=use_graphs)


def oracle_logits(oracle, tokens):
    return oracle.forward(tokens, oracle.new_state())


def frail_rows(oracle, tokens, dtype, want=None):
    """Rows that rest on a close call (a router's last choice, a read-out of nearly zero under its norm): the restatement
    itself, its products and norms shaken as rounding to 16 bits may shake them, leaves the tolerance there."""
    frail = torch.zeros(len(tokens), dtype=torch.bool)
    if dtype == torch.float32:
        return frail
    want = oracle_logits(oracle, tokens) if want is None else want
    for seed in range(2):
        with op.shaken(seed):
            frail |= pc.row_errors(oracle_logits(oracle, tokens), want) > TOL[dtype] / 2
    return frail


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
    """float32: every row within the tolerance.  bfloat16: the typical row is held to the tolerance and at most a tenth may
    exceed it (a choice may turn over with rounding where the restatement's own rounding does not turn it).  Faults of
    logic show in float32, and in the tests of single mechanisms, which hold every row in both formats."""
    if dtype == torch.float32:
        assert float(e.max()) < TOL[dtype], f"{what}: {float(e.max())}"
        return
    over = int((e > TOL[dtype]).sum())
    assert float(e.median()) < TOL[dtype] / 2 and over <= max(2, e.numel() // 10), \
        f"{what}: median {float(e.median())}, {over} of {e.numel()} rows over"


def assert_logits(got, want, dtype, what="", frail=None):
    e = pc.row_errors(got, want)
    if frail is not None and bool(frail.any()):
        assert int(frail.sum()) <= max(1, int(0.6 * e.numel())), f"{what}: too many frail rows to tell"
        assert bool(torch.isfinite(e).all())
        e = e[~frail]
    if e.numel():
        assert_rows(e, dtype, what)


def close(got, want, dtype, what="", tol=None):
    tol = tol or (2e-5 if dtype == torch.float32 else 2e-2)
    err = float((got.double().cpu() - want.double()).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), f"{what}: {err}"


# Two sequences in two of three state slots, fed in portions of 1, 2, fewer and more tokens than a filter has taps, and
# more than a tile or a chunk; the slots hold stale numbers of an old owner.
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
@pytest.mark.parametrize("W", [1, 42, 200, 1032])
@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_sum_without_norm_and_with_one_row_for_all(W, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(W)
    x, y = torch.randn(5, W, generator=g) * 3.0, torch.randn(5, W, generator=g).to(dtype)
    w = 0.5 + torch.rand(W, generator=g)
    both = torch.full((5, 2 * W + 8), 7.0, dtype=dtype, device=DEV)
    out, h = kernels.prenorm(x.to(DEV), y.to(DEV), None, 0.0, dtype, out=both[:, 8:8 + W])     # into a column block
    want = x.double() + y.double()
    close(out, want, torch.float32)
    assert torch.equal(both[:, 8:8 + W].cpu(), want.float().to(dtype)) and bool((both[:, :8] == 7.0).all())
    assert bool((both[:, 8 + W:] == 7.0).all())
    out, h = kernels.prenorm(x.to(DEV), y[2].to(DEV), w.to(DEV), EPS, dtype)                   # one row for all
    close(out, x.double() + y[2].double(), torch.float32)
    close(h, op.norm(x.double() + y[2].double(), w.double(), EPS), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_loop_input(dtype):
    from scalellm_b200.layers import LoopInput
    g = torch.Generator().manual_seed(1)
    W = 40
    w_in = (torch.randn(W, 2 * W, generator=g) / 9.0).to(torch.bfloat16)
    x0, x, y = (torch.randn(6, W, generator=g) for _ in range(3))
    loop = LoopInput(w_in.to(DEV), dtype)
    both = loop.start(x0.to(DEV))
    for yy in (y.to(dtype), None):                             # twice over the same rows: x_0 stays in place
        total_x = x.double() + (0.0 if yy is None else yy.double())
        got_x, got = loop(x.to(DEV), None if yy is None else yy.to(DEV), both)
        close(got_x, total_x, torch.float32)
        assert got.dtype == torch.float32
        # the sums are fp32; 16-bit rows go in
        rows = torch.cat([total_x.float().to(dtype), x0.to(dtype)], dim=1).double()
        close(got, rows @ w_in.double().T, torch.float32, tol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("blocks,n,k", [(0, 5, 33), (0, 64, 128), (3, 10, 7), (4, 64, 32), (1, 6, 40)])
def test_products_with_fp32_results(blocks, n, k, dtype):
    from scalellm_b200.layers import LinearF32
    g = torch.Generator().manual_seed(n)
    shape = (blocks, n, k) if blocks else (n, k)
    w = torch.randn(shape, generator=g).to(torch.bfloat16).float()
    x = torch.randn(9, max(blocks, 1) * k + 3, generator=g).to(dtype)
    xd = x.to(DEV)[:, 3:]
    for weight in (w, w * 1.001):                              # the second is no 16-bit number: it stays in fp32
        got = LinearF32(weight.to(DEV), dtype)(xd)
        assert got.dtype == torch.float32
        xs = x[:, 3:].double()
        want = (torch.stack([xs[:, b * k:(b + 1) * k] @ weight[b].double().T for b in range(blocks)]) if blocks
                else xs @ weight.double().T)
        close(got, want, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ch,taps", [(40, 4), (37, 3), (20, 1), (24, 9), (700, 6)])
def test_filter_of_biased_inputs_over_portions(ch, taps, dtype):
    """A bias of the inputs is not there before the first token: zeros, not biases, stand at the start."""
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(ch + taps)
    filt, ib, b = torch.randn(ch, taps, generator=g), torch.randn(ch, generator=g) * 2.0, torch.randn(ch, generator=g)
    data = {s: (torch.randn(total(s), ch + 4, generator=g).to(dtype),) for s in PLANS}
    fd, ibd, bd = filt.t().contiguous().to(DEV), ib.to(DEV), b.to(DEV)
    for bias in (None, bd):
        state = torch.full((3, taps - 1, ch), 5.0, device=DEV)
        got = over_portions(data, lambda step, rows, pos, par: kernels.causal_filter(
            rows[0][:, 4:], fd, bias, state, par.q_cu_seq_lens, pos, par.state_slots, 2, par.q_max_seq_len, False, in_bias=ibd))
        for s in PLANS:
            x = data[s][0][:, 4:].double() + ib.double()
            st = {}
            close(got[s], op.short_filter(x, filt.double(), st, "k") + (0.0 if bias is None else b.double()), dtype, s)
            if taps > 1:
                close(state[SLOT_OF[s]], st["k"], torch.float32, s)
        assert taps == 1 or bool((state[1] == 5.0).all())


MEMORY = [(3, 20, 12), (1, 9, 15), (2, 64, 64), (2, 128, 128), (1, 150, 136), (4, 16, 7), (1, 40, 300), (1, 300, 40),
          (2, 32, 16), (2, 8, 96), (1, 128, 256)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,N,V", MEMORY)
@pytest.mark.parametrize("form", ["", "simt"])
def test_matrix_memory_over_portions(H, N, V, dtype, form, monkeypatch):
    """Gates from nearly closed to loud, forget gates from nothing to everything: the running maximum moves, and rests at 0
    in the beginning; both sides of the denominator's maximum occur."""
    from scalellm_b200 import kernels
    monkeypatch.setenv("B200_SCAN_IMPL", form)                   # portions on the tensor cores where they fit, or never
    g = torch.Generator().manual_seed(H * N + V)
    cap, n, nv, parts = 7.0, H * N, H * V, kernels.memory_parts(N, V)
    ib, fb = torch.randn(H, generator=g) * 2.0 - 1.0, torch.randn(H, generator=g) * 3.0 + 2.0
    data = {}
    for s in PLANS:
        z = torch.randn(total(s), 2 * H + 1, generator=g) * 4.0
        z[:6, :H] -= 12.0                                        # the first tokens whisper: m stays at its start
        z[20, :H] += 30.0
        data[s] = (torch.randn(total(s), 2 * n + nv, generator=g).to(dtype), z)
    state = torch.full((3, H, N, V), 5.0, device=DEV)
    keys = torch.full((3, H, parts, N + 1), 5.0, device=DEV)
    d = [ib.to(DEV), fb.to(DEV)]
    got = over_portions(data, lambda step, rows, pos, par: kernels.memory_scan(
        rows[0][:, :n], rows[0][:, n:2 * n], rows[0][:, 2 * n:], rows[1][:, :H], rows[1][:, H:2 * H], *d, cap, N ** -0.5,
        state, keys, par.q_cu_seq_lens, pos, par.state_slots, 2, par.q_max_seq_len))
    for s in PLANS:
        p, z, T = data[s][0].double(), data[s][1].double(), total(s)
        i = cap * torch.tanh((z[:, :H] + ib.double()) / cap)
        f = op.log_sigmoid(cap * torch.tanh((z[:, H:2 * H] + fb.double()) / cap))
        S, ks, m = torch.zeros(H, N, V, dtype=torch.float64), torch.zeros(H, N, dtype=torch.float64), torch.zeros(H, dtype=torch.float64)
        want = op.matrix_memory(p[:, :n].reshape(T, H, N) * N ** -0.5, p[:, n:2 * n].reshape(T, H, N),
                                p[:, 2 * n:].reshape(T, H, V), i, f, S, ks, m).reshape(T, nv)
        # the walk is fp32 whatever the inputs' type is; a row whose denominator is near zero is compared at its own size
        err = ((got[s].double() - want).reshape(T, H, V).norm(dim=-1) / (want.reshape(T, H, V).norm(dim=-1) + 1.0)).max()
        assert float(err) < (2e-4 if dtype == torch.float32 else 1e-3), (s, float(err))
        close(state[SLOT_OF[s]], S, torch.float32, f"state {s}", tol=5e-5)
        for part in range(parts):                                # every copy of n and m
            close(keys[SLOT_OF[s], :, part, :N], ks, torch.float32, f"keys {s}", tol=5e-5)
            close(keys[SLOT_OF[s], :, part, N], m, torch.float32, f"maximum {s}", tol=5e-5)
    assert bool((state[1] == 5.0).all()) and bool((keys[1] == 5.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,parts", [(60, 4), (15, 3), (13, 13), (256, 1), (1024, 8), (1000, 20), (6, 1)])
def test_norm_in_parts_then_gate(n, parts, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(n + parts)
    y, w = torch.randn(5, n, generator=g) * 3.0, 0.5 + torch.rand(n, generator=g)
    y[:, : n // parts] *= 50.0                                   # a loud part must not quiet the others
    z = torch.randn(5, n + 4, generator=g).to(dtype)
    got = kernels.gated_part_norm(y.to(DEV), z.to(DEV)[:, 4:], w.to(DEV), parts, EPS, gate_after=True)
    want = op.norm(y.double().reshape(5, parts, -1), w.double().reshape(parts, -1), EPS).reshape(5, n)
    close(got, want * torch.sigmoid(z[:, 4:].double()), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,blocks", [(40, 5), (13, 1), (21, 7), (128, 2), (600, 3)])
@pytest.mark.parametrize("chunk", [0, 1, 5, 64])
def test_real_gated_recurrence_over_portions(width, blocks, chunk, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(width + blocks)
    n = width // blocks
    rb, ib, lam, yb = (torch.randn(width, generator=g) for _ in range(4))
    lam = lam * 4.0 - 2.0                                        # decays from nothing kept to nearly everything kept
    data = {s: (torch.randn(total(s), width, generator=g).to(dtype), torch.randn(total(s), width + 5, generator=g).to(dtype),
                torch.randn(total(s), 2 * width, generator=g) * 2.0) for s in PLANS}
    state = torch.full((3, width), 5.0, device=DEV)
    d = [t.to(DEV) for t in (rb, ib, lam, yb)]

    def run(step, rows, pos, par):
        z = rows[2].reshape(-1, blocks, 2 * n).transpose(0, 1).contiguous()
        return kernels.real_gated_scan(rows[0], rows[1][:, 5:], z, d[0], d[1], d[2], d[3], -8.0, state, par.q_cu_seq_lens,
                                       pos, par.state_slots, 2, par.q_max_seq_len, chunk_len=chunk)
    got = over_portions(data, run)
    for s in PLANS:
        u, y, z = (t.double() for t in data[s])
        z = z.reshape(-1, blocks, 2, n)
        r = torch.sigmoid(z[:, :, 0].reshape(-1, width) + rb.double())
        i = torch.sigmoid(z[:, :, 1].reshape(-1, width) + ib.double())
        S = torch.zeros(width, dtype=torch.float64)
        want = op.gated_scan(u, r, i, lam.double(), S) * op.gelu_tanh(y[:, 5:] + yb.double())
        close(got[s], want, dtype, s)
        close(state[SLOT_OF[s]], S, torch.float32, f"state {s}")
    assert bool((state[1] == 5.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,rot,norm", [(4, 2, 16, 24, 8, True), (3, 3, 10, 7, 2, True), (6, 2, 12, 20, 12, False),
                                                   (2, 1, 64, 130, 0, True), (5, 1, 6, 5, 6, False)])
def test_attention_inputs_biases_norms_turn_temperature(H, G, dim, vdim, rot, norm, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(H * dim)
    bs = 4
    (tok, pos, par), hb = _params([5, 1], [3, 9], block_size=bs)
    rows, nq, nk, nv = 6, H * dim, G * dim, G * vdim
    proj = torch.randn(rows, nq + nk + nv, generator=g)
    proj[:, :dim] *= 10.0                                        # one loud head
    proj = proj.to(dtype)
    qb, kb, vb = (torch.randn(n, generator=g) for n in (nq, nk, nv))
    qw, kw = 0.5 + torch.rand(dim, generator=g), 0.5 + torch.rand(dim, generator=g)
    f = torch.tensor([100.0 ** (-2.0 * i / max(rot, 1)) / 3.0 for i in range(rot // 2)], dtype=torch.float32)
    pd, p64, positions = proj.to(DEV), proj.double(), torch.tensor([3, 4, 5, 6, 7, 9])
    for biased, temp in ((True, True), (False, False)):
        kc = torch.full((256 * bs, G, dim), 7.0, dtype=dtype, device=DEV)
        vc = torch.full((256 * bs, G, vdim), 7.0, dtype=dtype, device=DEV)
        v_in = pd[:, nq + nk:] if biased else None               # without values: only keys are cached
        dv = lambda t, on: t.to(DEV) if on else None
        q = kernels.sink_attn_prepare_heads(pd[:, :nq], pd[:, nq:nq + nk], v_in, kc, vc, pos, par.new_cache_slots, H, G, dim,
                                            dv(qb, biased), dv(kb, biased), dv(vb, biased), dv(qw, norm), dv(kw, norm),
                                            f.to(DEV) if rot else None, rot, EPS, 0.5 if temp else 0.0, 5 if temp else 0)
        b = 1.0 if biased else 0.0
        wq = (p64[:, :nq] + b * qb.double()).reshape(rows, H, dim)
        wk = (p64[:, nq:nq + nk] + b * kb.double()).reshape(rows, G, dim)
        if norm:
            wq, wk = op.norm(wq, qw.double(), EPS), op.norm(wk, kw.double(), EPS)
        if rot:
            wq, wk = op.turn(wq, positions, 100.0, rot, 3.0), op.turn(wk, positions, 100.0, rot, 3.0)
        if temp:
            wq = wq * op.temperature(positions, 0.5, 5)[:, None, None]
        close(q, wq, torch.float32, "queries")
        written = _slots(hb, 0, 8, bs)[3:] + [_slots(hb, 1, 10, bs)[9]]
        close(kc[written], wk, dtype, "keys")
        mask = torch.ones(kc.shape[0], dtype=torch.bool)
        mask[written] = False
        assert bool((kc.cpu()[mask] == 7.0).all()) and bool((vc.cpu()[mask] == 7.0).all())
        if biased:
            close(vc[written], (p64[:, nq + nk:] + vb.double()).reshape(rows, G, vdim), dtype, "values")
        else:
            assert bool((vc == 7.0).all())


def _attend_case(dtype, H, G, dim, vdim, block_size, cached, n_new, loud, window, shared, quiet=-12.0, seed=0, n_splits=0,
                 prefill=True, sink=True):
    """A hand-made cache of one sequence: every key scores about `quiet` (far below the sink) but those at the positions
    `loud`, which score about +6: a row that sees one carries its value, a row that does not carries almost nothing."""
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(seed)
    n = cached + n_new
    (tok, pos, par), hb = _params([n_new], [cached], block_size=block_size)
    K, V = torch.randn(n, G, dim, generator=g) * 0.05, torch.randn(n, G, vdim, generator=g)
    q = torch.randn(n_new, H, dim, generator=g) * 0.05
    q[:, :, 0] = 4.0
    K[:, :, 0] = quiet / 4.0
    for j in loud:
        K[j, :, 0] = 1.5
    K, V = K.to(dtype), V.to(dtype)
    if shared:
        V = K
    gate = torch.randn(n_new, H + 8, generator=g).to(dtype)
    kc = torch.zeros((256 * block_size, G, dim), dtype=dtype, device=DEV)
    sl = _slots(hb, 0, n, block_size)
    kc[sl] = K.to(DEV)
    vc = kc
    if not shared:
        vc = torch.zeros((256 * block_size, G, vdim), dtype=dtype, device=DEV)
        vc[sl] = V.to(DEV)
    sk = torch.linspace(-1.0, 1.0, H)
    out = kernels.sink_attn(q.to(DEV), kc, vc, None, None, sk.to(DEV) if sink else None, par.q_cu_seq_lens, par.kv_cu_seq_lens,
                            par.block_tables, par.cu_block_lens, par.token_seq, block_size, 1.0, 1 if prefill else 0, n_new, n,
                            n_splits, gate=gate.to(DEV)[:, 8:], out_mul=0.6, window=window)
    want = op.attend(q.double(), K.double(), V.double(), torch.arange(cached, n), 1.0, window, sk.double() if sink else None)
    want = want * torch.sigmoid(gate[:, 8:].double())[:, :, None] * 0.6
    return out, want.reshape(n_new, -1)


HEADS = [(4, 2, 16, 24), (3, 3, 10, 7), (8, 1, 32, 32), (6, 2, 48, 96), (2, 2, 64, 130), (16, 4, 64, 64), (4, 1, 128, 128),
         (20, 1, 16, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
def test_attention_single_tokens_at_window_edges_and_block_borders(H, G, dim, vdim, dtype):
    for bs in (1, 4, 16):
        for cached, window in ((0, 1), (5, 1), (15, 9), (16, 16), (17, 5), (64, 64), (65, 33), (200, 64), (255, 100), (130, 0), (40, 90)):
            first = max(0, cached - window + 1) if window else 0
            for loud in ({first}, {max(first - 1, 0)}):          # just inside, and (where there is one) just outside
                for n_splits in ((0,) if bs != 4 else (0, 1, 3)):
                    for shared in ((False, True) if dim == vdim else (False,)):
                        got, want = _attend_case(dtype, H, G, dim, vdim, bs, cached, 1, loud, window, shared, seed=cached,
                                                 n_splits=n_splits)
                        close(got, want, dtype, f"cached {cached} window {window} loud {loud} blocks of {bs} shared {shared}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
def test_attention_in_portions_at_window_edges(H, G, dim, vdim, dtype):
    """Rows enter and leave the sight of a loud key inside a portion, at places that are no multiple of a tile."""
    for cached, n_new, loud, window in ((0, 2, 0, 1), (0, 40, 17, 9), (30, 4, 2, 29), (14, 13, 20, 4), (100, 70, 103, 31),
                                        (60, 10, 5, 64), (33, 130, 64, 65), (0, 90, 3, 40), (100, 70, 3, 0)):
        for prefill in (True, False):
            for shared in ((False, True) if dim == vdim else (False,)):
                got, want = _attend_case(dtype, H, G, dim, vdim, 4, cached, n_new, {loud}, window, shared, seed=cached + n_new,
                                         prefill=prefill)
                close(got, want, dtype, f"cached {cached} new {n_new} loud {loud} window {window} shared {shared}")
        if not shared:
            i = torch.arange(cached, cached + n_new)
            sees = (i >= loud) & ((i - loud < window) if window else True)
            size = want.abs().amax(dim=1)
            assert bool((size[sees] > 0.03).all()) and bool((size[~sees] < 0.02).all())
    got, want = _attend_case(dtype, H, G, dim, vdim, 4, 20, 9, set(), 7, False, seed=1, sink=False)
    close(got, want, dtype, "no sink")
    for n_new in (1, 20):                                        # nothing but quiet keys: the sink takes all the weight
        got, want = _attend_case(dtype, H, G, dim, vdim, 4, 50, n_new, set(), 30, False, seed=3)
        assert float(want.abs().max()) < 0.02 and float(got.float().abs().max()) < 0.02


@pytest.mark.parametrize("E,top,count,keep,best", [(8, 3, 2, 1, 2), (6, 2, 3, 2, 2), (5, 2, 1, 1, 2), (12, 4, 12, 7, 2), (64, 6, 8, 3, 2),
                                                   (1000, 32, 4, 2, 2), (1, 1, 1, 1, 2), (40, 5, 5, 3, 1), (96, 8, 48, 20, 3)])
def test_router_choice_under_group_limits(E, top, count, keep, best):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(E + top)
    z = torch.randn(37, E + 3, generator=g) * 2.0
    if E // count > best:                                        # one loud expert among quiet ones must not carry its group
        z[:, 3] = 6.0
        z[:, 4:3 + E // count] -= 8.0
    ids, wts = kernels.moe_route_sigmoid(z.to(DEV)[:, 3:], top, count, keep, best, 1e-20, 2.5)
    s = torch.sigmoid(z[:, 3:].double())
    score = s.reshape(37, count, -1).topk(min(best, E // count), dim=-1).values.sum(-1)
    alive = torch.zeros(37, count, dtype=torch.bool).scatter_(1, score.topk(keep, dim=-1).indices, True)
    c = s.masked_fill(~alive.repeat_interleave(E // count, dim=1), -1.0)
    want = c.topk(top, dim=-1)
    assert torch.equal(ids.cpu().long(), want.indices)
    close(wts, want.values / want.values.sum(-1, keepdim=True) * 2.5, torch.float32)
    if best == 2:
        oid, ow = op.route(z[:, 3:].double(), top, count, keep, 2.5)
        assert torch.equal(ids.cpu().long(), oid)
        close(wts, ow, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,E,top,N,K", [(1, 4, 2, 40, 24), (16, 8, 2, 128, 256), (50, 3, 2, 70, 136), (100, 2, 1, 33, 40),
                                            (90, 16, 4, 48, 64), (9, 5, 3, 10, 7)])
def test_expert_products_with_activation(rows, E, top, N, K, dtype):
    """Unequal expert loads (one expert takes most rows, one none), sizes that are no multiple of a tile."""
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(rows)
    ids = torch.stack([torch.randperm(E - 1, generator=g)[:top] if E - 1 >= top and r % 3 else torch.arange(top) for r in range(rows)])
    a, w = torch.randn(rows, K, generator=g).to(dtype), (torch.randn(E, N, K, generator=g) / math.sqrt(K)).to(dtype)
    scale = 0.5 + torch.rand(rows, top, generator=g)
    ids32 = ids.to(torch.int32).contiguous().to(DEV)
    offsets, sorted_pair, pos_of_pair = kernels.moe_plan(ids32, E)
    for act in ("", "relu_squared"):
        for sc in (None, scale):
            c = kernels.grouped_gemm(a.to(DEV), w.to(DEV), offsets, rows * top, sorted_pair,
                                     None if sc is None else sc.reshape(-1).contiguous().to(DEV), top, act=act)
            got = c[pos_of_pair.long()].reshape(rows, top, N)
            x = a.double()[:, None, :] * (torch.ones(rows, top, 1) if sc is None else sc[:, :, None]).double()
            want = torch.einsum("rtk,rtnk->rtn", x, w.double()[ids])
            close(got, torch.clamp(want, min=0.0) ** 2 if act else want, dtype, (act, sc is None))
            # from sorted rows, as the second product of an expert reads them
            xs = x.to(dtype).reshape(rows * top, K)[sorted_pair.cpu().long()].contiguous()
            c2 = kernels.grouped_gemm(xs.to(DEV), w.to(DEV), offsets, rows * top, act=act)
            close(c2[pos_of_pair.long()].reshape(rows, top, N), torch.clamp(want, min=0.0) ** 2 if act else want, dtype, act)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,f", [(64, pc.moe(24, 8, 3, 4, 2, scale=2.5, shared=40)), (42, pc.moe(10, 5, 2)),
                                 (40, pc.moe(16, 6, 1, 2, 1, scale=0.5, shared=8))])
def test_experts_layer(W, f, dtype):
    from scalellm_b200.layers import GroupSigmoidMoE, ReluSquaredMLP
    g = torch.Generator().manual_seed(W)
    E, ff, r = f["router"]["experts"], f["expert"]["ff"], f["router"]
    rnd = lambda *s: (torch.randn(*s, generator=g) / math.sqrt(s[-1])).to(torch.bfloat16)
    w = {"router": rnd(E, W) * 6}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = rnd(ff, W), rnd(W, ff)
    if "shared" in f:
        w["shared.up"], w["shared.down"] = rnd(f["shared"]["ff"], W), rnd(W, f["shared"]["ff"])
    d = lambda t: t.to(DEV).to(dtype)
    grp = r.get("groups") or {"count": 1, "keep": 1}
    stack = lambda leaf: torch.stack([d(w[f"e{e}.{leaf}"]) for e in range(E)])
    layer = GroupSigmoidMoE(w["router"].to(DEV), stack("up"), stack("down"), r["top"], grp["count"], grp["keep"], 2, 1e-20,
                            r["scale"], dtype, ReluSquaredMLP(d(w["shared.up"]), d(w["shared.down"])) if "shared" in f else None)
    for rows in (1, 19, 300):
        h = torch.randn(rows, W, generator=g).to(torch.bfloat16)
        want = op.moe_ff(h.double(), {k: v.double() for k, v in w.items()}, f)
        close(layer(d(h)), want, dtype, rows, tol=3e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("rows", [1, 16, 100])
def test_squared_relu_feed_forward_takes_split_k_partials(rows):
    from scalellm_b200 import kernels
    from scalellm_b200.layers import ReluSquaredMLP
    g = torch.Generator().manual_seed(rows)
    up, down = ((torch.randn(n, k, generator=g) / math.sqrt(k)).to(torch.bfloat16) for n, k in ((384, 256), (256, 384)))
    h = torch.randn(rows, 256, generator=g).to(torch.bfloat16)
    ff = ReluSquaredMLP(up.to(DEV), down.to(DEV))
    assert ff.up.supports_partials(rows)
    a = kernels.relu_squared(ff.up.forward_partials(h.to(DEV)), torch.bfloat16)
    close(a, torch.clamp(h.double() @ up.double().T, min=0.0) ** 2, torch.bfloat16)
    assert torch.equal(a, kernels.relu_squared(ff.up(h.to(DEV))))
    close(ff(h.to(DEV)), op.relu_squared_ff(h.double(), up.double(), down.double()), torch.bfloat16)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [42, 256])
def test_two_branches_join_without_a_norm_of_their_sum(W, dtype):
    from scalellm_b200 import kernels
    g = torch.Generator().manual_seed(W)
    x, a, b = torch.randn(5, W, generator=g), (torch.randn(5, W, generator=g) * 9).to(dtype), (torch.randn(5, W, generator=g) / 9).to(dtype)
    ba, wa, wb, wn = (torch.randn(W, generator=g) for _ in range(4))
    d = lambda t: t.to(DEV)
    D = lambda t: t.double()
    out, h = kernels.branch_norm_residual(d(x), d(a), d(b), d(wa), d(wb), None, d(wn), EPS, bias_a=d(ba))
    want = D(x) + (op.norm(D(a) + D(ba), D(wa), EPS) + op.norm(D(b), D(wb), EPS)) / 2
    close(out, want, torch.float32)
    close(h, op.norm(want, D(wn), EPS), dtype)
    out, h = kernels.branch_norm_residual(d(x), d(a), None, None, None, None, None, EPS, want_h=False, bias_a=d(ba))
    close(out, D(x) + D(a) + D(ba), torch.float32)
    assert h is None


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_rows_of_single_tokens_and_portions_in_the_recurrences(dtype):
    """A step with one long portion and many single tokens, each sequence against itself alone."""
    from scalellm_b200 import kernels
    H, N, V = 2, 24, 16
    n, nv = H * N, H * V
    g = torch.Generator().manual_seed(4)
    lens, cached, slots = [1, 45, 1, 2, 1], [3, 0, 7, 1, 0], [4, 2, 0, 1, 3]
    proj, z = torch.randn(sum(lens), 2 * n + nv, generator=g).to(dtype).to(DEV), torch.randn(sum(lens), 2 * H, generator=g).to(DEV)
    b = torch.ones(H, device=DEV)
    st0, ks0 = torch.randn(5, H, N, V, generator=g).to(DEV), torch.randn(5, H, 1, N + 1, generator=g).to(DEV)

    def run(p, zz, lens, cached, slots, st, ks):
        (tok, pos, par), _ = _params(lens, cached, slots=slots)
        return kernels.memory_scan(p[:, :n], p[:, n:2 * n], p[:, 2 * n:], zz[:, :H], zz[:, H:], b, b, 5.0, N ** -0.5, st, ks,
                                   par.q_cu_seq_lens, pos, par.state_slots, len(lens), max(lens))
    st, ks = st0.clone(), ks0.clone()
    both = run(proj, z, lens, cached, slots, st, ks)
    at = 0
    for m, c, sl in zip(lens, cached, slots):
        s1, k1 = st0.clone(), ks0.clone()
        one = run(proj[at:at + m].contiguous(), z[at:at + m].contiguous(), [m], [c], [sl], s1, k1)
        tol = 2e-5 if dtype == torch.float32 else 1e-3       # (alone a single token takes another form of the walk)
        close(both[at:at + m], one.cpu(), torch.float32, sl, tol=tol)
        close(st[sl], s1[sl].cpu(), torch.float32, sl, tol=tol)
        close(ks[sl], k1[sl].cpu(), torch.float32, sl, tol=tol)
        at += m


# ------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(pc.CONFIGS))
def test_whole_prompt_layers_and_logits(name, dtype):
    from scalellm_b200.decode_step import build_step_batch
    cfg = pc.CONFIGS[name]
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
    assert len(got_layers) == len(lo) == len(op.layer_runs(cfg))
    frail = frail_rows(oracle, tokens, dtype, want)
    for a, b in zip(got_layers, lo):
        assert_rows(((a.cpu().double() - b).abs().amax(dim=1) / float(b.abs().max()))[~frail], dtype)
    assert_logits(got, want, dtype, "", frail)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(pc.CONFIGS))
def test_prefill_decode_and_portions_agree_with_the_oracle(name, dtype):
    cfg = pc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=1)
    tokens = toks(90, cfg["vocab"], 2)
    want = oracle_logits(oracle, tokens)
    frail = frail_rows(oracle, tokens, dtype, want)
    for cuts in ([90], [58], [1] * 3, [2, 2, 5, 2, 31, 1, 2, 17, 2], [7] * 13, [33, 4, 4, 4, 40], [2] * 45):
        assert_logits(run_schedule(engine_for(model, block_size=4), tokens, cuts), want, dtype, cuts, frail)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiles", "mix"])
def test_long_portions_over_many_tiles_and_chunks(name, dtype):
    """Portions cut at places that are no multiple of a key tile, a cache block or a chunk of a scan."""
    cfg = pc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=6)
    tokens = toks(333, cfg["vocab"], 7)
    want = oracle_logits(oracle, tokens)
    frail = frail_rows(oracle, tokens, dtype, want)
    for cuts in ([333], [150, 2, 181], [129, 130, 71], [63, 1, 1, 64, 100]):
        assert_logits(run_schedule(engine_for(model, max_tokens=400, block_size=16), tokens, cuts), want, dtype, cuts, frail)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "tiles", "loop"])
def test_mixed_batches_with_reused_blocks_and_slots(name, dtype):
    """Five unequal requests through a pool and state slots for three: portions beside single tokens, requests that
    pause, blocks and slots handed on without being cleared."""
    from scalellm_b200.engine import StepEntry
    cfg = pc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=2, max_seqs=3)
    lens = {"a": 61, "b": 9, "c": 40, "d": 1, "e": 33}
    T = {k: toks(n, cfg["vocab"], 10 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: oracle_logits(oracle, v) for k, v in T.items()}
    frail = {k: frail_rows(oracle, v, dtype, want[k]) for k, v in T.items()}
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
        assert_logits(torch.cat(got[k]), want[k], dtype, k, frail[k])
    for k in ("a", "e"):       # each request alone gives the same rows as in the batch, beyond rounding
        alone = run_schedule(engine_for(model, max_tokens=128, block_size=4, max_seqs=3), T[k], [lens[k]], rid=k)
        assert_logits(torch.cat(got[k]), alone, dtype, k, frail[k])
    assert eng.pool.n_free_blocks() == 32 and len(eng.slots.free) == 3 and not eng.seqs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "odd"])
def test_long_decoding_over_small_blocks(name, dtype):
    cfg = pc.CONFIGS[name]
    model, oracle = build(cfg, dtype, seed=3)
    tokens = toks(160, cfg["vocab"], 4)
    want = oracle_logits(oracle, tokens)
    frail = frail_rows(oracle, tokens, dtype, want)
    assert_logits(run_schedule(engine_for(model, max_tokens=168, block_size=2), tokens, [3]), want, dtype, "", frail)


@pytest.mark.parametrize("name", ["mix", "tiles"])
def test_graph_replay_of_single_token_steps(name):
    cfg = pc.CONFIGS[name]
    model, oracle = build(cfg, torch.bfloat16, seed=4)
    tokens = toks(40, cfg["vocab"], 5)
    eng = engine_for(model, block_size=4, use_graphs=True)
    got = run_schedule(eng, tokens, [6])
    assert eng._graphs, "no graph was captured"
    assert_logits(got, oracle_logits(oracle, tokens), torch.bfloat16, "", frail_rows(oracle, tokens, torch.bfloat16))


@pytest.mark.parametrize("name", ["mix", "tiles"])
def test_greedy_generation_through_the_scheduler(name):
    """More requests than places; the ids must be those of greedy decoding with the oracle wherever its two best
    logits are not a near tie."""
    from scalellm_b200.engine import SamplingParams
    cfg = pc.CONFIGS[name]
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
    cfg = pc.CONFIGS["odd"]
    w = pc.weights(cfg, 8)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    checkpoint.write_safetensors(str(tmp_path / "model.safetensors"), w)
    model = registry.load_model(str(tmp_path), torch.float32, DEV, max_seqs=2)
    tokens = toks(30, cfg["vocab"], 9)
    got = run_schedule(engine_for(model, max_tokens=64, block_size=16, max_seqs=2), tokens, [11, 2])
    assert_logits(got, oracle_logits(op.Palulorn(cfg, w), tokens), torch.float32)
    with pytest.raises(ValueError):
        model.load_weights(dict(w, **{"l0.mix.left.o": w["l0.mix.left.o"][:, 1:]}))
    with pytest.raises(KeyError):
        model.load_weights({k: v for k, v in w.items() if k != "final.norm"})
