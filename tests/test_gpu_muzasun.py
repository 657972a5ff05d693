"""The Muzasun design in the engine against the plain implementation (`plain_muzasun.py`): every mechanism alone, prompts
against decoding, prompts in pieces, unequal batches, slots and pages that are used again, far keys and chunk borders, the
first tokens, long decoding, other sizes, greedy generation through the library's entry points."""
import dataclasses
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import herbert_rs_b200 as hb
import muzasun_util as U
import plain_muzasun as P
from gpu_util import DTYPES, assert_close as plain_assert_close, bound_for, engine_for, replay_batches, replay_tail_one_by_one, replay_whole, to_np, tol_for
from herbert_rs_b200 import ops

pytestmark = pytest.mark.gpu
DEV = "cuda"
VOCAB = 131
F64 = torch.float64


def ids_for(rng, vocab, n):
    return rng.integers(0, vocab, n).tolist()


_model_own: dict = {}


def assert_close(got, ref, dtype, what="", bound=None, plain=None, ids=None, rows=None, arith=torch.float64):
    """gpu_util's comparison, with steadier bounds for whole models: a head's read-out is divided by its own root mean square, so
    where it is short a rounding grows by a factor that depends on its direction.  bfloat16: three times what bfloat16 storage
    between kernels does to the plain implementation at most, over all rows of the request and over one fixed 64-token request
    of the model; at most one row in fifty (or one row) may lie above it, and none above one and a half times it.  float32:
    the usual bound, or six times what float32 arithmetic does to the plain implementation, whichever is larger."""
    if bound is not None or plain is None:
        return plain_assert_close(got, ref, dtype, what, bound=bound, plain=plain, ids=ids, rows=rows, arith=arith)

    def own_error(tokens):
        if dtype == "bfloat16":
            return float((plain.logits(tokens, arith, P.bf16_storage) - plain.logits(tokens, arith)).abs().max())
        return float((plain.logits(tokens, torch.float32).double() - plain.logits(tokens)).abs().max())
    key = (id(plain), dtype)
    if key not in _model_own:
        _model_own[key] = (plain, own_error(ids_for(np.random.default_rng(77), VOCAB, 64)))
    own = max(own_error(ids), _model_own[key][1])
    if dtype == "float32":
        return plain_assert_close(got, ref, dtype, what, bound=max(tol_for(dtype, np.asarray(ref)), 6.0 * own))
    bound = 3.0 * own
    ref = np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, (what, got.shape, ref.shape)
    err = np.abs(got - ref).max(axis=-1)
    over = int((err > bound).sum())
    assert err.max() <= 1.5 * bound and over <= max(1, len(err) // 50), \
        f"{what} [bfloat16]: {over} of {len(err)} rows over {bound:.3e}, the largest error {err.max():.3e} at row {int(err.argmax())}"
    return float(err.max())


def td_of(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def scratch(shape, dt):
    return torch.empty(shape, dtype=dt, device=DEV)


def step_of(lens, slots, pos0=None):
    """The device arrays of a step that the kernels of this file read: sequences of `lens` new tokens in `slots`."""
    pos0 = pos0 or [0] * len(lens)
    starts = np.concatenate([[0], np.cumsum(lens)])
    tok_seq = [b for b, n in enumerate(lens) for _ in range(n)]
    tok_pos = [pos0[b] + i for b, n in enumerate(lens) for i in range(n)]
    return SimpleNamespace(seq_slot=i32(slots), seq_start=i32(starts.tolist()), seq_pos0=i32(pos0), tok_seq=i32(tok_seq),
                           tok_pos=i32(tok_pos), n_seqs=len(lens), n_tokens=int(sum(lens)), max_q_len=max(lens),
                           seq_len=i32([p + n for p, n in zip(pos0, lens)]), is_decode=all(n == 1 for n in lens))


def in_cuts(data, cuts, slots, run):
    """Feeds sequences (lists of row tensors) in steps of the given cuts; run(rows of this step, batch) -> output rows.
    Returns per sequence the outputs at all of its rows."""
    done, got = [0] * len(cuts), [[] for _ in cuts]
    for r in range(max(len(c) for c in cuts)):
        live = [i for i in range(len(cuts)) if r < len(cuts[i])]
        cnt = [cuts[i][r] for i in live]
        rows = [torch.cat([data[i][j][done[i]:done[i] + c] for i, c in zip(live, cnt)]).to(DEV) for j in range(len(data[0]))]
        out, o = run(rows, step_of(cnt, [slots[i] for i in live], [done[i] for i in live])), 0
        for i, c in zip(live, cnt):
            got[i].append(to_np(out[o:o + c])); o += c; done[i] += c
    return [np.concatenate(g) for g in got]


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    """All three mixers, both feed-forwards and none; three attention layers that blend values and one that does not."""
    layers = [(U.attention(heads=2, kv_heads=1, dim=8, vdim=16, v_mix=False), U.dense()),
              (U.attention(heads=4, kv_heads=2, dim=16, vdim=24, rot_dims=8), U.moe()),
              (U.mlstm(heads=3, dim=16, vdim=20), U.dense(ff=40)),
              (U.delta(heads=4, kv_heads=2, dim=16, vdim=24), None),
              (U.attention(heads=4, kv_heads=2, dim=24, vdim=24), None),
              (U.attention(heads=6, kv_heads=3, dim=16, vdim=16), U.moe(experts=9, top=3, ff=24, shared=0))]
    return U.make(tmp_path_factory.mktemp("muzasun_mixed"), layers, seed=13)


# ---- each mechanism alone -------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [1, 47, 48, 1000, 2048])
def test_norms_without_statistics_behind_the_residual_sum(dtype, dim):
    g = torch.Generator().manual_seed(dim)
    T = 7
    X, y, yb = torch.randn(T, dim, generator=g) * 3.0, torch.randn(T, dim + 4, generator=g), torch.randn(dim, generator=g)
    n1, n2 = [(a, 1.0 + 0.2 * torch.randn(dim, generator=g), torch.randn(dim, generator=g)) for a in (0.6, 1.7)]
    dev = [(a, w.to(DEV), b.to(DEV)) for a, w, b in (n1, n2)]

    def want(x, n):
        return P.squash_norm(x, torch.tensor(n[0], dtype=F64), n[1].double(), n[2].double()).numpy()
    for bias in (None, yb):
        ref = X.double() + 0.3 * (y.double()[:, :dim] + (bias.double() if bias is not None else 0.0))
        for count in (0, 1, 2):
            x, hs = X.clone().to(DEV), [torch.empty(T, dim, dtype=td_of(dtype), device=DEV) for _ in range(count)]
            ops.residual_tanh(x, list(zip(dev, hs)), y=y.to(DEV)[:, :dim], mult=0.3, bias=bias.to(DEV) if bias is not None else None)
            assert_close(to_np(x), ref.numpy(), "float32", "stream")
            for h, n in zip(hs, (n1, n2)):
                assert_close(to_np(h), want(ref, n), dtype, "norm")
    x, rows = X.clone().to(DEV), [4, 0, 4]
    h = torch.empty(3, dim, dtype=td_of(dtype), device=DEV)
    ops.residual_tanh(x, [(dev[1], h)], rows=i32(rows))
    assert_close(to_np(h), want(X.double()[rows], n2), dtype, "chosen rows")
    assert torch.equal(x.cpu(), X)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv", [(1, 1, 1), (3, 5, 7), (2, 8, 16), (4, 16, 20)])
def test_gates_running_maximum_and_packed_rows(dtype, H, dk, dv):
    """Three sequences in steps of 1 to 300 tokens (a warp, a block, several rounds of it), gates that forget everything, keep
    everything, and barely write; every step continues the slot's running maximum."""
    g = torch.Generator().manual_seed(H * dk)
    cap, slots, lens = 6.0, [3, 0, 2], [620, 1, 50]
    cuts = [[300, 1, 31, 33, 255], [1], [20, 30]]
    dvp = (dv + 8) // 8 * 8
    W = 2 * H * dk + H * dv
    data = []
    for L in lens:
        rows = torch.randn(L, W + 2 * H + 1, generator=g)
        rows[:, W:W + 2 * H] *= 4.0
        rows[::7, W + H:W + 2 * H] = -40.0
        rows[100:160, W:W + H] = -40.0
        data.append([rows])
    bi, bf = torch.randn(H, generator=g), torch.randn(H, generator=g)
    m = torch.zeros(5, H, device=DEV)
    m[1] = 7.0
    ld = (H * (dvp + 2 * dk) + 7) // 8 * 8

    def run(rows, batch):
        T = rows[0].shape[0]
        packed = torch.full((T, ld), 9.0, dtype=td_of(dtype), device=DEV)
        ld_, wt, fl = (torch.empty(T, H, device=DEV) for _ in range(3))
        ops.matrix_memory_prepare(rows[0], 0, H * dk, 2 * H * dk, W, W + H, bi.to(DEV), bf.to(DEV), cap, m, batch, packed, ld_, wt, fl, H, dk, dv, dvp)
        return torch.cat([ld_, wt, fl, packed.float()], dim=1)
    got = in_cuts(data, cuts, slots, run)
    for b, L in enumerate(lens):
        z = data[b][0].double()
        i = P.capped(z[:, W:W + H] + bi.double(), cap)
        f = P.log_sigmoid(P.capped(z[:, W + H:W + 2 * H] + bf.double(), cap))
        run_m, want = torch.zeros(H, dtype=F64), []
        for t in range(L):
            new = torch.maximum(run_m + f[t], i[t])
            want.append(torch.cat([f[t] + run_m - new, torch.exp(i[t] - new), torch.exp(-new)]))
            run_m = new
        want = torch.stack(want).numpy()
        assert np.abs(got[b][:, :H] - want[:, :H]).max() < 3e-5
        assert np.abs(got[b][:, H:3 * H] / want[:, H:] - 1).max() < 3e-5
        assert np.abs(to_np(m[slots[b]]) - run_m.numpy()).max() < 1e-5
        p = got[b][:, 3 * H:]
        v = np.zeros((L, H, dvp))
        v[:, :, :dv], v[:, :, dv] = z[:, 2 * H * dk:W].reshape(L, H, dv).numpy(), 1.0
        rows = np.concatenate([v.reshape(L, -1), z[:, H * dk:2 * H * dk].numpy(), z[:, :H * dk].numpy()], axis=1)
        assert_close(p[:, :rows.shape[1]], rows, dtype, "packed rows")
    assert float((m[1] - 7.0).abs().max()) == 0.0 and float(m[4].abs().max()) == 0.0


MEMORY_SIZES = [(1, 1, 1), (3, 7, 5), (2, 16, 20), (4, 32, 40), (2, 128, 64), (1, 64, 130), (2, 24, 248), (1, 256, 96), (1, 300, 24)]


def memory_run(dtype, H, dk, dv, bi, bf, cap, m, state, w, eps, read_eps):
    """rows [q | k | v | g | i | f] -> the mixer's part between its products: prepare, recurrence, division and gated norm."""
    dvp = (dv + 8) // 8 * 8
    W = 2 * H * dk + 2 * H * dv

    def run(rows, batch):
        rows = rows[0]
        T = rows.shape[0]
        packed = torch.zeros(T, (H * (dvp + 2 * dk) + 7) // 8 * 8, dtype=td_of(dtype), device=DEV)
        ld_, wt, fl = (torch.empty(T, H, device=DEV) for _ in range(3))
        ops.matrix_memory_prepare(rows, 0, H * dk, 2 * H * dk, W, W + H, bi.to(DEV), bf.to(DEV), cap, m, batch, packed, ld_, wt, fl, H, dk, dv, dvp)
        o = torch.full((T, H * dvp), 9.0, device=DEV)
        ops.ssd_scan(packed, H * dvp, H * (dvp + dk), wt, None, None, None, state, batch, o, H, H, dk, dvp, scratch, logd=ld_)
        y = torch.empty(T, H * dv, dtype=td_of(dtype), device=DEV)
        ops.gated_rmsnorm(o, w.to(DEV), eps, rows[:, W - H * dv:W], y, H, dv, sigmoid_gate=True, unit_stride=dvp, divide=(fl, dk ** -0.5, read_eps))
        return y
    return run


@pytest.mark.parametrize("dtype,chunked", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("H,dk,dv", MEMORY_SIZES)
def test_matrix_memory_in_steps_of_any_size(H, dk, dv, dtype, chunked):
    """Three sequences in slots out of order, in steps of 1, 2, 16, 63, 64, 65 tokens and more, token by token and chunk by chunk
    (also mixed).  The norm's eps is large, so the division by max(|n . q|, e^-m) is part of the result, not only its direction."""
    g = torch.Generator().manual_seed(H * dk + dv)
    cap, eps, slots, lens = 5.0, 0.3, [4, 1, 2], [213, 1, 145]
    cuts = [[65, 1, 2, 64, 81], [1], [16, 129]]
    W = 2 * H * dk + 2 * H * dv
    data = []
    for L in lens:
        rows = torch.randn(L, W + 2 * H, generator=g)
        rows[:, :W] = rows[:, :W].to(torch.bfloat16).float()
        rows[:, W + H:] = 2.0 + 2.0 * rows[:, W + H:]
        rows[40::50, W + H:] = -30.0                                             # everything before is forgotten
        rows[90:120, W:W + H] -= 6.0                                             # tokens that barely write: the floor takes over
        data.append([rows])
    bi, bf, w = torch.randn(H, generator=g), torch.randn(H, generator=g), 1.0 + 0.3 * torch.randn(H * dv, generator=g)
    dvp = (dv + 8) // 8 * 8
    state, m = torch.zeros(6, H, dk, dvp, device=DEV), torch.zeros(6, H, device=DEV)
    state[3] = 7.0
    saved, ops.options.ssd_chunked = ops.options.ssd_chunked, chunked
    try:
        got = in_cuts(data, cuts, slots, memory_run(dtype, H, dk, dv, bi, bf, cap, m, state, w, eps, P.READ_EPS))
    finally:
        ops.options.ssd_chunked = saved
    floor_seen = False
    for b, L in enumerate(lens):
        z = data[b][0].double()
        q, k, v = z[:, :H * dk].reshape(L, H, dk) * dk ** -0.5, z[:, H * dk:2 * H * dk].reshape(L, H, dk), z[:, 2 * H * dk:W - H * dv].reshape(L, H, dv)
        i = P.capped(z[:, W:W + H] + bi.double(), cap)
        f = P.log_sigmoid(P.capped(z[:, W + H:] + bf.double(), cap))
        o, (S, n, mm) = P.matrix_memory(q, k, v, i, f)
        ref = (P.unit_rms(o, eps).reshape(L, -1) * w.double() * P.sigmoid(z[:, W - H * dv:W])).numpy()
        tol = 4e-5 if dtype == "float32" else 1e-2
        assert np.abs(got[b] - ref).max() < tol * max(1.0, np.abs(ref).max()), b
        Sg = to_np(state[slots[b]])
        stol = 3e-4 if chunked else 3e-5
        assert np.abs(Sg[:, :, :dv] - S.numpy()).max() < stol * max(1.0, float(S.abs().max())), b
        assert np.abs(Sg[:, :, dv] - n.numpy()).max() < stol * max(1.0, float(n.abs().max())), b
        assert np.abs(Sg[:, :, dv + 1:]).max(initial=0.0) == 0.0 and np.abs(to_np(m[slots[b]]) - mm.numpy()).max() < 1e-5
        floor_seen = floor_seen or L > 100
    assert floor_seen and float((state[3] - 7.0).abs().max()) == 0.0 and float(state[[0, 5]].abs().max()) == 0.0


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("source", [0, 62, 63, 64, 127, 128])
def test_one_write_seen_across_chunk_borders(source, chunked):
    """Nothing is forgotten and every token writes as strongly as the next; one token writes under the direction e1 along which
    every later one reads: its values come back at every later position, and none before it."""
    H, dk, dv, T = 1, 16, 8, 200
    rows = torch.zeros(T, 2 * dk + 2 * dv + 2)
    rows[:, 1] = 4.0                                                   # q = 4 e1, times dk^-1/2: e1
    rows[:, dk] = 1.0                                                  # k = e0 for everyone ...
    rows[source, dk:2 * dk] = torch.eye(dk)[1]                         # ... but the source writes under e1
    rows[:, 2 * dk:2 * dk + dv] = 1.0
    rows[source, 2 * dk:2 * dk + dv] = torch.arange(1.0, 9.0)
    rows[:, 2 * dk + dv:2 * dk + 2 * dv] = 30.0                        # the gate is open
    rows[:, 2 * dk + 2 * dv + 1] = 1e4                                 # forget gate: sigmoid(30)
    state, m = torch.zeros(1, H, dk, 16, device=DEV), torch.zeros(1, H, device=DEV)
    saved, ops.options.ssd_chunked = ops.options.ssd_chunked, chunked
    try:
        y = memory_run("bfloat16", H, dk, dv, torch.zeros(1), torch.zeros(1), 30.0, m, state, torch.ones(dv), 1e6, 0.0)([rows.to(DEV)], step_of([T], [0]))
    finally:
        ops.options.ssd_chunked = saved
    want = torch.zeros(T, dv)
    want[source:] = torch.arange(1.0, 9.0) / 1e3                       # an eps of 1e6: o / 1000, whatever its length
    assert np.abs(to_np(y) - want.numpy()).max() < 1e-4


DELTA_SIZES = [(1, 1, 1, 1), (3, 1, 7, 5), (4, 2, 16, 24), (2, 2, 64, 40), (2, 1, 128, 16), (1, 1, 200, 130), (2, 2, 320, 8)]


@pytest.mark.parametrize("H,G,dk,dv", DELTA_SIZES)
def test_channel_delta_rule_in_steps_of_any_size(H, G, dk, dv):
    """Three sequences in slots out of order, in steps of 1 to 129 tokens; channels that decay at once and channels that never do."""
    g = torch.Generator().manual_seed(H * dk + dv)
    slots, lens, cuts = [4, 1, 2], [213, 1, 145], [[65, 1, 2, 64, 81], [1], [16, 129]]
    data = []
    for L in lens:
        z = torch.randn(L, H * dk, generator=g) * 2.0 - 2.0
        z[:, ::5], z[5::9, 1::7] = -30.0, 30.0
        data.append([torch.randn(L, 2 * G * dk, generator=g), torch.randn(L, H * dv, generator=g), z, torch.randn(L, H, generator=g) * 2.0])
    bias, a_log = torch.randn(H * dk, generator=g), torch.rand(H, generator=g) * 3 - 2
    state = torch.zeros(6, H, dk, dv, device=DEV)
    state[3] = 7.0

    def run(rows, batch):
        qk, v, z, b = rows
        prep = torch.empty(qk.shape[0], H, 5, dk, device=DEV)
        wide = torch.cat([z, v], dim=1)                                          # rows that hold more than z
        ops.channel_delta_prepare(qk, 0, G * dk, wide[:, :H * dk], b, bias.to(DEV), a_log.to(DEV), P.UNIT_EPS, dk ** -0.5, prep, H, G, dk)
        o = torch.full((qk.shape[0], H * dv), 9.0, device=DEV)
        ops.general_delta_scan(prep, v, state, batch, o, H, dk, dv)
        return o
    got = in_cuts(data, cuts, slots, run)
    grp = [h // (H // G) for h in range(H)]
    for b, L in enumerate(lens):
        qk, v, z, bb = (x.double() for x in data[b])
        q, k = (P.unit_vector(qk[:, n * G * dk:(n + 1) * G * dk].reshape(L, G, dk))[:, grp] for n in (0, 1))
        dec = torch.exp(-torch.exp(a_log.double())[:, None] * P.softplus(z + bias.double()).reshape(L, H, dk))
        o, S = P.channel_delta(q * dk ** -0.5, k, v.reshape(L, H, dv), dec, P.sigmoid(bb))
        assert np.abs(got[b].reshape(L, H, dv) - o.numpy()).max() < 3e-5 * max(1.0, float(o.abs().max())), b
        assert np.abs(to_np(state[slots[b]]) - S.numpy()).max() < 3e-5 * max(1.0, float(S.abs().max())), b
    assert float((state[3] - 7.0).abs().max()) == 0.0 and float(state[[0, 5]].abs().max()) == 0.0


@pytest.mark.parametrize("fine,coarse,pad", [(1, 1, 5), (10, 13, 7), (64, 32, 0), (16, 0, 0), (0, 8, 0)])
def test_low_rank_rows_as_two_parts(fine, coarse, pad):
    g = torch.Generator().manual_seed(fine)
    x = torch.randn(9, fine + coarse + 2, generator=g) * 3.0
    out = torch.full((9, 2 * fine + coarse + pad), 9.0, dtype=torch.bfloat16, device=DEV)
    ops.operand_parts(x.to(DEV)[:, :fine + coarse], fine, coarse, out)
    got = to_np(out)
    assert np.abs(got[:, :fine] + got[:, fine:2 * fine] - x[:, :fine].double().numpy()).max(initial=0.0) < 3e-5 * 10
    assert np.array_equal(got[:, 2 * fine:2 * fine + coarse], to_np(x[:, fine:fine + coarse].to(torch.bfloat16)))
    assert np.abs(got[:, 2 * fine + coarse:]).max(initial=0.0) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 16, 24, 16), (2, 2, 12, 10, 6), (3, 1, 8, 40, 0), (4, 4, 16, 16, 8), (5, 1, 7, 3, 2)])
def test_projection_rows_normed_head_by_head_with_blended_values(dtype, H, G, dk, dv, rot):
    g = torch.Generator().manual_seed(dk + dv)
    T, page, eps, lam = 40, 16, 0.02, 0.3
    hd = (max(dk, dv) + 15) // 16 * 16
    cols = H * dk + G * (dk + dv)
    rows, bias = torch.randn(T, cols + 3, generator=g), torch.randn(cols, generator=g)
    wq, wk = 1.0 + 0.3 * torch.randn(dk, generator=g), 1.0 + 0.3 * torch.randn(dk, generator=g)
    first = torch.randn(T, G * dv, generator=g)
    batch, pages = step_of([25, 15], [0, 1], [3, 20]), i32([[2, 0, 5], [1, 4, 3]])
    fq = torch.tensor([500.0 ** (-2.0 * i / rot) for i in range(rot // 2)]).float().to(DEV) if rot else None
    x = rows.double()[:, :cols] + bias.double()
    pos = batch.tok_pos.cpu().tolist()
    qr = P.rotate(P.unit_rms(x[:, :H * dk].reshape(T, H, dk), eps) * wq.double(), pos, 500.0, rot)
    kr = P.rotate(P.unit_rms(x[:, H * dk:(H + G) * dk].reshape(T, G, dk), eps) * wk.double(), pos, 500.0, rot)
    own = x[:, (H + G) * dk:]
    for blend in (False, True):
        kc, vc = (torch.full((6, G, page, hd), 9.0, dtype=td_of(dtype), device=DEV) for _ in range(2))
        q = torch.empty(T, H * hd, dtype=td_of(dtype), device=DEV)
        keep = torch.empty(T, G * dv, device=DEV)
        ops.qkv_rotary_cache(rows.to(DEV)[:, :cols], wq.to(DEV), wk.to(DEV), eps, fq, rot, True, None, batch, pages, q, kc, vc, H, G, dk, dv, hd, page,
                             bias=bias.to(DEV), head_norm=True, blend=(first.to(DEV), lam) if blend else None, keep=keep)
        assert_close(to_np(keep), own.numpy(), "float32", "kept values")
        vr = (P.blend_values(own, first.double(), lam) if blend else own).reshape(T, G, dv)
        want_q = torch.zeros(T, H, hd, dtype=F64)
        want_q[:, :, :dk] = qr
        assert_close(to_np(q), want_q.reshape(T, -1).numpy(), dtype, "queries")
        seqs, tab = batch.tok_seq.cpu().tolist(), pages.cpu().tolist()
        for t in range(T):
            at = (tab[seqs[t]][pos[t] // page], slice(None), pos[t] % page)
            for cache, want, n in ((kc, kr, dk), (vc, vr, dv)):
                row = to_np(cache[at])
                assert_close(row[:, :n], want[t].numpy(), dtype, f"cache row {t}")
                assert np.abs(row[:, n:]).max(initial=0.0) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("units,n,pad", [(1, 24, 1), (3, 7, 1), (4, 64, 8), (2, 512, 8), (2, 516, 8), (3, 2050, 2), (5, 128, 4)])
def test_division_and_gated_norm_of_heads_apart(dtype, units, n, pad):
    """Every path of the kernel: a warp per head, a block per head, rows longer than a block keeps; floors above and below |z|."""
    g = torch.Generator().manual_seed(n)
    T, scale, deps, eps = 6, 0.4, 1e-3, 0.2
    o = torch.randn(T, units, n + pad, generator=g) * 3.0
    floor, gate = torch.rand(T, units, generator=g) * 2.0 + 0.01, torch.randn(T, units * n + 3, generator=g)
    for w_all in (True, False):
        w = 1.0 + 0.3 * torch.randn(units * n if w_all else n, generator=g)
        for div in (True, False):
            y = torch.empty(T, units * n, dtype=td_of(dtype), device=DEV)
            ops.gated_rmsnorm(o.reshape(T, -1).to(DEV), w.to(DEV), eps, gate.to(DEV)[:, :units * n], y, units, n, sigmoid_gate=True, unit_stride=n + pad,
                              divide=(floor.to(DEV), scale, deps) if div else None)
            x = o.double()[:, :, :n]
            if div:
                x = x * scale / (torch.maximum((o.double()[:, :, n] * scale).abs(), floor.double()) + deps)[:, :, None]
            ref = P.unit_rms(x, eps).reshape(T, -1) * (w if w_all else w.repeat(units)).double() * P.sigmoid(gate.double()[:, :units * n])
            assert_close(to_np(y), ref.numpy(), dtype, f"divide {div}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,top,D,F", [(1, 6, 1, 64, 40), (5, 7, 3, 48, 33), (40, 5, 2, 64, 48), (300, 8, 3, 128, 96), (700, 4, 1, 64, 64)])
def test_weights_that_multiply_the_experts_inputs_in_every_kernel(dtype, T, E, top, D, F):
    """One expert's weight in four is tiny and one is 1: it matters on which side of the activation a weight stands."""
    from herbert_rs_b200.parts.swiglu import join_gate_up
    g = torch.Generator().manual_seed(T + E)
    h = (torch.randn(T, D, generator=g) * 2.0).to(torch.bfloat16).float()
    Wg, Wu, Wd = ((torch.randn(E, *s, generator=g) * (1.5 / math.sqrt(s[1]))).to(torch.bfloat16).float() for s in ((F, D), (F, D), (D, F)))
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    wts = torch.rand(T, top, generator=g)
    wts[::4], wts[1::4] = 0.02, 1.0
    ref, wrong = torch.zeros(T, D, dtype=F64), torch.zeros(T, D, dtype=F64)
    for r in range(top):
        for e in range(E):
            at = (ids[:, r] == e).nonzero()[:, 0]
            x, k = h.double()[at], wts.double()[at, r][:, None]
            ref[at] += (P.silu(k * x @ Wg[e].double().T) * (k * x @ Wu[e].double().T)) @ Wd[e].double().T
            wrong[at] += k * ((P.silu(x @ Wg[e].double().T) * (x @ Wu[e].double().T)) @ Wd[e].double().T)
    assert (ref - wrong).abs().max() > 0.1 * wrong.abs().max()
    td = td_of(dtype)
    joined = [join_gate_up(Wg[e].to(td).to(DEV), Wu[e].to(td).to(DEV)) for e in range(E)]
    layout = ops.GATED_GROUPS_OF_8 if joined[0][1] else ops.GATED_HALVES
    up, down, hd_ = torch.stack([j[0] for j in joined]).contiguous(), Wd.to(td).to(DEV), h.to(td).to(DEV)
    idd, wd = ids.to(DEV), wts.to(DEV)
    y = torch.full((T, D), 5.0, device=DEV)
    ops.moe_experts(hd_, up, down, idd, wd, torch.empty(T * top, F, dtype=td, device=DEV), y, ops.ACT_SILU, gated=layout, weigh_input=True)
    assert_close(to_np(y), ref.numpy(), dtype, "few tokens")
    if dtype == "bfloat16" and layout == ops.GATED_GROUPS_OF_8:
        y2 = torch.full((T, D), 5.0, device=DEV)
        ops.moe_experts_grouped(hd_, up, down, idd, wd, y2, ops.ACT_SILU, True, scratch, gated=layout, weigh_input=True)
        assert_close(to_np(y2) - 5.0, ref.numpy(), dtype, "grouped")
        y3 = torch.full((T, D), 5.0, device=DEV)
        ops.moe_experts_tc(hd_, up, down, idd, wd, y3, True, scratch, weigh_input=True)
        ops.check_kernel_errors()
        assert_close(to_np(y3) - 5.0, ref.numpy(), dtype, "tcgen05")
        ops.moe_experts_tc(hd_, up, down, idd, wd, y3, False, scratch)                    # and the other side still is the default
        assert_close(to_np(y3), wrong.numpy(), dtype, "tcgen05, weights on the outputs")


# ---- whole models ---------------------------------------------------------------------------------
ALONE = {
    "attention": ([(U.attention(), None)], {}),
    "attention_blended_ff": ([(U.attention(), U.dense()), (U.attention(), U.dense())], {}),
    "attention_no_rotation": ([(U.attention(heads=1, kv_heads=1, dim=16, vdim=16, rot_dims=0, v_mix=False), U.dense(ff=20))], {}),
    "attention_sharp_heads_of_64": ([(U.attention(heads=4, kv_heads=1, dim=64, vdim=64, sharp=3.0, rot_dims=16), None)] * 2, {"eps": 1e-3}),
    "mlstm": ([(U.mlstm(), None)], {}),
    "mlstm_large_eps_ff": ([(U.mlstm(heads=2, dim=24, vdim=40, cap=15.0), U.dense())], {"eps": 0.05}),
    "mlstm_small_cap": ([(U.mlstm(heads=1, dim=40, vdim=8, cap=0.7), None)], {"logit_scale": 1.0}),
    "delta": ([(U.delta(), None)], {}),
    "delta_one_tap_one_head_ff": ([(U.delta(heads=1, kv_heads=1, dim=24, vdim=40, conv=1, rank=8), U.dense())], {"mult": 1.0}),
    "delta_five_taps": ([(U.delta(heads=6, kv_heads=2, dim=8, vdim=16, conv=5, rank=3), None)], {}),
    "experts": ([(U.mlstm(), U.moe())], {"eps": 0.05}),
    "experts_top_one": ([(U.delta(), U.moe(experts=4, top=1, ff=32, shared=24))], {}),
    "all_experts_none_shared": ([(U.delta(), U.moe(experts=5, top=5, ff=17, shared=0))], {}),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(ALONE))
def test_one_layer_of_each_kind(tmp_path, which, dtype):
    layers, kw = ALONE[which]
    d, pm = U.make(tmp_path / which, layers, seed=len(which), **kw)
    ids = ids_for(np.random.default_rng(1), VOCAB, 70)
    eng = engine_for(d, dtype, max_tokens=512)
    ref = pm.logits(ids).numpy()
    assert_close(replay_whole(eng, ids), ref, dtype, which, plain=pm, ids=ids)
    assert_close(replay_tail_one_by_one(eng, ids, 69), ref, dtype, which + " token by token", plain=pm, ids=ids)


def test_the_residual_stream_after_every_layer(mixed):
    d, pm = mixed
    ids = ids_for(np.random.default_rng(4), VOCAB, 33)
    want = pm.layers(ids)
    eng = engine_for(d, "float32", max_tokens=256)
    got = []
    for b in eng.model.blocks:
        def run(x, batch, cache, inner=b.forward, **kw):
            out = inner(x, batch, cache, **kw)
            got.append(to_np(x))
            return out
        b.forward = run
    replay_whole(eng, ids)
    assert len(got) == len(want) == 6
    for i, (a, b) in enumerate(zip(got, want)):
        assert np.abs(a - b.numpy()).max() < 3e-5 * float(b.abs().max()), i


@pytest.mark.parametrize("dtype", DTYPES)
def test_blended_values_of_three_layers(tmp_path, dtype):
    """The first layer that blends keeps its values for all later ones (not the layer just before), a layer between them that
    does not blend leaves them alone; lambda 1 hands the first layer's values on as they are, lambda 0 none of them."""
    def edit(lams):
        def fn(w):
            for i, v in lams.items():
                w[f"l{i}.mix.vmix"] = torch.tensor(v)
        return fn
    layers = [(U.attention(v_mix=False), None)] + [(U.attention(), None)] * 2 + [(U.attention(heads=2, kv_heads=1, dim=8, vdim=8, v_mix=False), None), (U.attention(), None)]
    ids = ids_for(np.random.default_rng(3), VOCAB, 60)
    refs = []
    for n, lams in enumerate(({2: 0.5, 4: 0.5}, {2: 1.0, 4: 0.0}, {1: 0.9, 2: 0.0, 4: 1.0}, {1: 0.1, 2: 0.0, 4: 1.0})):
        d, pm = U.make(tmp_path / str(n), layers, seed=5, edit=edit(lams))
        eng = engine_for(d, dtype, max_tokens=512)
        refs.append(pm.logits(ids).numpy())
        assert_close(replay_whole(eng, ids), refs[-1], dtype, f"case {n}", plain=pm, ids=ids)
        assert_close(replay_tail_one_by_one(eng, ids, 40), refs[-1], dtype, f"case {n} decoded", plain=pm, ids=ids)
    assert np.abs(refs[0] - refs[1]).max() > 0.3 and np.abs(refs[1] - refs[2]).max() > 0.3 and np.array_equal(refs[2], refs[3])


@pytest.mark.parametrize("dtype", DTYPES)
def test_two_norms_with_statistics_and_a_norm_that_cannot_carry_the_logits_factor(tmp_path, dtype, monkeypatch):
    """The same block with RMS norms (its norms are then kernels of their own), and the factor as a kernel on the logits."""
    from herbert_rs_b200.config.muzasun import MuzasunConfig
    from herbert_rs_b200.config.specs import NormSpec
    from herbert_rs_b200.models import DecoderModel
    from herbert_rs_b200.parts.norm import RMSNorm
    from herbert_rs_b200.weights.loader import fill_model
    monkeypatch.setattr(RMSNorm, "scale_result", lambda self, factor: False)
    monkeypatch.setattr(P, "squash_norm", lambda x, alpha, w, b: P.unit_rms(x, 1e-4) * w)
    cfg = U.config([(U.attention(), U.dense()), (U.mlstm(), None), (U.delta(), U.dense())], logit_scale=0.6)
    spec = MuzasunConfig.from_dict(cfg).model_spec()
    rms = lambda n: None if n is None else NormSpec(n.dim, 1e-4, weight_name=n.weight_name)      # noqa: E731
    blocks = tuple(dataclasses.replace(b, norm1=rms(b.norm1), norm2=rms(b.norm2)) for b in spec.blocks)
    rt = hb.Runtime("cuda", td_of(dtype))
    model = DecoderModel(dataclasses.replace(spec, blocks=blocks, final_norm=rms(spec.final_norm)), rt)
    t = U.weights(cfg, 3)
    fill_model(model, lambda n: t[n], rt)
    assert model.scale_logits
    pm = P.PlainMuzasun(config=cfg, tensors=t)
    ids = ids_for(np.random.default_rng(8), VOCAB, 40)
    eng = hb.Engine(model, max_tokens=512)
    assert_close(replay_whole(eng, ids), pm.logits(ids).numpy(), dtype, "RMS norms", plain=pm, ids=ids)
    assert_close(replay_tail_one_by_one(eng, ids, 20), pm.logits(ids).numpy(), dtype, "RMS norms, decoded", plain=pm, ids=ids)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_against_token_by_token_and_pieces(mixed, dtype):
    d, pm = mixed
    ids = ids_for(np.random.default_rng(2), VOCAB, 150)
    ref = pm.logits(ids).numpy()
    eng = engine_for(d, dtype, max_tokens=1024)
    assert_close(replay_whole(eng, ids), ref, dtype, "whole", plain=pm, ids=ids)
    assert_close(replay_tail_one_by_one(eng, ids, 149), ref, dtype, "one by one", plain=pm, ids=ids)
    for piece in (2, 3, 16, 21, 64, 71):
        s, rows = eng.alloc_slot(), []
        for at in range(0, len(ids), piece):
            rows.append(to_np(eng.step([(s, ids[at:at + piece])], "all")))
        eng.free_slot(s)
        assert_close(np.concatenate(rows), ref, dtype, f"pieces of {piece}", plain=pm, ids=ids)
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batches_in_slots_and_pages_that_were_used_before(mixed, dtype):
    """Three slots serve eight requests: the states, running maxima, convolutions' inputs and pages of a slot's former user must
    not reach its next one (a request of one token reads nothing but zeros)."""
    d, pm = mixed
    rng = np.random.default_rng(3)
    reqs = [ids_for(rng, VOCAB, n) for n in (1, 37, 80, 5, 64, 23, 2, 70)]
    refs = [pm.logits(r).numpy() for r in reqs]
    eng = engine_for(d, dtype, max_tokens=64 * 5, max_slots=3)
    got = replay_batches(eng, reqs, [1, 30, 64, 2, 40, 23, 1, 65], [[0, 1, 2], [3, 4], [5, 6, 7]])
    for i, (g, ref) in enumerate(zip(got, refs)):
        assert_close(g, ref, dtype, f"request {i}", plain=pm, ids=reqs[i])
    assert eng.cache.slots.free_count == 3


def test_a_key_that_is_lost_shows_at_page_borders(tmp_path):
    """Sharp attention in 32-bit over pages of 16 keys: a copy of the model in which one token is replaced differs from that
    token's position on, and the engine follows the right one at every position, whatever page the token lies in."""
    layer = U.attention(heads=2, kv_heads=1, dim=16, vdim=32, sharp=4.0)
    d, pm = U.make(tmp_path / "edge", [(layer, None), (layer, None)], seed=7)
    ids = ids_for(np.random.default_rng(7), VOCAB, 100)
    ref = pm.logits(ids).numpy()
    eng = engine_for(d, "float32", max_tokens=16 * 40, page_size=16)
    s = eng.alloc_slot()
    cut = np.concatenate([to_np(eng.step([(s, ids[a:b])], "all")) for a, b in ((0, 17), (17, 48), (48, 49), (49, 100))])
    eng.free_slot(s)
    runs = {"whole": replay_whole(eng, ids), "decoded": replay_tail_one_by_one(eng, ids, 90), "portions": cut}
    for what, got in runs.items():
        assert np.abs(got - ref).max() < 1e-4 * max(1.0, np.abs(ref).max()), what
    for j in (0, 15, 16, 47, 48):
        other = list(ids)
        other[j] = (ids[j] + 1) % VOCAB
        moved = np.abs(pm.logits(other).numpy() - ref).max(axis=-1)
        assert moved[:j].max(initial=0.0) == 0.0 and (moved[j:] > 1e-3).mean() > 0.5
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_tokens_far_back_stay_in_the_state_and_in_the_keys(tmp_path, dtype):
    """Gates that keep: the first tokens of 400 still move the last logits, and the engine has them whether the prompt came at
    once, in portions, or mostly token by token."""
    def slow(w):
        w["l0.mix.f.b"], w["l1.mix.A_log"] = w["l0.mix.f.b"] * 0 + 9.0, w["l1.mix.A_log"] * 0 - 6.0
        w["l0.mix.i"] *= 0.3
    d, pm = U.make(tmp_path / "far", [(U.mlstm(cap=12.0), None), (U.delta(), None), (U.attention(), None)], seed=21, edit=slow)
    ids = ids_for(np.random.default_rng(6), VOCAB, 400)
    rows = list(range(380, 400))
    ref = pm.logits(ids).numpy()[rows]
    other = pm.logits([(t + 1) % VOCAB for t in ids[:4]] + ids[4:]).numpy()[rows]
    assert np.abs(other - ref).max(axis=-1).min() > 1e-3
    eng = engine_for(d, dtype, max_tokens=2048)
    for cuts in ([400], [7, 200, 193], [300] + [1] * 100):
        s, got, at = eng.alloc_slot(), [], 0
        for n in cuts:
            want = [r - at for r in rows if at <= r < at + n]
            out = eng.step([(s, ids[at:at + n])], [want])
            if want:
                got.append(to_np(out))
            at += n
        eng.free_slot(s)
        assert_close(np.concatenate(got), ref, dtype, f"cuts {cuts[:3]}", plain=pm, ids=ids, rows=rows)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_of_a_sequence(mixed, dtype):
    """Prompts of 1 to 5 tokens (shorter than a convolution's taps, a chunk and a page), alone and as a batch."""
    d, pm = mixed
    rng = np.random.default_rng(8)
    reqs = [ids_for(rng, VOCAB, n) for n in (1, 2, 3, 4, 5)]
    eng = engine_for(d, dtype, max_tokens=512)
    for r in reqs:
        assert_close(replay_whole(eng, r), pm.logits(r).numpy(), dtype, f"{len(r)} tokens", plain=pm, ids=r)
        assert_close(replay_tail_one_by_one(eng, r, len(r) - 1), pm.logits(r).numpy(), dtype, f"{len(r)} tokens one by one", plain=pm, ids=r)
    got = replay_batches(eng, reqs, [1, 1, 2, 4, 3], [[0, 1, 2, 3, 4]])
    for g, r in zip(got, reqs):
        assert_close(g, pm.logits(r).numpy(), dtype, "batch of short prompts", plain=pm, ids=r)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_small_pages(tmp_path, dtype):
    layers = [(U.attention(sharp=2.0), U.dense()), (U.mlstm(), None), (U.delta(), U.moe()), (U.attention(sharp=2.0), None)]
    d, pm = U.make(tmp_path / "long", layers, seed=9)
    ids = ids_for(np.random.default_rng(9), VOCAB, 190)
    ref = pm.logits(ids).numpy()
    page = 16 if dtype == "float32" else 64       # the tensor-core kernels read pages in tiles of 64 keys
    eng = engine_for(d, dtype, max_tokens=page * 20, page_size=page)
    assert_close(replay_tail_one_by_one(eng, ids, 170), ref, dtype, "170 decoded tokens", plain=pm, ids=ids)
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_and_its_continuation(tmp_path, dtype):
    """600 tokens at once and in two portions (several tiles of queries and keys, ten chunks of the recurrence, experts on
    tcgen05), then 24 more; heads of 64 and 128, so that prompts take the tcgen05 attention."""
    layers = [(U.attention(heads=2, kv_heads=1, dim=64, vdim=48, rot_dims=32), U.dense(ff=256)), (U.mlstm(heads=2, dim=64, vdim=128), U.moe(experts=4, top=2, ff=64, shared=64)),
              (U.attention(heads=2, kv_heads=1, dim=128, vdim=48), None), (U.delta(heads=2, kv_heads=1, dim=64, vdim=64, conv=4, rank=16), U.dense(ff=256))]
    d, pm = U.make(tmp_path / "p600", layers, seed=12, width=128)
    ids = ids_for(np.random.default_rng(12), VOCAB, 624)
    rows = [0, 1, 63, 64, 65, 127, 128, 299, 300, 511, 512, 599] + list(range(600, 624))
    ref = pm.logits(ids, torch.float32).double().numpy()[rows]
    eng = engine_for(d, dtype, max_tokens=2048)
    for cuts in ([600], [300, 300]):
        s, got, at = eng.alloc_slot(), [], 0
        for n in cuts + [1] * 24:
            want = [r - at for r in rows if at <= r < at + n]
            out = eng.step([(s, ids[at:at + n])], [want])
            if want:
                got.append(to_np(out))
            at += n
        eng.free_slot(s)
        bound = None if dtype == "bfloat16" else 1e-3 * max(1.0, float(np.abs(ref).max()))
        assert_close(np.concatenate(got), ref, dtype, f"cuts {cuts}", plain=pm, ids=ids, rows=rows, arith=torch.float32, bound=bound)


OTHER = {
    "one_of_everything": ([(U.attention(heads=1, kv_heads=1, dim=2, vdim=1), U.dense(ff=1)), (U.mlstm(heads=1, dim=1, vdim=1), U.moe(experts=1, top=1, ff=1, shared=1)),
                           (U.delta(heads=1, kv_heads=1, dim=1, vdim=1, conv=1, rank=1), None), (U.attention(heads=1, kv_heads=1, dim=1, vdim=1, rot_dims=0), U.dense(ff=8))],
                          {"width": 24, "eps": 0.01}),
    "sizes_no_tile_divides": ([(U.attention(heads=6, kv_heads=3, dim=10, vdim=37, rot_dims=6), U.dense(ff=76)), (U.mlstm(heads=5, dim=11, vdim=27), U.moe(experts=7, top=3, ff=33, shared=21)),
                               (U.delta(heads=6, kv_heads=3, dim=9, vdim=13, conv=7, rank=5), U.dense(ff=33)), (U.attention(heads=9, kv_heads=3, dim=14, vdim=37), None)], {"width": 91}),
    "values_narrower_than_keys": ([(U.attention(heads=3, kv_heads=3, dim=48, vdim=16), U.dense()), (U.attention(heads=6, kv_heads=3, dim=40, vdim=16), None)], {}),
    "many_query_heads_wide_values": ([(U.attention(heads=20, kv_heads=1, dim=8, vdim=72), None), (U.attention(heads=4, kv_heads=2, dim=8, vdim=36), None)], {}),
    "wide_states": ([(U.mlstm(heads=2, dim=264, vdim=24), None), (U.mlstm(heads=1, dim=96, vdim=264), None), (U.delta(heads=1, kv_heads=1, dim=264, vdim=40), None)], {"eps": 1e-3}),
    "heads_of_256_and_320": ([(U.attention(heads=2, kv_heads=1, dim=256, vdim=48, rot_dims=64), None), (U.attention(heads=1, kv_heads=1, dim=320, vdim=48), None)], {}),
    "recurrences_only": ([(U.delta(), U.moe(experts=16, top=4)), (U.mlstm(), U.moe(experts=16, top=4)), (U.mlstm(heads=8, dim=8, vdim=8), U.dense())], {"mult": 0.2, "logit_scale": 4.0}),
    "negative_multiplier_and_alpha": ([(U.mlstm(), U.dense()), (U.attention(), U.dense())], {"mult": -0.7, "logit_scale": -1.0}),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(OTHER))
def test_other_sizes_and_orders(tmp_path, which, dtype):
    layers, kw = OTHER[which]

    def edit(w):
        if which == "negative_multiplier_and_alpha":
            w["l0.norm1.alpha"], w["final.norm.alpha"] = -w["l0.norm1.alpha"], w["final.norm.alpha"] * 0 + 1.0
    d, pm = U.make(tmp_path / which, layers, seed=len(which), edit=edit, **kw)
    ids = ids_for(np.random.default_rng(5), VOCAB, 90)
    ref = pm.logits(ids).numpy()
    eng = engine_for(d, dtype, max_tokens=1024)
    assert_close(replay_whole(eng, ids), ref, dtype, which, plain=pm, ids=ids)
    assert_close(replay_tail_one_by_one(eng, ids, 50), ref, dtype, which + " decoded", plain=pm, ids=ids)
    s = eng.alloc_slot()
    rows = [to_np(eng.step([(s, ids[:37])], "all")), to_np(eng.step([(s, ids[37:39])], "all")), to_np(eng.step([(s, ids[39:])], "all"))]
    eng.free_slot(s)
    assert_close(np.concatenate(rows), ref, dtype, which + " in portions", plain=pm, ids=ids)
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_captured_decode_steps_equal_eager_ones(mixed, dtype):
    d, pm = mixed
    rng = np.random.default_rng(11)
    reqs = [ids_for(rng, VOCAB, n) for n in (40, 70)]
    out = []
    for graphs in (True, False):
        eng = engine_for(d, dtype, max_tokens=1024, use_graphs=graphs)
        out.append(replay_batches(eng, reqs, [10, 33], [[0, 1]]))
        if graphs:
            assert eng.graph_replays > 20
    for a, b in zip(*out):
        assert np.array_equal(a, b)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_any_shape_kernels_agree_with_the_tensor_core_ones(mixed, dtype):
    d, pm = mixed
    ids = ids_for(np.random.default_rng(12), VOCAB, 100)
    ref = pm.logits(ids).numpy()
    ops.options.attention, ops.options.ssd_chunked, ops.options.moe_grouped = "simt", False, False
    try:
        eng = engine_for(d, dtype, max_tokens=512)
        assert_close(replay_tail_one_by_one(eng, ids, 20), ref, dtype, "any-shape kernels", plain=pm, ids=ids)
    finally:
        ops.options.attention, ops.options.ssd_chunked, ops.options.moe_grouped = "auto", True, True


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(mixed, dtype):
    d, pm = mixed
    eng = engine_for(d, dtype, max_tokens=2048)
    rng = np.random.default_rng(15)
    prompts = [ids_for(rng, VOCAB, n) for n in (9, 1, 30, 4, 17)]
    res = hb.generate(eng, prompts, hb.GenerationOptions(max_tokens=10, ignore_eos=True, max_batch=3),
                      hb.SamplingParams(temperature=0.0))
    assert res.stats.batches == 2 and all(len(t) == 10 for t in res.tokens)
    for p, got in zip(prompts, res.tokens):
        ids = list(p)
        for tok in got:
            ref = pm.logits(ids)[-1].numpy()
            margin = 1e-4 * max(1.0, np.abs(ref).max()) if dtype == "float32" else 2 * bound_for(pm, ids, dtype, ref)
            assert ref.max() - ref[tok] <= margin
            ids.append(tok)
    eng.cache.check()
    assert eng.cache.slots.free_count == eng.cache.num_slots


def test_random_weights_from_the_configuration(tmp_path):
    cfg = U.config([(U.attention(), U.dense()), (U.mlstm(), None), (U.delta(rank=12), U.moe(experts=4, top=4)), (U.attention(), None)])
    hb.write_random_model(cfg, str(tmp_path), seed=1)
    pm = P.PlainMuzasun(str(tmp_path))
    assert set(pm.W) == set(U.weights(cfg)) and tuple(pm.W["l2.mix.a1"].shape) == (12, 64)
    ids = ids_for(np.random.default_rng(1), VOCAB, 50)
    eng = engine_for(str(tmp_path), "float32", max_tokens=256)
    ref = pm.logits(ids).numpy()
    own = np.abs(pm.logits(ids, torch.float32).double().numpy() - ref).max()
    assert np.abs(replay_whole(eng, ids) - ref).max() < max(1e-4 * max(1.0, np.abs(ref).max()), 5 * own)


def test_command_line_trace_replay_and_prompts_in_pieces(mixed, tmp_path, capsys):
    """The design through the library's other entry points: the command line, `bin/trace_run`, and the generation loop with
    prompts fed in pieces and sampling on the device."""
    import json
    import os
    import subprocess
    import sys
    from herbert_rs_b200 import cli
    d, pm = mixed
    rng = np.random.default_rng(21)
    a, b = ids_for(rng, VOCAB, 40), ids_for(rng, VOCAB, 7)
    assert cli.main(["--model", d, "--prompt-ids", ",".join(map(str, a)), "--prompt-ids", ",".join(map(str, b)),
                     "--max-tokens", "5", "--temperature", "0", "--ignore-eos", "--backend", "cuda-fp32"]) == 0
    lines = capsys.readouterr().out.strip().splitlines()
    assert len(lines) == 2
    ids = list(a)
    for tok in map(int, lines[0].split(",")):
        ref = pm.logits(ids)[-1].numpy()
        assert ref.max() - ref[tok] <= 1e-4 * max(1.0, np.abs(ref).max())
        ids.append(tok)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:6], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": [0]}, {"id": "b", "tokens": b[6:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:32], "want": [0]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype in DTYPES:
        out = tmp_path / ("trace_" + dtype)
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True)
        assert r.returncode == 0 and [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
        ra, rb = pm.logits(a).numpy(), pm.logits(b).numpy()
        read = lambda n, rows: np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(rows, VOCAB).astype(np.float64)      # noqa: E731
        assert_close(read(0, 2), ra[[0, 29]], dtype, "trace step 0", plain=pm, ids=a, rows=[0, 29])
        assert_close(read(1, 2)[:1], ra[[30]], dtype, "trace step 1 a", plain=pm, ids=a, rows=[30])
        assert_close(read(1, 2)[1:], rb[[6]], dtype, "trace step 1 b", plain=pm, ids=b, rows=[6])
        assert_close(read(2, 1), ra[[31]], dtype, "trace step 2", plain=pm, ids=a, rows=[31])
    outs = []
    for piece in (None, 16):
        eng = engine_for(d, "float32", max_tokens=1024)
        res = hb.generate(eng, [a, b], hb.GenerationOptions(max_tokens=8, ignore_eos=True, prefill_chunk_size=piece),
                          hb.SamplingParams(temperature=0.8, top_k=20, top_p=0.95, seed=5))
        outs.append(res.tokens)
    assert outs[0] == outs[1]
