"""The Putazen design in the engine against the plain implementation (`plain_putazen.py`): every mechanism alone, prompts
against decoding, prompts in pieces, unequal batches, slots and pages that are used again, far keys and chunk borders, the
first tokens, long decoding, looped layers, other sizes, greedy generation through the library's entry points."""
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import herbert_rs_b200 as hb
import plain_putazen as P
import putazen_util as U
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
    """gpu_util's comparison, with steadier bounds for whole models.  A layer norm over a mixture of copies, or the norm of a
    difference of two maps, brings a small vector to full size, so at single positions any rounding is amplified by a factor
    that depends on its direction.  bfloat16: the bound is three times what bfloat16 storage between kernels does to the plain
    implementation at most, over all rows of the request and over one fixed 64-token request of the model; at most one row
    in fifty (or one row) may lie above it, and none above one and a half times it.  float32: the usual bound, or six times
    what float32 arithmetic does to the plain implementation over the same rows, whichever is larger."""
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


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    """All three mixers, two of them in a loop of three passes; a partly rotated attention; a layer without a feed-forward;
    three copies of the stream."""
    layers = [(U.attention(heads=4, kv_heads=2, dim=16, vdim=24, rot_dims=8), U.dense()),
              (U.mamba(heads=4, vdim=16, state=24, groups=2, norm_groups=2, conv=3), U.dense(ff=72)),
              (U.latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=32), None),
              (U.attention(heads=2, kv_heads=2, dim=8, vdim=16), U.dense())]
    return U.make(tmp_path_factory.mktemp("putazen_mixed"), layers, seed=13, loop=(1, 3, 3))


# ---- each mechanism alone -------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,dim", [(1, 48), (2, 1000), (3, 47), (4, 2048), (6, 96), (7, 336), (16, 260)])
def test_streams_mixed_and_normed(dtype, n, dim):
    g = torch.Generator().manual_seed(n * dim)
    T = 5
    X, y = torch.randn(n, T, dim, generator=g) * 2.0, torch.randn(T, dim + 4, generator=g)
    M, b, a = torch.randn(n, n, generator=g), torch.randn(n, generator=g), torch.randn(n, generator=g)
    w, nb = 1.0 + 0.2 * torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    ref = P.stream_out(X.double(), y.double()[:, :dim], M.double(), b.double())
    wd, nbd = w.to(DEV), nb.to(DEV)
    for with_h in (True, False):
        x = X.transpose(0, 1).contiguous().to(DEV)
        h = torch.empty(T, dim, dtype=td_of(dtype), device=DEV) if with_h else None
        ops.streams_join(x, y.to(DEV)[:, :dim], M.to(DEV), b.to(DEV), in_w=a.to(DEV) if with_h else None,
                         norm=(wd, nbd, 1e-5, False) if with_h else None, h=h)
        assert_close(to_np(x), ref.transpose(0, 1).numpy(), "float32", "copies")
        if with_h:
            assert_close(to_np(h), P.layer_norm(P.stream_in(ref, a.double()), w.double(), nb.double(), 1e-5).numpy(), dtype, "input")
    # nothing joins: the rows asked for, their plain sum, and an RMS norm without a bias
    x, rows = X.transpose(0, 1).contiguous().to(DEV), [4, 0, 4]
    h = torch.empty(3, dim, dtype=td_of(dtype), device=DEV)
    ops.streams_join(x, norm=(wd, nbd, 1e-5, False), h=h, rows=i32(rows))
    assert_close(to_np(h), P.layer_norm(X.double().sum(0)[rows], w.double(), nb.double(), 1e-5).numpy(), dtype, "sum of the copies")
    h = torch.empty(T, dim, dtype=td_of(dtype), device=DEV)
    ops.streams_join(x, in_w=a.to(DEV), norm=(wd, None, 3e-5, True), h=h)
    assert_close(to_np(h), (P.unit_rms(P.stream_in(X.double(), a.double()), 3e-5) * w.double()).numpy(), dtype, "RMS norm")
    assert torch.equal(x.cpu(), X.transpose(0, 1))


@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_norm_with_a_bias_and_an_embedding_of_several_copies(dtype):
    g = torch.Generator().manual_seed(1)
    x, w, b = torch.randn(6, 72, generator=g) * 3.0 + 1.0, 1.0 + 0.2 * torch.randn(72, generator=g), torch.randn(72, generator=g)
    out = torch.empty(2, 72, dtype=td_of(dtype), device=DEV)
    ops.layernorm(x.to(DEV), w.to(DEV), out, 1e-5, i32([5, 1]), bias=b.to(DEV))
    assert_close(to_np(out), P.layer_norm(x.double()[[5, 1]], w.double(), b.double(), 1e-5).numpy(), dtype, "layer norm with a bias")
    table = torch.randn(11, 40, generator=g).to(td_of(dtype))
    e = torch.empty(4, 3, 40, device=DEV)
    ops.embed(table.to(DEV), i32([3, 0, 10, 3]), e, 2.5)
    assert_close(to_np(e), (table.double()[[3, 0, 10, 3]] * 2.5)[:, None].expand(4, 3, 40).numpy(), "float32", "copies of the embedding")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 9, 17])
def test_convolution_with_a_bias_continues_from_its_state(dtype, taps):
    g = torch.Generator().manual_seed(taps)
    C, slots, lens, cuts = 150, [2, 0, 3], [90, 1, 40], [[1, 2, 3, 84], [1], [33, 7]]
    data = [torch.randn(L, C + 5, generator=g) for L in lens]
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    state = torch.zeros(5, taps - 1, C, device=DEV) if taps > 1 else None
    done, got = [0] * 3, [[] for _ in lens]
    for r in range(4):
        live = [i for i in range(3) if r < len(cuts[i])]
        cnt = [cuts[i][r] for i in live]
        rows = torch.cat([data[i][done[i]:done[i] + c] for i, c in zip(live, cnt)]).to(DEV)
        out = torch.zeros(rows.shape[0], C + 2, dtype=td_of(dtype), device=DEV)
        ops.short_conv(rows[:, :C], w.to(DEV), state, step_of(cnt, [slots[i] for i in live], [done[i] for i in live]), out, silu=True, bias=b.to(DEV))
        o = 0
        for i, c in zip(live, cnt):
            got[i].append(to_np(out[o:o + c, :C])); o += c; done[i] += c
    for i in range(3):
        ref = P.silu(P.causal_conv(data[i].double()[:, :C], w.double(), b.double()))
        assert_close(np.concatenate(got[i]), ref.numpy(), dtype, f"sequence {i}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("parts,n", [(1, 64), (2, 48), (3, 7), (4, 1024), (2, 5000)])
def test_the_gate_before_the_norm_in_parts(dtype, parts, n):
    g = torch.Generator().manual_seed(n)
    T, W = 7, parts * n
    y, z, w = torch.randn(T, W, generator=g) * 3.0, torch.randn(T, W + 8, generator=g) * 2.0, 1.0 + 0.3 * torch.randn(W, generator=g)
    out = torch.empty(T, W, dtype=td_of(dtype), device=DEV)
    ops.gated_rmsnorm(y.to(DEV), w.to(DEV), 1e-5, z.to(DEV)[:, :W], out, parts, n, gate_first=True)
    assert_close(to_np(out), P.gated_group_norm(y.double(), z.double()[:, :W], w.double(), parts, 1e-5).numpy(), dtype, "gate, norm")


SSD_SIZES = [(4, 2, 24, 16), (6, 3, 56, 24), (2, 1, 128, 64), (8, 4, 16, 8), (3, 3, 7, 5), (2, 2, 130, 12), (1, 1, 256, 128), (2, 1, 40, 150), (4, 4, 5, 100)]


def _ssd_inputs(g, T, H, G, N, dv, dtype, extreme):
    C = H * dv + 2 * G * N
    xbc = torch.zeros(T, (C + 7) // 8 * 8)
    xbc[:, :C] = torch.randn(T, C, generator=g)
    xbc = xbc.to(td_of(dtype))
    raw = torch.randn(T, H + 3, generator=g)
    if extreme:                       # step sizes near 0 and large ones: nothing forgotten, everything forgotten
        raw[::7, 0], raw[3::11, 0] = -30.0, 12.0
    return xbc, raw


def _ssd_plain(xbc, raw, bias, a_log, dskip, H, G, N, dv, S=None):
    d, T = xbc.double(), xbc.shape[0]
    x, B, C = d[:, :H * dv], d[:, H * dv:H * dv + G * N], d[:, H * dv + G * N:H * dv + 2 * G * N]
    dt = P.softplus(raw.double()[:, :H] + bias.double())
    return P.state_space_scan(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), dt, torch.exp(a_log.double()), dskip.double(), S)


@pytest.mark.parametrize("dtype,chunked", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("H,G,N,dv", SSD_SIZES)
def test_state_space_recurrence_in_steps_of_any_size(H, G, N, dv, dtype, chunked):
    """Three sequences in slots out of order, in steps of 1, 2, 16, 63, 64, 65 tokens and more: every step continues from the
    slot's state, token by token and chunk by chunk (also mixed); step sizes that keep everything and that keep nothing."""
    g = torch.Generator().manual_seed(H * N + dv)
    slots, lens = [4, 1, 2], [213, 1, 145]
    cuts = [[65, 1, 2, 64, 81], [1], [16, 129]]
    data = [_ssd_inputs(g, L, H, G, N, dv, dtype, True) for L in lens]
    bias, a_log, dskip = torch.randn(H, generator=g), torch.rand(H, generator=g) * 3 - 2, torch.randn(H, generator=g)
    state = torch.zeros(6, H, N, dv, device=DEV)
    state[3] = 7.0                                                              # a slot nobody uses stays as it is
    done, got = [0, 0, 0], [[] for _ in lens]
    saved, ops.options.ssd_chunked = ops.options.ssd_chunked, chunked
    try:
        for r in range(5):
            live = [b for b in range(3) if r < len(cuts[b])]
            cnt = [cuts[b][r] for b in live]
            xbc = torch.cat([data[b][0][done[b]:done[b] + c] for b, c in zip(live, cnt)]).to(DEV)
            raw = torch.cat([data[b][1][done[b]:done[b] + c] for b, c in zip(live, cnt)]).to(DEV)
            out = torch.full((xbc.shape[0], H * dv), 9.0, device=DEV)
            ops.ssd_scan(xbc, H * dv, H * dv + G * N, raw[:, :H], bias.to(DEV), a_log.to(DEV), dskip.to(DEV), state,
                         step_of(cnt, [slots[b] for b in live], [done[b] for b in live]), out, H, G, N, dv, scratch)
            o = 0
            for b, c in zip(live, cnt):
                got[b].append(to_np(out[o:o + c])); o += c; done[b] += c
    finally:
        ops.options.ssd_chunked = saved
    tol = 2e-4 if chunked else 2e-5            # products of 16-bit parts against float sums
    for b, L in enumerate(lens):
        ref, S = _ssd_plain(*data[b], bias, a_log, dskip, H, G, N, dv)
        assert np.abs(np.concatenate(got[b]).reshape(L, H, dv) - ref.numpy()).max() < tol * max(1.0, float(ref.abs().max())), b
        assert np.abs(to_np(state[slots[b]]) - S.numpy()).max() < tol * max(1.0, float(S.abs().max())), b
    assert float((state[3] - 7.0).abs().max()) == 0.0 and float(state[[0, 5]].abs().max()) == 0.0


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("source", [0, 62, 63, 64, 127, 128])
def test_one_token_seen_across_chunk_borders(source, chunked):
    """A single token writes under the direction e1, every later token reads along it, nothing decays: its x comes back
    at every later position, none before it, and the tokens' own writes stay out of it."""
    H, N, dv, T = 1, 16, 8, 200
    xbc = torch.zeros(T, H * dv + 2 * N)
    xbc[:, :dv] = 1.0
    xbc[source, :dv] = torch.arange(1.0, 9.0)
    xbc[:, dv] = 1.0                                        # B = e0 for everyone ...
    xbc[source, dv:dv + N] = torch.eye(N)[1]                # ... but the source writes under e1
    xbc[:, dv + N + 1] = 1.0                                # C = e1
    raw = torch.full((T, 1), math.log(math.e - 1.0))        # softplus = 1
    state = torch.zeros(1, H, N, dv, device=DEV)
    out = torch.empty(T, dv, device=DEV)
    saved, ops.options.ssd_chunked = ops.options.ssd_chunked, chunked
    try:
        ops.ssd_scan(xbc.to(torch.bfloat16).to(DEV), dv, dv + N, raw.to(DEV), torch.zeros(1, device=DEV), torch.full((1,), -40.0, device=DEV),
                     torch.zeros(1, device=DEV), state, step_of([T], [0]), out, H, 1, N, dv, scratch)
    finally:
        ops.options.ssd_chunked = saved
    want = torch.zeros(T, dv)
    want[source:] = torch.arange(1.0, 9.0)
    assert np.abs(to_np(out) - want.numpy()).max() < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,rot,halves,scaled", [(4, 2, 16, 32, 16, True, True), (2, 2, 12, 10, 6, True, True), (3, 1, 8, 40, 0, True, False),
                                                         (4, 4, 16, 16, 8, False, False)])
def test_projection_rows_with_bias_two_maps_and_scaled_angles(dtype, H, G, dk, dv, rot, halves, scaled):
    g = torch.Generator().manual_seed(dk + dv)
    T, maps, page = 40, 2, 16
    hd = max(maps * dk, dv) + 4                                   # a cache head wider than both
    cols = H * maps * dk + G * (maps * dk + dv)
    rows, bias = torch.randn(T, cols + 3, generator=g), torch.randn(cols, generator=g)
    f, m = P.frequencies(rot, 500.0, {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 1.0} if scaled else None) if rot else ([], 1.0)
    batch = step_of([25, 15], [0, 1], [3, 20])
    pages = i32([[2, 0, 5], [1, 4, 3]])
    kc, vc = (torch.full((6, G, page, hd), 9.0, dtype=td_of(dtype), device=DEV) for _ in range(2))
    q = torch.empty(T, H * maps * hd, dtype=td_of(dtype), device=DEV)
    ops.qkv_rotary_cache(rows.to(DEV)[:, :cols], None, None, 0.0, torch.tensor(f).float().to(DEV) if rot else None, rot, halves, None, batch, pages,
                         q, kc, vc, H, G, dk, dv, hd, page, bias=bias.to(DEV), mscale=m, maps=maps)
    x = rows.double()[:, :cols] + bias.double()
    pos = batch.tok_pos.cpu().tolist()
    qr = P.rotate(x[:, :H * maps * dk].reshape(T, H * maps, dk), pos, f, m, rot, not halves)
    kr = P.rotate(x[:, H * maps * dk:(H + G) * maps * dk].reshape(T, G * maps, dk), pos, f, m, rot, not halves).reshape(T, G, maps * dk)
    vr = x[:, (H + G) * maps * dk:].reshape(T, G, dv)
    want_q = torch.zeros(T, H * maps, hd, dtype=F64)
    for i in range(H * maps):
        want_q[:, i, (i % maps) * dk:(i % maps + 1) * dk] = qr[:, i]
    assert_close(to_np(q), want_q.reshape(T, -1).numpy(), dtype, "queries")
    seqs, tab = batch.tok_seq.cpu().tolist(), pages.cpu().tolist()
    for t in range(T):
        at = (tab[seqs[t]][pos[t] // page], slice(None), pos[t] % page)
        for cache, want, n in ((kc, kr, maps * dk), (vc, vr, dv)):
            row = to_np(cache[at])
            assert_close(row[:, :n], want[t].numpy(), dtype, f"cache row {t}")
            assert np.abs(row[:, n:]).max() == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("halves", [True, False])
def test_latent_rows_rotated_in_either_layout(dtype, halves):
    g = torch.Generator().manual_seed(3)
    T, rank, rot, H, dn, page = 20, 24, 10, 3, 6, 16
    f, _ = P.frequencies(rot, 300.0)
    fd = torch.tensor(f).float().to(DEV)
    kv, w = torch.randn(T, rank + rot + 2, generator=g), 1.0 + 0.2 * torch.randn(rank, generator=g)
    batch, pages = step_of([T], [0], [7]), i32([[1, 0]])
    cache = torch.zeros(2, 1, page, rank + rot, dtype=td_of(dtype), device=DEV)
    ops.latent_kv_store(kv.to(DEV), w.to(DEV), 1e-5, fd, 1.0, rank, rot, batch.tok_seq, batch.tok_pos, pages, cache, page, halves=halves)
    pos = list(range(7, 7 + T))
    want = torch.cat([P.unit_rms(kv.double()[:, :rank], 1e-5) * w.double(),
                      P.rotate(kv.double()[:, rank:rank + rot], pos, f, 1.0, rot, not halves)], dim=-1)
    got = np.stack([to_np(cache[1 - p // page, 0, p % page]) for p in pos])
    assert_close(got, want.numpy(), dtype, "cached rows")
    q = torch.randn(T, H * (dn + rot), generator=g)
    out = torch.zeros(T, H * (rank + rot), device=DEV)
    ops.rotate_heads(q.to(DEV), dn + rot, dn, out, rank + rot, rank, fd, 1.0, batch.tok_pos, H, rot, scale=0.3, halves=halves)
    want = P.rotate(q.double().view(T, H, dn + rot)[:, :, dn:], pos, f, 1.0, rot, not halves) * 0.3
    assert_close(to_np(out.view(T, H, rank + rot)[:, :, rank:]), want.numpy(), "float32", "rotated parts of the queries")


@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 32, 64), (2, 1, 8, 16), (8, 2, 64, 128), (2, 2, 24, 40), (6, 3, 40, 80), (2, 1, 64, 100), (4, 1, 20, 50), (4, 2, 120, 200), (2, 1, 150, 40)])
def test_difference_of_two_maps_in_every_attention_kernel(H, G, dk, dv):
    """One sequence of 300 cached keys in pages that are not in order; the queries of the last 150 positions as a prompt's
    portion and the last one alone.  Scaled queries make one far key, keys at page borders and the query's own key stand
    out, some in the first map, some in the second."""
    g = torch.Generator().manual_seed(dk + dv)
    T, page, diff, lam, eps = 300, 64, 0.35, 0.8, 1e-5
    hd = (max(2 * dk, dv) + 15) // 16 * 16
    order = [3, 0, 4, 1, 2]
    q, k, v = (torch.randn(T, n, d, generator=g).to(torch.bfloat16).float() for n, d in ((2 * H, dk), (2 * G, dk), (G, dv)))
    scale, last = 1.0 / math.sqrt(dk), T - 1
    for j, m in ((3, 0), (63, 1), (64, 0), (last, 1), (255, 1)):
        k[j, m] = (q[last, m] * 3.0).to(torch.bfloat16).float()
    a = torch.stack([P.softmax_attention(q[:, i].double(), k[:, (i // 2 // (H // G)) * 2 + i % 2].double(), v[:, i // 2 // (H // G)].double(), scale)
                     for i in range(2 * H)], dim=1)
    ref = P.combine_maps(a[:, 0::2], a[:, 1::2], lam, diff, eps).reshape(T, H * dv)
    # it shows when the second map is left out, and when a far key is lost
    assert (P.combine_maps(a[:, 0::2], 0 * a[:, 1::2], lam, diff, eps).reshape(T, H * dv)[last] - ref[last]).abs().max() > 0.1
    rows = list(range(T - 150, T))
    for dtype in DTYPES:
        kc, vc = (torch.zeros(5, G, page, hd) for _ in range(2))
        qq = torch.zeros(T, 2 * H, hd)
        for j in range(T):
            kc[order[j // page], :, j % page, :2 * dk] = k[j].reshape(G, 2 * dk)
            vc[order[j // page], :, j % page, :dv] = v[j]
        for i in range(2 * H):
            qq[:, i, (i % 2) * dk:(i % 2 + 1) * dk] = q[:, i]
        kc, vc = kc.to(td_of(dtype)).to(DEV), vc.to(td_of(dtype)).to(DEV)
        qd, pages = qq.view(T, 2 * H * hd).to(td_of(dtype)).to(DEV), i32([order])
        for kern in ["simt"] + (["auto", "mma"] if dtype == "bfloat16" else []):      # "auto": tcgen05 for prompts of heads of 64 / 128
            ops.options.attention = "simt" if kern == "simt" else "auto"
            ops.options.prefill_attention = "mma" if kern == "mma" else "tcgen05"
            try:
                for n in (150, 1):
                    out = torch.empty(n, H * dv, dtype=td_of(dtype), device=DEV)
                    ops.attention(qd[T - n:], 2 * H * hd, out, kc, vc, step_of([n], [0], [T - n]), 2 * H, G, hd, page, scale, None, pages,
                                  scratch=scratch, difference=(lam, 1.0 - diff, eps, dv))
                    want = ref[rows if n > 1 else [last]].numpy()
                    bound = 2e-5 if dtype == "float32" else 2.5e-2
                    assert np.abs(to_np(out) - want).max() < bound * max(1.0, np.abs(want).max()), (dtype, kern, n)
                ops.check_kernel_errors()
            finally:
                ops.options.attention, ops.options.prefill_attention = "auto", "tcgen05"


def test_difference_over_an_unequal_batch_with_prompts_of_several_tiles():
    """Three prompts of 1, 130 and 300 tokens in one step, two of them after cached keys: the difference is taken row by row
    where a tile of queries is not full and where a sequence has none."""
    g = torch.Generator().manual_seed(11)
    H, G, dk, dv, page, hd, diff, lam, eps = 4, 2, 64, 128, 64, 128, 0.2, 0.6, 1e-5
    lens, pos0 = [1, 130, 300], [70, 0, 40]
    tot = [n + p for n, p in zip(lens, pos0)]
    q = [torch.randn(t, 2 * H, dk, generator=g).to(torch.bfloat16) for t in tot]
    k = [torch.randn(t, 2 * G, dk, generator=g).to(torch.bfloat16) for t in tot]
    v = [torch.randn(t, G, dv, generator=g).to(torch.bfloat16) for t in tot]
    width = -(-max(tot) // page)
    pages = torch.randperm(3 * width, generator=g).view(3, width)
    kc, vc = (torch.zeros(3 * width, G, page, hd, dtype=torch.bfloat16) for _ in range(2))
    for b in range(3):
        for j in range(tot[b]):
            kc[pages[b, j // page], :, j % page] = k[b][j].reshape(G, 2 * dk)
            vc[pages[b, j // page], :, j % page] = v[b][j]
    qq = torch.cat([q[b][pos0[b]:] for b in range(3)])
    wide = torch.zeros(len(qq), 2 * H, hd, dtype=torch.bfloat16)
    wide[:, 0::2, :dk], wide[:, 1::2, dk:] = qq[:, 0::2], qq[:, 1::2]
    out = torch.empty(len(qq), H * dv, dtype=torch.bfloat16, device=DEV)
    ops.attention(wide.view(len(qq), -1).to(DEV), 2 * H * hd, out, kc.to(DEV), vc.to(DEV), step_of(lens, [0, 1, 2], pos0), 2 * H, G, hd, page, dk ** -0.5,
                  None, i32(pages.tolist()), scratch=scratch, difference=(lam, 1.0 - diff, eps, dv))
    ops.check_kernel_errors()
    o = 0
    for b in range(3):
        a = torch.stack([P.softmax_attention(q[b][:, i].double(), k[b][:, (i // 4) * 2 + i % 2].double(), v[b][:, i // 4].double(), dk ** -0.5)
                         for i in range(2 * H)], dim=1)
        ref = P.combine_maps(a[:, 0::2], a[:, 1::2], lam, diff, eps).reshape(tot[b], H * dv)[pos0[b]:].numpy()
        assert np.abs(to_np(out[o:o + lens[b]]) - ref).max() < 2.5e-2 * max(1.0, np.abs(ref).max()), b
        o += lens[b]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,F,D", [(1, 96, 64), (8, 4096, 128), (13, 40, 72), (30, 4096, 512), (64, 96, 256), (70, 88, 64), (300, 1024, 512), (500, 384, 256),
                                   (5, 20, 36), (90, 20, 36)])
def test_clamped_gated_product_in_every_kernel(dtype, M, F, D):
    g = torch.Generator().manual_seed(M + F)
    limit = 1.25
    h = torch.randn(M, D, generator=g).to(torch.bfloat16).float()
    Wg, Wu = ((torch.randn(F, D, generator=g) * (2.0 / math.sqrt(D))).to(torch.bfloat16).float() for _ in range(2))
    gate, up = h.double() @ Wg.double().T, h.double() @ Wu.double().T
    assert gate.max() > limit and up.min() < -limit and up.max() > limit           # every clamp is reached
    ref = P.clamped_glu(gate, up, limit).numpy()
    from herbert_rs_b200.parts.swiglu import join_gate_up
    wgu, inter = join_gate_up(Wg.to(td_of(dtype)).to(DEV), Wu.to(td_of(dtype)).to(DEV))
    hd_ = h.to(td_of(dtype)).to(DEV)
    out = torch.empty(M, F, dtype=td_of(dtype), device=DEV)
    ops.gemm_swiglu(hd_, wgu, out, inter, scratch, limit)
    assert_close(to_np(out), ref, dtype, "chosen kernel")
    if dtype == "bfloat16" and inter == 8:
        kernels = [ops.gemm_tcgen05] + ([ops.gemm_skinny, ops.gemm_stream] if M <= 64 else [])
        for fn in kernels:
            out.zero_()
            fn(hd_, wgu, out, ops.EPI_SWIGLU, limit)
            ops.check_kernel_errors()
            assert_close(to_np(out), ref, dtype, fn.__name__)


# ---- whole models ---------------------------------------------------------------------------------
ALONE = {
    "attention": ([(U.attention(), None)], {}),
    "attention_ff_no_scaling": ([(U.attention(heads=2, kv_heads=1, dim=8, vdim=24, scaling=None, diff=0.0), U.dense())], {}),
    "attention_no_rotation": ([(U.attention(rot_dims=0, heads=1, kv_heads=1, dim=16, vdim=16), U.dense(ff=20, limit=0.5))], {"streams": 1}),
    "attention_sharp_heads_of_64": ([(U.attention(heads=4, kv_heads=1, dim=32, vdim=64, sharp=2.0, rot_dims=16), None)], {"streams": 2}),
    "latent": ([(U.latent(), None)], {}),
    "latent_no_rotation": ([(U.latent(heads=3, rot_dim=0, dim=20, vdim=12, kv_rank=24), U.dense())], {"streams": 5}),
    "latent_one_head": ([(U.latent(heads=1, dim=8, rot_dim=16, vdim=40, kv_rank=64, sharp=2.0), None)], {}),
    "mamba": ([(U.mamba(), None)], {}),
    "mamba_one_group_ff": ([(U.mamba(heads=3, vdim=20, state=16, groups=1, norm_groups=1, conv=4), U.dense())], {"streams": 4}),
    "mamba_conv_of_one": ([(U.mamba(heads=2, vdim=8, state=64, groups=2, norm_groups=4, conv=1), None)], {}),
    "looped": ([(U.mamba(), None), (U.attention(), None)], {"loop": (0, 2, 2)}),
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


def test_the_residual_stream_after_every_layer_run(mixed):
    d, pm = mixed
    ids = ids_for(np.random.default_rng(4), VOCAB, 33)
    want = pm.layers(ids)
    eng = engine_for(d, "float32", max_tokens=256)
    got = []
    for b in eng.model.blocks:
        def run(x, batch, cache, inner=b.forward, **kw):
            out = inner(x, batch, cache, **kw)
            got.append(to_np(x.sum(1)))
            return out
        b.forward = run
    replay_whole(eng, ids)
    assert len(got) == len(want) == 1 + 2 * 3 + 1
    for i, (a, b) in enumerate(zip(got, want)):
        assert np.abs(a - b.numpy()).max() < 3e-5 * float(b.abs().max()), i


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
    """Three slots serve eight requests: the states, the convolutions' inputs and the pages of a slot's former user, one set
    per pass of the loop, must not reach its next one (a request of one token reads nothing but zeros)."""
    d, pm = mixed
    rng = np.random.default_rng(3)
    reqs = [ids_for(rng, VOCAB, n) for n in (1, 37, 80, 5, 64, 23, 2, 70)]
    refs = [pm.logits(r).numpy() for r in reqs]
    eng = engine_for(d, dtype, max_tokens=64 * 5, max_slots=3)
    got = replay_batches(eng, reqs, [1, 30, 64, 2, 40, 23, 1, 65], [[0, 1, 2], [3, 4], [5, 6, 7]])
    for i, (g, ref) in enumerate(zip(got, refs)):
        assert_close(g, ref, dtype, f"request {i}", plain=pm, ids=reqs[i])
    assert eng.cache.slots.free_count == 3


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_a_key_that_is_lost_shows_at_page_borders(tmp_path, kind):
    """Sharp attention in 32-bit over pages of 16 keys: a copy of the model in which one token is replaced differs from that
    token's position on, and the engine follows the right one at every position, whatever page the token lies in."""
    layer = U.attention(heads=2, kv_heads=1, dim=16, vdim=32, sharp=4.0) if kind == "attention" else U.latent(heads=2, sharp=4.0)
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
    """Slow decay (small step sizes): the first tokens of 400 still move the last logits, and the engine has them whether the
    prompt came at once, in portions, or mostly token by token."""
    def slow(w):
        w["l0.mix.dt_bias"], w["l0.mix.A_log"] = w["l0.mix.dt_bias"] * 0 - 2.0, w["l0.mix.A_log"] * 0 - 5.0
        w["l0.mix.in"][-4:] *= 0.1
    d, pm = U.make(tmp_path / "far", [(U.mamba(), None), (U.latent(), None), (U.attention(), None)], seed=21, edit=slow)
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
    layers = [(U.attention(sharp=2.0), U.dense()), (U.mamba(), None), (U.latent(sharp=2.0), None)]
    d, pm = U.make(tmp_path / "long", layers, seed=9, loop=(0, 2, 2))
    ids = ids_for(np.random.default_rng(9), VOCAB, 190)
    ref = pm.logits(ids).numpy()
    page = 16 if dtype == "float32" else 64       # the tensor-core kernels read pages in tiles of 64 keys
    eng = engine_for(d, dtype, max_tokens=page * 20, page_size=page)
    assert_close(replay_tail_one_by_one(eng, ids, 170), ref, dtype, "170 decoded tokens", plain=pm, ids=ids)
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_and_its_continuation(tmp_path, dtype):
    """600 tokens at once and in two portions (several tiles of queries and keys, ten chunks of the recurrence), then 24
    more; heads of 128 value channels, so that prompts take the tcgen05 attention."""
    layers = [(U.attention(heads=2, kv_heads=1, dim=64, vdim=128, rot_dims=32), U.dense(ff=256)), (U.mamba(heads=4, vdim=64, state=128, groups=2, conv=4), None),
              (U.latent(heads=4, dim=32, rot_dim=32, vdim=32, kv_rank=128), U.dense(ff=256))]
    d, pm = U.make(tmp_path / "p600", layers, seed=12, width=128, streams=4)
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
    "one_of_everything": ([(U.attention(heads=1, kv_heads=1, dim=2, vdim=1), U.dense(ff=1)), (U.mamba(heads=1, vdim=1, state=1, groups=1, norm_groups=1, conv=1), U.dense(ff=8)),
                           (U.latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1), None)], {"streams": 1, "width": 24}),
    "sizes_no_tile_divides": ([(U.attention(heads=6, kv_heads=3, dim=10, vdim=37, rot_dims=6), U.dense(ff=76)),
                               (U.mamba(heads=6, vdim=11, state=27, groups=3, norm_groups=6, conv=7), U.dense(ff=33)),
                               (U.latent(heads=3, dim=9, rot_dim=6, vdim=13, kv_rank=21), None)], {"width": 92, "streams": 7, "loop": (1, 3, 2)}),
    "values_narrower_than_both_maps": ([(U.attention(heads=3, kv_heads=3, dim=24, vdim=16), U.dense()), (U.mamba(), None)], {"loop": (1, 2, 4)}),
    "many_query_heads_wide_values": ([(U.attention(heads=10, kv_heads=1, dim=8, vdim=72, diff=0.9), None)], {"streams": 4}),
    "wide_states_and_heads": ([(U.mamba(heads=2, vdim=160, state=264, groups=1, norm_groups=5), None), (U.mamba(heads=2, vdim=96, state=160, groups=2), None),
                               (U.latent(heads=2, dim=40, rot_dim=24, vdim=96, kv_rank=200), None)], {"streams": 2}),
    "everything_looped": ([(U.latent(), U.dense(limit=0.4)), (U.mamba(), U.dense()), (U.attention(), None)], {"loop": (0, 3, 2), "streams": 9}),
    "heads_of_320": ([(U.attention(heads=2, kv_heads=1, dim=160, vdim=48, rot_dims=32), None)], {"streams": 2}),
    "heads_of_256": ([(U.attention(heads=2, kv_heads=1, dim=128, vdim=256, rot_dims=64), None)], {"streams": 2}),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(OTHER))
def test_other_sizes_and_orders(tmp_path, which, dtype):
    layers, kw = OTHER[which]
    d, pm = U.make(tmp_path / which, layers, seed=len(which), **kw)
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
    ops.options.attention = ops.options.latent_attention = "simt"
    ops.options.ssd_chunked = False
    try:
        eng = engine_for(d, dtype, max_tokens=512)
        assert_close(replay_tail_one_by_one(eng, ids, 20), ref, dtype, "any-shape kernels", plain=pm, ids=ids)
    finally:
        ops.options.attention, ops.options.latent_attention, ops.options.ssd_chunked = "auto", "mma", True


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
    cfg = U.config([(U.attention(), U.dense()), (U.mamba(), None), (U.latent(), U.dense())], loop=(0, 2, 2))
    hb.write_random_model(cfg, str(tmp_path), seed=1)
    pm = P.PlainPutazen(str(tmp_path))
    assert {k: tuple(v.shape) for k, v in pm.W.items()} == {k: tuple(v.shape) for k, v in U.weights(cfg).items()}
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
