"""The Putazen design without a GPU: configuration reading and its error messages, the tensor declaration, cache needs,
and the plain implementation against second forms of its own mechanisms."""
import copy
import math

import numpy as np
import pytest
import torch

import herbert_rs_b200 as hb
import plain_putazen as P
import putazen_util as U
from herbert_rs_b200.cache import SequenceCache
from herbert_rs_b200.config.putazen import PutazenConfig
from herbert_rs_b200.config.specs import ScaledRotarySpec
from herbert_rs_b200.errors import ConfigError
from herbert_rs_b200.parts.rope import pair_frequencies, scaled_frequencies
from herbert_rs_b200.weights.loader import build_model

F64 = torch.float64


def test_configuration_is_read_from_the_nested_keys():
    cfg = U.config([(U.attention(heads=6, kv_heads=3, dim=24, vdim=40, rot_dims=10, base=777.0, scale=0.3, diff=0.7,
                                 scaling={"factor": 5.0, "original": 100, "fast": 9.0, "slow": 2.0}), U.dense(ff=56, limit=2.5)),
                    (U.mamba(heads=6, vdim=8, state=20, groups=3, norm_groups=4, conv=5), None),
                    (U.latent(heads=5, dim=12, rot_dim=6, vdim=10, kv_rank=18, base=333.0), U.dense())],
                   vocab=99, width=72, eps=3e-6, streams=5, loop=(1, 3, 4), scale=1.25)
    spec = PutazenConfig.from_dict(cfg).model_spec()
    assert (spec.vocab_size, spec.hidden_size, spec.streams, spec.embedding_scale) == (99, 72, 5, 1.25)
    assert [s.layer for s in spec.schedule] == [0] + [1, 2] * 4 and all(s.reads_cache_of is None for s in spec.schedule)
    b0, b1, b2 = spec.blocks
    assert (b0.kind, b0.streams, b0.norm1.kind, b0.norm1.bias, b0.norm1.eps, b0.norm2.weight_name) == ("streams", 5, "layernorm", True, 3e-6, "norm2")
    a = b0.mixer
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.scale, a.difference, a.difference_eps) == (6, 3, 24, 40, 0.3, 0.7, 3e-6)
    assert a.bias and a.position == ScaledRotarySpec(10, 777.0, 5.0, 100.0, 9.0, 2.0)
    assert (b0.ffn.intermediate_size, b0.ffn.act_limit, b0.ffn.activation) == (56, 2.5, "swish_clamp") and b1.ffn is None
    m = b1.mixer
    assert (m.num_heads, m.value_dim, m.state_dim, m.groups, m.norm_groups, m.conv_taps, m.norm_eps) == (6, 8, 20, 3, 4, 5, 3e-6)
    t = b2.mixer
    assert (t.num_heads, t.nope_dim, t.rope_dim, t.v_dim, t.kv_rank, t.q_rank, t.gate, t.sink, t.window) == (5, 12, 6, 10, 18, None, False, False, None)
    assert (t.position.layout, t.position.rotary_dim, t.position.theta) == ("interleaved", 6, 333.0)
    assert hb.registry.architecture_for(cfg) == "Putazen"
    del cfg["loop"], cfg["embedding"], cfg["layers"][0]["mixer"]["rot"]["scaling"]
    spec = PutazenConfig.from_dict(cfg).model_spec()
    assert [s.layer for s in spec.schedule] == [0, 1, 2] and spec.embedding_scale == 1.0
    assert spec.blocks[0].mixer.position == ScaledRotarySpec(10, 777.0)
    del cfg["layers"][0]["mixer"]["rot"]
    assert PutazenConfig.from_dict(cfg).model_spec().blocks[0].mixer.position is None


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "multiple of groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "rot_dim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda c: c.update(loop={"start": 2, "stop": 1, "times": 2}), "loop"),
    (lambda c: c.update(loop={"start": 0, "stop": 4, "times": 2}), "loop"),
    (lambda c: c.update(loop={"start": 0, "stop": 1, "times": 0}), "times"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(edit, message):
    cfg = U.config([(U.attention(), U.dense()), (U.mamba(), None), (U.latent(), None)])
    edit(cfg)
    with pytest.raises(ConfigError, match=message):
        PutazenConfig.from_dict(cfg)


def test_blocks_and_model_agree_on_the_number_of_copies():
    import dataclasses
    from herbert_rs_b200.models import DecoderModel
    spec = PutazenConfig.from_dict(U.config([(U.mamba(), None)], streams=3)).model_spec()
    with pytest.raises(ConfigError, match="copies of the stream"):
        DecoderModel(dataclasses.replace(spec, streams=2), hb.Runtime("cpu", torch.bfloat16))


def test_declared_tensors_and_cache_need(tmp_path):
    cfg = U.config([(U.attention(heads=4, kv_heads=2, dim=12, vdim=20), U.dense()), (U.mamba(heads=4, vdim=16, state=24, groups=2, conv=4), None),
                    (U.latent(kv_rank=32, rot_dim=8), U.dense()), (U.mamba(conv=1), U.dense())], loop=(1, 3, 2), streams=4)
    model = build_model(cfg, hb.Runtime("cpu", torch.bfloat16))
    specs, t = model.param_specs(), U.weights(cfg)
    assert {k: tuple(v.shape) for k, v in specs.items()} == {k: tuple(v.shape) for k, v in t.items()}
    assert "l1.norm2" not in specs and "l1.hc2.mix" not in specs and specs["l0.hc1.mix"].shape == (4, 4)
    needs = model.cache_needs()
    assert len(needs) == 6
    # both maps' keys side by side, beside values of 20, in steps of 16 channels
    assert (needs[0].kv.num_kv_heads, needs[0].kv.head_dim, needs[0].kv.planes) == (2, 32, 2)
    assert tuple(needs[1].state.shape) == (4, 24, 16) and dict(needs[1].states)["conv"].shape == (3, 4 * 16 + 2 * 2 * 24)
    assert (needs[2].kv.head_dim, needs[2].kv.planes) == (40, 1) and needs[5].states == ()
    cache = SequenceCache(needs, model.reads_cache_of(), num_pages=8, num_slots=2, page_size=16)
    # every run of a looped layer has an entry of its own
    assert cache.step_state[1] != cache.step_state[3] and cache.step_kv[2] != cache.step_kv[4]
    U.write(cfg, t, tmp_path)
    assert P.PlainPutazen(str(tmp_path)).logits([1, 2, 3]).shape == (3, 131)


def test_a_missing_or_misshapen_tensor_is_reported(tmp_path):
    from herbert_rs_b200.errors import WeightError
    from herbert_rs_b200.weights.loader import check_tensors
    from herbert_rs_b200.weights.safetensors_io import ModelFiles
    cfg = U.config([(U.attention(), U.dense()), (U.mamba(), None)])
    t = U.weights(cfg)
    del t["l1.mix.dt_bias"], t["final.norm.b"]
    t["l0.hc2.mix"] = t["l0.hc2.mix"][:, :-1].contiguous()
    t["l0.mix.k"] = t["l0.mix.k"][:-1].contiguous()
    U.write(cfg, t, tmp_path)
    files = ModelFiles(str(tmp_path))
    with pytest.raises(WeightError) as e:
        check_tensors(build_model(cfg, hb.Runtime("cpu", torch.bfloat16)), files)
    files.close()
    assert all(n in str(e.value) for n in ("l1.mix.dt_bias", "final.norm.b", "l0.hc2.mix", "l0.mix.k"))


# ---- the plain implementation against second forms of its mechanisms --------------------------------
def test_small_functions_against_torch():
    g = torch.Generator().manual_seed(0)
    F = torch.nn.functional
    x = torch.randn(5, 24, generator=g, dtype=F64) * 3
    w, b = 1 + 0.1 * torch.randn(24, generator=g, dtype=F64), torch.randn(24, generator=g, dtype=F64)
    assert (P.layer_norm(x, w, b, 1e-5) - F.layer_norm(x, (24,), w, b, 1e-5)).abs().max() < 1e-12
    assert (P.unit_rms(x, 1e-5) - F.rms_norm(x, (24,), None, 1e-5)).abs().max() < 1e-12
    assert (P.silu(x) - F.silu(x)).abs().max() < 1e-12 and (P.softplus(x * 30) - torch.logaddexp(x * 30, torch.zeros_like(x))).abs().max() < 1e-12
    cw = torch.randn(24, 4, generator=g, dtype=F64)
    ref = F.conv1d(F.pad(x.T[None], (3, 0)), cw[:, None, :], b, groups=24)[0].T
    assert (P.causal_conv(x, cw, b) - ref).abs().max() < 1e-12
    y = P.gated_group_norm(x, x.flip(0), w, 3, 1e-5)
    v = (x * F.silu(x.flip(0)))
    for j in range(3):
        part = slice(8 * j, 8 * j + 8)
        assert (y[:, part] - F.rms_norm(v[:, part], (8,), w[part], 1e-5)).abs().max() < 1e-12


def test_the_streams_as_one_matrix():
    g = torch.Generator().manual_seed(1)
    n, T, D = 4, 3, 5
    X, y = torch.randn(n, T, D, generator=g, dtype=F64), torch.randn(T, D, generator=g, dtype=F64)
    M, a, b = (torch.randn(*s, generator=g, dtype=F64) for s in ((n, n), (n,), (n,)))
    assert (P.stream_in(X, a) - torch.einsum("s,std->td", a, X)).abs().max() < 1e-12
    new = P.stream_out(X, y, M, b)
    assert (new - (torch.einsum("st,sid->tid", M, X) + b[:, None, None] * y)).abs().max() < 1e-12
    assert (new - (torch.einsum("ts,sid->tid", M, X) + b[:, None, None] * y)).abs().max() > 0.1       # from, to: not the transpose


def test_frequencies_band_by_band_and_the_library_s_own():
    sc = {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 1.0}
    f, m = P.frequencies(32, 10000.0, sc)
    plain, one = P.frequencies(32, 10000.0)
    assert one == 1.0 and abs(m - (0.1 * math.log(4.0) + 1.0)) < 1e-15
    kinds = {"kept" if a == b else "divided" if abs(a - b / 4) < 1e-18 else "between" for a, b in zip(f, plain)}
    assert kinds == {"kept", "divided", "between"} and f[0] == plain[0] and abs(f[-1] - plain[-1] / 4) < 1e-18
    lib, lm = scaled_frequencies(ScaledRotarySpec(32, 10000.0, 4.0, 256.0, 8.0, 1.0))
    assert np.abs(lib.numpy() - np.array(f)).max() < 1e-12 and lm == m
    assert np.abs(pair_frequencies(32, 10000.0).double().numpy() - np.array(plain)).max() < 1e-7


@pytest.mark.parametrize("interleaved", [False, True])
def test_rotation_makes_scores_depend_on_distance_only(interleaved):
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 2, 16, generator=g, dtype=F64), torch.randn(1, 2, 16, generator=g, dtype=F64)
    f, m = P.frequencies(8, 100.0, {"factor": 2.0, "original": 64, "fast": 4.0, "slow": 1.0})

    def score(i, j):
        return float((P.rotate(q, [i], f, m, 8, interleaved)[0, 0] * P.rotate(k, [j], f, m, 8, interleaved)[0, 0]).sum())
    assert abs(score(10, 3) - score(107, 100)) < 1e-9 and abs(score(10, 3) - score(10, 4)) > 1e-3
    r = P.rotate(q, [5], f, m, 8, interleaved)[0, 1]
    assert torch.equal(r[8:], q[0, 1, 8:]) and abs(float(r[:8].norm() - m * q[0, 1, :8].norm())) < 1e-12
    u, v = (q[0, 1, 2], q[0, 1, 3]) if interleaved else (q[0, 1, 1], q[0, 1, 5])
    a = 5 * f[1]
    assert abs(float(r[2 if interleaved else 1]) - m * float(u * math.cos(a) - v * math.sin(a))) < 1e-12


def test_two_maps_subtracted():
    g = torch.Generator().manual_seed(3)
    T, dk, dv, diff, eps = 9, 4, 6, 0.3, 1e-5
    q, k, v = torch.randn(2, T, dk, generator=g, dtype=F64), torch.randn(2, T, dk, generator=g, dtype=F64), torch.randn(T, dv, generator=g, dtype=F64)
    a = [P.softmax_attention(q[i], k[i], v, 0.7) for i in range(2)]
    for i in range(2):
        for t in range(T):
            w = torch.softmax(k[i, :t + 1] @ q[i, t] * 0.7, -1)
            assert (a[i][t] - w @ v[:t + 1]).abs().max() < 1e-12
    lv = torch.randn(4, dk, generator=g, dtype=F64) * 0.5
    lam = P.difference_factor(*lv, diff)
    assert abs(lam - (math.exp(float(lv[0] @ lv[1])) - math.exp(float(lv[2] @ lv[3])) + diff)) < 1e-12
    o = P.combine_maps(a[0], a[1], lam, diff, eps)
    assert (o.pow(2).mean(-1).sqrt() - (1 - diff)).abs().max() < 1e-3          # rows of one length, 1 - diff
    assert (o - (1 - diff) * torch.nn.functional.rms_norm(a[0] - lam * a[1], (dv,), None, eps)).abs().max() < 1e-12


def test_the_state_space_recurrence_as_a_masked_matrix_and_from_a_saved_state():
    g = torch.Generator().manual_seed(4)
    T, H, G, N, dv = 11, 4, 2, 5, 3
    x, B, C = (torch.randn(T, *s, generator=g, dtype=F64) for s in ((H, dv), (G, N), (G, N)))
    dt, A, D = torch.rand(T, H, generator=g, dtype=F64), torch.rand(H, generator=g, dtype=F64) * 3, torch.randn(H, generator=g, dtype=F64)
    y, S = P.state_space_scan(x, B, C, dt, A, D)
    cum = torch.cumsum(-A * dt, 0)
    for h in range(H):
        L = torch.exp(cum[:, None, h] - cum[None, :, h]).tril()
        M = (C[:, h // 2] @ B[:, h // 2].T) * L * dt[None, :, h]
        assert (y[:, h] - (M @ x[:, h] + D[h] * x[:, h])).abs().max() < 1e-12
    y1, S1 = P.state_space_scan(x[:4], B[:4], C[:4], dt[:4], A, D)
    y2, S2 = P.state_space_scan(x[4:], B[4:], C[4:], dt[4:], A, D, S1)
    assert (torch.cat([y1, y2]) - y).abs().max() < 1e-12 and (S2 - S).abs().max() < 1e-12


def test_the_clamps_one_by_one():
    sw = lambda z: z / (1 + math.exp(-1.702 * z))      # noqa: E731
    y = P.clamped_glu(torch.tensor([5.0, -5.0, 0.3], dtype=F64), torch.tensor([-7.0, 9.0, -0.5], dtype=F64), 2.0)
    assert abs(float(y[0]) - sw(2.0) * (-2.0 + 1)) < 1e-12            # gate capped from above, up clamped from below
    assert abs(float(y[1]) - sw(-5.0) * (2.0 + 1)) < 1e-12            # the gate has no lower limit, up clamped from above
    assert abs(float(y[2]) - sw(0.3) * (-0.5 + 1)) < 1e-12


def test_order_of_layers():
    assert P.order_of_layers(4, None) == [0, 1, 2, 3]
    assert P.order_of_layers(5, {"start": 1, "stop": 3, "times": 3}) == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert P.order_of_layers(3, {"start": 0, "stop": 3, "times": 2}) == [0, 1, 2, 0, 1, 2]
    assert P.order_of_layers(3, {"start": 1, "stop": 1, "times": 2}) == [0, 1, 2]


def test_leaving_out_a_mechanism_moves_the_logits(tmp_path):
    layers = [(U.attention(rot_dims=8), U.dense()), (U.mamba(), U.dense()), (U.latent(), None)]
    d, pm = U.make(tmp_path / "m", layers, seed=8, loop=(1, 3, 2))
    ids = np.random.default_rng(5).integers(0, 131, 40).tolist()
    ref = pm.logits(ids)
    low = float((pm.logits(ids, F64, P.bf16_storage) - ref).abs().max())

    def moved(cfg=None, W=None):
        return float((P.PlainPutazen(config=cfg or pm.cfg, tensors=W or pm.W).logits(ids) - ref).abs().max())

    def edited(fn):
        cfg = copy.deepcopy(pm.cfg)
        fn(cfg)
        return cfg
    att, scan, lat = (lambda c, i=i: c["layers"][i]["mixer"] for i in range(3))
    for what, fn in {
        "loop": lambda c: c.update(loop=None), "one pass fewer": lambda c: c["loop"].update(times=1), "embedding scale": lambda c: c.update(embedding=None),
        "no rotation": lambda c: att(c).pop("rot"), "all rotated": lambda c: att(c)["rot"].update(dims=16),
        "no stretching": lambda c: att(c)["rot"].pop("scaling"), "slow": lambda c: att(c)["rot"]["scaling"].update(slow=3.0),
        "scale": lambda c: att(c).update(scale=0.5), "diff": lambda c: att(c).update(diff=0.2),
        "latent base": lambda c: lat(c)["rot"].update(base=50.0), "latent scale": lambda c: lat(c).update(scale=0.4),
        "norm groups": lambda c: scan(c).update(norm_groups=1), "limit": lambda c: c["layers"][0]["mlp"].update(limit=50.0),
    }.items():
        assert moved(edited(fn)) > 3 * low, what
    for name in ("l0.mix.q.b", "l0.mix.v.b", "l0.mix.lq1", "l1.mix.conv.b", "l1.mix.dt_bias", "l1.mix.D", "l0.norm1.b", "final.norm.b"):
        assert moved(W=dict(pm.W, **{name: torch.zeros_like(pm.W[name])})) > 3 * low, name
    for name in ("l0.hc1.mix", "l1.hc2.mix"):
        assert moved(W=dict(pm.W, **{name: pm.W[name].T.contiguous()})) > 3 * low, name
    for name in ("l0.hc2.in", "l1.hc1.in", "l2.hc1.out"):
        assert moved(W=dict(pm.W, **{name: pm.W[name].roll(1) * 1.5})) > 3 * low, name
    # the rows of B and C belong to groups of neighbouring heads, the maps of a head lie side by side
    m = pm.cfg["layers"][1]["mixer"]
    inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
    w_in = pm.W["l1.mix.in"].clone()
    w_in[2 * inner:2 * inner + gn] = w_in[2 * inner:2 * inner + gn].reshape(m["groups"], -1, 64).flip(0).reshape(gn, 64)
    assert moved(W=dict(pm.W, **{"l1.mix.in": w_in})) > 3 * low
