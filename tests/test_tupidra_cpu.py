"""Host-side logic of the latent-attention / selective-scan / capped-attention decoder: configuration, registry, parameter
layouts, sequence state, argument validation of its kernels; the plain restatement on known answers."""
import copy
import ctypes
import json

import pytest
import torch

import tulezen_plain as T
import tupidra_plain as P
from energonai_b200 import _lib, registry
from energonai_b200.attention import distance_slopes, yarn_rotation
from energonai_b200.model import (CappedAttention, GenerationModel, LayeredDecoder, ParallelDecoder, ParallelDecoderConfig, RecurrentState, RingCache,
                                  RotaryLatentAttention, SelectiveScan, SequenceState)
from energonai_b200.utils import processing_Tupidra

YARN = (4.0, 30, 4.0, 0.5)


def config():
    return P.make_config([P.scan_layer(44, 6, 5, 3, P.dense_mlp(44)), P.attention_layer(6, 2, 12, 20, 0.3, 4.0, (9, 3), P.dense_mlp(36)),
                          P.latent_layer(3, 12, 6, 10, 20, 18, 0.25, 100.0, YARN), P.attention_layer(2, 2, 9, 9, 0.3),
                          P.latent_layer(5, 20, 6, 24, 12, 18, 0.2, 100.0, YARN, kv_from=2, mlp=P.dense_mlp(20))], width=52, vocab=83, taps=3)


def changed(path, value):
    d = copy.deepcopy(config())
    at = d
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return d


def test_configuration_reads_every_size_and_rejects_what_it_does_not_know():
    c = ParallelDecoderConfig.from_dict(config())
    assert (c.vocab, c.width, c.eps, c.taps, len(c.layers)) == (83, 52, 2e-5, 3, 5)
    s, a, m, b, k = (x.mixer for x in c.layers)
    assert (s.inner, s.state, s.dt_rank, s.conv) == (44, 6, 5, 3) and c.layers[0].mlp.ff == 44
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.window, a.keep_first) == (6, 2, 12, 20, 0.3, 4.0, 9, 3)
    assert (b.softcap, b.window, b.keep_first) == (0.0, 0, 0) and c.layers[2].mlp is None
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.rot_base, m.rot_scaling, m.kv_from) == (3, 12, 6, 10, 20, 18, 0.25, 100.0, YARN, None)
    assert (k.kv_from, k.dim, k.q_rank) == (2, 20, 12)
    bad = [(("layers", 0, "type"), "mamba9"), (("layers", 0, "mixer", "state"), 300), (("layers", 0, "mixer", "skip"), 1), (("layers", 1, "mixer", "kv_heads"), 4),
           (("layers", 1, "mixer", "rot"), {"dims": 2}), (("layers", 1, "mixer", "softcap"), -1.0), (("layers", 1, "mixer", "mask", "keep_first"), -1),
           (("layers", 1, "mlp", "kind"), "moe"), (("layers", 2, "mixer", "rot", "dims"), 4), (("layers", 2, "mixer", "rot_dim"), 7), (("layers", 2, "mixer", "mask"), {"size": 3}),
           (("layers", 4, "mixer", "kv_from"), 1), (("layers", 4, "mixer", "kv_from"), 4), (("layers", 4, "mixer", "kv_rank"), 20),
           (("layers", 4, "mixer", "rot", "base"), 50.0), (("layers", 4, "mixer", "rot", "scaling", "factor"), 2.0), (("canon", "taps"), 17), (("canon", "bias"), True), (("tied",), True)]
    for path, value in bad:
        with pytest.raises(ValueError):
            ParallelDecoderConfig.from_dict(changed(path, value))
    for path in (("canon", "taps"), ("norm", "eps"), ("layers", 0, "mixer", "dt_rank"), ("layers", 1, "mixer", "scale"), ("layers", 2, "mixer", "rot"),
                 ("layers", 2, "mixer", "rot", "scaling", "slow")):
        with pytest.raises(KeyError):
            ParallelDecoderConfig.from_dict(changed(path, None))
    chain = config()
    chain["layers"].append(copy.deepcopy(chain["layers"][4]))
    chain["layers"][5]["mixer"]["kv_from"] = 4
    with pytest.raises(ValueError, match="no latents"):
        ParallelDecoderConfig.from_dict(chain)


def test_registry_knows_the_design():
    assert "Tupidra" in registry.architectures()
    model = registry.build_model("Tupidra", config_dict=config(), dtype=torch.float32)
    assert isinstance(model, ParallelDecoder) and isinstance(model, LayeredDecoder) and isinstance(model, GenerationModel)
    assert [type(b.mixer) for b in model.layers] == [SelectiveScan, CappedAttention, RotaryLatentAttention, CappedAttention, RotaryLatentAttention]
    assert model.head is not model.embed and [b.bias is not None for b in model.layers] == [False, True, False, True, False]


def test_padded_sizes():
    m = registry.build_model("Tupidra", config_dict=config(), dtype=torch.bfloat16).layers
    assert (m[0].mixer.inner, m[0].mixer.states, m[0].mixer.rank) == (48, 8, 8)
    assert (m[1].mixer.dk, m[1].mixer.dv, m[1].mixer.tensor_core) == (64, 64, True)
    assert (m[2].mixer.dk, m[2].mixer.dv, m[2].mixer.rank, m[2].mixer.rot_at, m[2].mixer.rot_col, m[2].mixer.q_cols) == (64, 64, 64, 16, 24, 24)
    m = registry.build_model("Tupidra", config_dict=config(), dtype=torch.float32).layers
    assert (m[1].mixer.dk, m[1].mixer.dv, m[1].mixer.tensor_core) == (16, 24, False)
    assert (m[2].mixer.dk, m[2].mixer.dv, m[2].mixer.rank) == (24, 16, 32) and (m[4].mixer.dk, m[4].mixer.dv) == (32, 24)
    wide = P.make_config([P.latent_layer(2, 64, 40, 60, 8, 250, 0.1, 10.0), P.latent_layer(2, 120, 10, 64, 8, 500, 0.1, 10.0), P.latent_layer(2, 30, 10, 100, 8, 20, 0.1, 10.0),
                          P.latent_layer(2, 190, 10, 64, 8, 600, 0.1, 10.0)], 64, 50)
    m = registry.build_model("Tupidra", config_dict=wide, dtype=torch.bfloat16).layers
    at = lambda i: (m[i].mixer.dk, m[i].mixer.dv, m[i].mixer.rank, m[i].mixer.tensor_core_prompt, m[i].mixer.tensor_core_step)
    assert at(0) == (128, 64, 320, True, True) and at(1) == (192, 64, 576, True, True) and at(2) == (128, 128, 64, True, True)
    assert at(3) == (208, 64, 616, False, False)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_parameters_in_kernel_layout_hold_the_checkpoint(tmp_path, dtype):
    cfg = config()
    t = P.make_tensors(cfg, 3)
    T.save_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    model = registry.load_model(str(tmp_path), dtype=dtype, device="cpu")
    f = lambda name: t[name].float()
    g = torch.Generator().manual_seed(1)
    W, w = model.hidden_size, cfg["width"]
    h = torch.zeros(4, W)
    h[:, :w] = torch.randn(4, w, generator=g)
    hs = h[:, :w]
    close = lambda a, b: torch.allclose(a, b, atol=5e-5)

    def heads(y, n, padded, dim):
        y = y.reshape(*y.shape[:-1], n, padded)
        assert float(y[..., dim:].abs().sum()) == 0
        return y[..., :dim].reshape(*y.shape[:-2], -1)
    assert torch.equal(model.embed[:83, :w].float(), f("embed")) and torch.equal(model.head[:83, :w].float(), f("head")) and model.embed.data_ptr() != model.head.data_ptr()
    for i, ly in enumerate(cfg["layers"]):
        blk, m, p = model.layers[i], ly["mixer"], f"l{i}."
        at, q = blk.mixer, p + "mix."
        for k, table in ((1, blk.taps1), (2, blk.taps2)):
            if k == 2 and ly["mlp"] is None:
                assert table is None and blk.mlp is None
                continue
            want = f(f"{p}canon{k}").T.clone()
            want[-1] += 1
            assert table.dtype == torch.float32 and torch.equal(table[:, :w], want * f(f"{p}norm{k}")) and float(table[:, w:].abs().sum()) == 0
        y = h @ at.in_proj.float().T
        if isinstance(at, SelectiveScan):
            C, N, R = m["inner"], m["state"], m["dt_rank"]
            for got, ref in zip(y.split([at.inner, at.inner], 1), (hs @ f(q + "in").T).split([C, C], 1)):
                assert close(heads(got, 1, at.inner, C), ref)
            x = torch.zeros(4, at.inner)
            x[:, :C] = torch.randn(4, C, generator=g)
            parts = (x @ at.x_proj.float().T).split([at.rank, at.states, at.states], 1)
            for got, ref, n in zip(parts, (x[:, :C] @ f(q + "x").T).split([R, N, N], 1), (R, N, N)):
                assert close(heads(got, 1, got.shape[1], n), ref)
            assert close((parts[0] @ at.dt_proj.float().T)[:, :C], parts[0][:, :R] @ f(q + "dt").T)
            assert torch.equal(at.conv_w[:, :C].float().T, f(q + "conv")) and torch.equal(at.conv_b[:C].float(), f(q + "conv.b"))
            for got, name in ((at.dt_bias, "dt.b"), (at.skip, "D")):
                assert got.dtype == torch.float32 and torch.equal(got[:C], f(q + name))
            assert at.a_log.dtype == torch.float32 and torch.equal(at.a_log[:C, :N], f(q + "A_log"))
            H, dv, pad = 1, C, at.inner
        elif isinstance(at, CappedAttention):
            H, G, dv, pad = m["heads"], m["kv_heads"], m["vdim"], at.dv
            y = y + at.bias.float()
            for got, name, n, to, d in zip(y.split(at.splits, 1), "qkvg", (H, G, G, H), (at.dk, at.dk, at.dv, at.dv), (m["dim"], m["dim"], dv, dv)):
                assert close(heads(got, n, to, d), hs @ f(q + name).T + (f(f"{q}{name}.b") if name != "g" else 0))
            assert torch.equal(blk.bias[:w].float(), f(q + "o.b"))
        else:
            H, d, r, dv, qr, kr, pad = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], at.dv
            own = m.get("kv_from") is None
            parts = y.split([at.q_cols] + ([at.rank] if own else []) + [at.columns], 1)
            assert close(heads(parts[0], 1, at.q_cols, qr), hs @ f(q + "dq").T) and close(heads(parts[-1], H, at.dv, dv), hs @ f(q + "g").T)
            if own:
                row = parts[1]
                c, kp = (hs @ f(q + "dkv").T).split([kr, r], 1)
                assert close(heads(row[:, :at.rot_col], 1, at.rot_col, kr), c) and close(row[:, at.rot_col:at.rot_col + r], kp) and float(row[:, at.rot_col + r:].abs().sum()) == 0
                assert torch.equal(at.latent_norm[:kr].float(), f(q + "dkv.norm"))
            else:
                assert at.latent_norm is None
            qs = (parts[0] @ at.q_up.float().T).view(4, H, at.dk)
            want = (parts[0][:, :qr] @ f(q + "uq").T).view(4, H, d + r)
            assert close(qs[..., :d], want[..., :d]) and close(qs[..., at.rot_at:at.rot_at + r], want[..., d:])
            row = torch.zeros(4, at.rank)
            row[:, :kr], row[:, at.rot_col:at.rot_col + r] = torch.randn(4, kr, generator=g), torch.randn(4, r, generator=g)
            kv = row @ at.kv_up.float().T
            keys = kv[:, :at.q_rows].view(4, H, at.dk)
            assert close(keys[..., :d].reshape(4, -1), row[:, :kr] @ f(q + "uk").T) and torch.equal(keys[..., at.rot_at:at.rot_at + r], row[:, None, at.rot_col:at.rot_col + r].expand(4, H, r))
            assert close(heads(kv[:, at.q_rows:], H, at.dv, dv), row[:, :kr] @ f(q + "uv").T)
            # a score by the absorbed query is the score by the key
            absorbed = torch.einsum("bhk,hrk->bhr", qs, at.k_absorb.float())
            assert torch.allclose((absorbed * row[:, None]).sum(-1), (qs * keys).sum(-1), atol=1e-3, rtol=1e-3)
            assert at.sinks.dtype == torch.float32 and torch.equal(at.sinks, f(q + "sink")) and torch.equal(at.q_norm[:qr].float(), f(q + "dq.norm"))
        z = torch.zeros(4, H, pad)
        z[..., :dv] = torch.randn(4, H, dv, generator=g)
        inner, want = z.view(4, -1), z[..., :dv].reshape(4, -1) @ f(q + "o").T
        if ly["mlp"] is not None:
            ff = ly["mlp"]["ff"]
            u = (h @ blk.mlp.gate_up.float().T).view(4, -1, 2, 8)
            for j, name in enumerate(("gate", "up")):
                assert close(u[:, :, j].reshape(4, -1)[:, :ff], hs @ f(f"{p}mlp.{name}").T)
            e = torch.zeros(4, blk.mlp.ff_padded)
            e[:, :ff] = torch.randn(4, ff, generator=g)
            inner, want = torch.cat([inner, e], 1), want + e[:, :ff] @ f(p + "mlp.down").T
        assert close((inner @ blk.out_proj.float().T)[:, :w], want)


def test_checkpoint_conversion_complains_about_missing_surplus_and_misshapen_tensors():
    cfg = config()
    t = P.make_tensors(cfg, 3)
    model = registry.build_model("Tupidra", config_dict=cfg, dtype=torch.float32)
    processing_Tupidra(t, model)
    for name in ("head", "l0.canon1", "l0.mix.A_log", "l1.mix.o.b", "l1.mix.g", "l2.mix.dkv.norm", "l4.mix.sink", "l4.canon2"):
        with pytest.raises(KeyError, match="lacks"):
            processing_Tupidra({k: v for k, v in t.items() if k != name}, model)
    for name in ("l2.norm2", "l4.mix.dkv", "l0.mix.o.b"):
        with pytest.raises(KeyError, match=name):
            processing_Tupidra(dict(t, **{name: t["l0.norm1"]}), model)
    with pytest.raises(ValueError, match="l0.mix.x"):
        processing_Tupidra(dict(t, **{"l0.mix.x": t["l0.mix.x"][:-1]}), model)


def test_state_of_every_kind_is_prepared_kept_grown_and_forked():
    m = registry.build_model("Tupidra", config_dict=config(), dtype=torch.float32)
    s = m.new_state()
    assert isinstance(s, SequenceState)
    kinds = {k: type(c) for k, c in s.caches.items()}
    rows = {(i, "rows"): RingCache for i in range(5)}
    assert kinds == {**rows, (0, "conv"): RingCache, (0, "state"): RecurrentState, (1, "keys"): RingCache, 2: RingCache, (3, "keys"): RingCache}      # (layer 4 reads layer 2's)
    assert (s.caches[1, "keys"].window, s.caches[1, "keys"].kept, s.caches[3, "keys"].window, s.caches[0, "rows"].window, s.caches[2].window) == (9, 3, 0, 3, 0)
    dev = torch.device("cpu")
    s.begin([2, 0, 1], 20, 5, torch.float32, dev)
    assert s.caches[1, "keys"].buf.shape[1] == 12 and s.caches[0, "rows"].buf.shape[1] == 3 and s.caches[2].buf.shape[1] == 25 and s.capacity() == 25
    assert s.caches[0, "state"].tensors[0].shape == (3, 48, 8)
    s.caches[1, "keys"].buf[:] = torch.arange(3.0)[:, None, None]
    two = s.fork([1])
    s.keep([0, 2])
    assert two.caches[1, "keys"].kept == 3 and two.caches[1, "keys"].buf[0, 0, 0] == 1 and s.caches[1, "keys"].buf[:, 0, 0].tolist() == [0, 2]
    s.begin([0], 2, 0, torch.float32, dev)                   # shorter than the rings: they grow, rows stay where they are
    assert s.caches[1, "keys"].buf.shape[1] == 5 and s.capacity() == 2
    s.caches[1, "keys"].buf[0, :, 0] = torch.arange(1.0, 6.0)
    s.ensure(3)
    buf = s.caches[1, "keys"].buf
    assert buf.shape[1] == 12 and buf[0, :5, 0].tolist() == [1, 2, 3, 4, 5] and float(buf[0, 5:].abs().sum()) == 0 and s.capacity() >= 3


def test_slopes_and_rotation_tables():
    for H in (1, 3, 4, 20):
        assert torch.allclose(distance_slopes(H).double(), P.slopes(H))
    for dims, base, scaling in ((16, 1e4, None), (64, 3e5, (6.0, 1024, 24.0, 1.0)), (8, 100.0, YARN), (12, 50.0, (8.0, 10, 100.0, 50.0)), (2, 7.0, (2.0, 10, 1.0, 1.0))):
        freq, factor = yarn_rotation(dims, base, scaling)
        want, wf = P.yarn(dims, base, dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None)
        assert torch.allclose(freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6) and abs(factor - wf) < 1e-12


def test_plain_restatement_on_known_answers():
    """The equations by other means: closed forms, torch's own functions, step-by-step sums."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    z = r(50)
    assert torch.allclose(P.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh")) and torch.allclose(P.silu(z), torch.nn.functional.silu(z))
    x, w = r(9, 4), r(4, 3)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T[None], (2, 0)), w[:, None], groups=4)[0].T
    assert torch.allclose(P.causal_conv(x, w), ref) and torch.allclose(P.mixed_input(x, w), x + ref)
    # one decay for all: a geometric sum
    n, C, N = 6, 2, 3
    xx, B, Cn, dt = r(n, C), r(n, N), r(n, N), torch.full((n, C), 0.5, dtype=torch.float64)
    y, S = P.selective_scan(xx, dt, -torch.ones(C, N, dtype=torch.float64), B, Cn, torch.ones(C, dtype=torch.float64))
    want = xx[-1] + sum(torch.exp(torch.tensor(-0.5 * (n - 1 - s))) * 0.5 * (B[s] @ Cn[-1]) * xx[s] for s in range(n))
    assert torch.allclose(y[-1], want) and S.shape == (C, N)
    # pairs that turn often keep their pace, slow ones are slowed down, and both factors stand in the rotated vector
    f0, f = P.yarn(32, 1e4, None)[0], P.yarn(32, 1e4, {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0})
    assert f[0][0] == f0[0] and abs(f[0][-1] - f0[-1] / 4) < 1e-15 and all(a >= b for a, b in zip(f0, f[0])) and abs(f[1] - (1 + 0.1 * 1.3862943611198906)) < 1e-12
    rot = {"dims": 6, "base": 50.0, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    q, k = r(1, 1, 8).expand(10, 1, 8), r(1, 1, 8).expand(10, 1, 8)
    a, c = P.rotate(q, range(10), rot), P.rotate(k, range(10), rot)
    m = 1 + 0.1 * 1.0986122886681098
    assert torch.allclose(a[..., :6].norm(dim=-1), q[..., :6].norm(dim=-1) * m) and torch.equal(a[..., 6:], q[..., 6:])
    assert torch.allclose((a[7, :, :6] * c[4, :, :6]).sum(), (a[5, :, :6] * c[2, :, :6]).sum())
    seen = P.window_mask(7, 2, 1)
    assert [int(v) for v in seen.sum(-1)] == [1, 2, 3, 3, 3, 3, 3] and bool(seen[5, 0]) and not bool(seen[5, 1]) and bool(P.window_mask(5, None, 0)[4, 0])
    assert [int(v) for v in P.window_mask(6, 1, 9).sum(-1)] == [1, 2, 3, 4, 5, 6]
    # a sink of the size of the only score takes half; scores beyond the cap count as the cap; the bias is the slope times the distance
    p = P.softmax_with_sink(torch.full((1, 1, 1), 0.7, dtype=torch.float64), torch.ones(1, 1, dtype=torch.bool), torch.tensor([0.7], dtype=torch.float64))
    assert float(p) == 0.5
    q, v = torch.full((2, 1, 1), 1e3, dtype=torch.float64), torch.tensor([[[1.0]], [[0.0]]], dtype=torch.float64)
    o = P.capped_attention(q, q, v, 1.0, 2.0, P.window_mask(2, None, 0))
    e = torch.exp(torch.tensor([2.0 - 2.0 ** -8, 2.0], dtype=torch.float64))
    assert torch.allclose(o[1, 0, 0], e[0] / (1 + e.sum()))


def test_kernels_validate_before_any_cuda_call():
    L = _lib.lib()
    buf = ctypes.create_string_buffer(64)
    a = (ctypes.addressof(buf) + 15) & ~15
    B16, F32 = _lib.BF16, _lib.F32
    err = _lib.last_error
    conv = lambda x=a, out=a + 16, taps=4, n2=8, ring=a, h2=None, k2=None, pos=None, seq=4, y=a: L.eb_stream_conv(
        None, 8, x, 8, y, 8, out, a, k2, taps, a, h2, 8, ring, 32, 8, 4, 1, seq, n2, 8, 1e-5, None, pos, B16, None)
    assert conv(out=a) == -1 and "in place" in err() and conv(taps=5) == -1 and conv(n2=12) == -1 and conv(ring=None) == -1 and conv(h2=a) == -1 and conv(x=None) == -1
    assert conv(pos=a) == -1 and "one row per sequence" in err()
    scan = lambda inner=8, states=4, z=a, ldz=8, dtype=B16, ldbc=8: L.eb_selective_scan(a, 8, a, 8, z, ldz, a, ldbc, a, a, a, None, a, 8, a, 1, 2, inner, states, dtype, None)
    assert scan(inner=12) == -1 and scan(states=6) == -1 and scan(states=260) == -1 and scan(z=None) == -1 and scan(ldz=4) == -1 and scan(dtype=9) == -1 and scan(ldbc=4) == -1
    step = lambda rank=8, w=a: L.eb_selective_step(a, 8, a, 8, a, 8, w, rank, a, 8, a, a, a, a, 8, a, 1, 8, 4, B16, None)
    assert step(rank=12) == -1 and "rank" in err() and step(w=None) == -1
    cstep = lambda C=8, pos=a: L.eb_short_conv_step(a, 8, a, a, a, 8, 1, C, 4, pos, None, a, 32, 8, 4, B16, None)
    assert cstep(C=12) == -1 and cstep(pos=None) == -1
    val = lambda dk=8, count=8, keep=0, rows=4, ld=16: L.eb_attention_values(a, a, ld, 1, dk, 8, count, 1e-5, a, 64, 8, a, 64, 8, keep, rows, 1, 1, None, None, B16, None)
    assert val(dk=12) == -1 and val(count=9) == -1 and val(keep=-1) == -1 and val(rows=0) == -1 and val(ld=4) == -1
    assert L.eb_sigmoid_gate(a, 8, a, 8, a, 8, 1, 12, B16, None) == -1 and L.eb_sigmoid_gate(a, 8, None, 8, a, 8, 1, 8, B16, None) == -1
    lat = lambda q=8, ring=a, rot=8, cols=16, pairs=2, rows=None, norm=a: L.eb_latent_inputs(a, 64, q, 8, a, a, 8, cols, rot, 8, norm, pairs, a, 1.0, 1e-5, rows, 16, ring, 64, 16, 4,
                                                                                             1, 1, None, None, B16, None)
    assert lat(q=12) == -1 and lat(pairs=5) == -1 and "rotated part" in err() and lat(cols=12) == -1 and lat(norm=None) == -1 and lat(ring=None, rows=a) == -1
    assert L.eb_rotate_heads(a, 16, 1, 16, 8, 5, a, 1.0, 1, 1, None, None, B16, None) == -1 and L.eb_rotate_heads(a, 16, 1, 16, 7, 2, a, 1.0, 1, 1, None, None, B16, None) == -1
    pre = lambda k=64, v=64, group=1, window=0, keep=0, cap=1.0, scale=0.1, gate=None: L.eb_attention_prefill_capped_tc(
        a, a, a, a, gate, *[64] * 10, 1, 2, group, 8, k, v, window, keep, None, a, cap, 1, scale, B16, None)
    assert pre(group=3) == -1 and pre(k=96) == -1 and pre(k=192) == -1 and pre(v=128) == -1 and pre(keep=-1) == -1 and pre(cap=-1.0) == -1 and pre(scale=0.0) == -1 and pre(window=-1) == -1
    assert pre(gate=a + 2) == -1 and "gate" in err()
    gated = lambda k=64, v=64, group=1: L.eb_attention_prefill_gated_tc(a, a, a, a, None, *[64] * 10, 1, 2, group, 8, k, v, None, None, 0.1, B16, None)
    assert gated(group=3) == -1 and gated(k=32) == -1 and gated(v=32) == -1 and gated(k=192, v=192) == -1 and gated(k=256) == -1
    dec = lambda kv=2, keep=0, cap=0.0, nsplit=1, window=4: L.eb_attention_group_decode_capped(a, a, a, a, None, 256, 640, 128, 640, 128, 256, 0, 1, 4, kv, 64, keep, 5, window, a, None,
                                                                                              None, cap, 1, 1.0, B16, nsplit, None, 0, None)
    assert dec(kv=3) == -1 and dec(keep=-1) == -1 and dec(cap=-1.0) == -1 and dec(nsplit=2) == -1 and dec(window=-1) == -1
    plain = lambda keep=0, kept=0, cap=0.0: L.eb_attention_plain_capped(a, a, a, a, *[8] * 12, 1, 2, 1, 1, 8, 8, 4, keep, kept, 4, None, None, None, cap, 1, 1.0, F32, None)
    assert plain(keep=-1) == -1 and plain(keep=2, kept=1) == -1 and "first positions" in err() and plain(cap=-1.0) == -1
    sink = lambda rank=64: L.eb_latent_decode_sink(a, 64, a, 640, 64, 10, a, 64, 1, 1, rank, 4, a, None, a, 1.0, B16, 1, None, 0, None)
    assert sink(rank=96) == -1 and "latent width" in err()
