"""Host-side logic of the state-space / chunk-attention / gated-linear decoder: configuration, registry, parameter
layouts, sequence state, padding rules, argument validation of its kernels; the plain restatement on known
answers."""
import ctypes
import json

import pytest
import torch

import moponex_plain as P
import tulezen_plain as T
from energonai_b200 import _lib, registry
from energonai_b200.decay import chunk_heads
from energonai_b200.model import (GenerationModel, HybridDecoder, HybridDecoderConfig, LayeredDecoder, RecurrentState, RingCache, RoutedExperts, SequenceState,
                                  StateSpace)
from energonai_b200.moe import unit_code
from energonai_b200.utils import processing_Moponex


def config():
    return P.make_config([P.parallel_layer((6, 2, 12, 0.4, 9, (8, 100.0, 3.0)), (3, 20, 28, 4.0, 5), P.dense_mlp(44)),
                          P.ssm_layer(6, 10, 12, groups=3, conv=3, norm_groups=4, mlp=P.moe_mlp(7, 3, 20, identity=2, groups=(3, 2), shared=12)),
                          P.parallel_layer((2, 2, 10, 0.5, 0, None), (1, 8, 12, 1.0, 16), P.moe_mlp(5, 2, 12)),
                          P.ssm_layer(4, 16, 24, groups=4, conv=2)], width=52, vocab=83)


def test_configuration_reads_every_size_and_rejects_what_it_does_not_know():
    c = HybridDecoderConfig.from_dict(P.file_config(config()))
    assert (c.vocab, c.width, c.eps, c.residual_mult, c.logit_scale, len(c.layers)) == (83, 52, 2e-5, 0.6, 0.3, 4)
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur) == (97, 29, 11)
    a, r = c.layers[0].mixer.left, c.layers[0].mixer.right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.rot_dims, a.rot_base, a.rot_factor) == (6, 2, 12, 12, 0.4, 9, 8, 100.0, 3.0)
    assert (r.heads, r.dim, r.vdim, r.tau, r.rank) == (3, 20, 28, 4.0, None) and c.layers[0].mlp.ff == 44
    s, f = c.layers[1].mixer, c.layers[1].mlp
    assert (s.heads, s.vdim, s.state, s.groups, s.conv, s.norm_groups) == (6, 10, 12, 3, 3, 4)
    assert (f.experts, f.top, f.ff, f.identity, f.groups, f.keep, f.shared_ff) == (7, 3, 20, 2, 3, 2, 12)
    b, f = c.layers[2].mixer.left, c.layers[2].mlp
    assert (b.chunk, b.rot_dims) == (0, 0) and (f.identity, f.groups, f.keep, f.shared_ff) == (0, 1, 1, 0) and c.layers[3].mlp is None
    c.with_shapes({"l0.mix.right.a1": (5, 52), "l2.mix.right.a1": (16, 52), "embed": (83, 52)})
    assert [c.layers[i].mixer.right.rank for i in (0, 2)] == [5, 16]
    with pytest.raises(ValueError, match="rank"):
        c.with_shapes({"l0.mix.right.a1": (6, 52)})
    left, right = lambda d: d["layers"][0]["mixer"]["left"], lambda d: d["layers"][0]["mixer"]["right"]
    ssm, moe = lambda d: d["layers"][1]["mixer"], lambda d: d["layers"][1]["mlp"]
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="other"), lambda d: left(d).update(kv_heads=4),
                   lambda d: left(d).update(vdim=16), lambda d: left(d)["mask"].update(size=0), lambda d: left(d)["rot"].update(dims=7),
                   lambda d: left(d)["rot"].update(dims=14), lambda d: left(d)["rot"]["scaling"].update(factor=0.0), lambda d: right(d).update(tau=0.0),
                   lambda d: left(d).update(window=8), lambda d: right(d).update(conv=4), lambda d: ssm(d).update(groups=4), lambda d: ssm(d).update(norm_groups=7),
                   lambda d: ssm(d).update(conv=0), lambda d: moe(d)["router"].update(top=7), lambda d: moe(d)["router"]["groups"].update(count=2),
                   lambda d: moe(d)["router"]["groups"].update(keep=4), lambda d: moe(d)["router"].update(scale=2.0), lambda d: moe(d)["expert"].update(limit=7.0),
                   lambda d: d["embedding"].update(scale=2.0), lambda d: d.update(softcap=30.0), lambda d: d["embedding"]["bigram"].update(buckets=0)):
        d = json.loads(json.dumps(P.file_config(config())))
        change(d)
        with pytest.raises(ValueError):
            HybridDecoderConfig.from_dict(d)
    d = P.file_config(config())
    d["layers"][0]["mixer"]["left"].update(window=None)     # says that there is none
    d["embedding"] = {}
    assert HybridDecoderConfig.from_dict(d).bigram is None
    del d["residual_mult"]
    with pytest.raises(KeyError):
        HybridDecoderConfig.from_dict(d)


def test_registry_knows_the_design():
    assert "Moponex" in registry.architectures()
    model = registry.build_model("Moponex", config_dict=P.with_ranks(config()), dtype=torch.float32)
    assert isinstance(model, HybridDecoder) and isinstance(model, LayeredDecoder) and isinstance(model, GenerationModel)
    assert model.head is model.embed and isinstance(model.layers[1].mlp, RoutedExperts)
    with pytest.raises(ValueError, match="rank"):
        registry.build_model("Moponex", config_dict=P.file_config(config()), dtype=torch.float32)


def test_padding_of_heads():
    assert chunk_heads(48, 48, torch.bfloat16) == (64, 48) and chunk_heads(65, 130, torch.bfloat16) == (128, 136)
    assert chunk_heads(129, 8, torch.bfloat16) is None and chunk_heads(8, 8, torch.float32) is None and chunk_heads(8, 8, torch.float16) is None
    m = registry.build_model("Moponex", config_dict=P.with_ranks(config()), dtype=torch.bfloat16)
    assert (m.layers[0].mixer.left.dk, m.layers[0].mixer.right.dk, m.layers[0].mixer.right.dv) == (64, 64, 32)
    assert (m.layers[1].mixer.dk, m.layers[1].mixer.dv) == (64, 64)         # (two heads of 64 columns share a tile)
    m = registry.build_model("Moponex", config_dict=P.with_ranks(config()), dtype=torch.float32)
    assert (m.layers[0].mixer.left.dk, m.layers[0].mixer.right.dk, m.layers[0].mixer.right.dv, m.layers[1].mixer.dk, m.layers[1].mixer.dv) == (16, 24, 32, 16, 16)
    assert torch.allclose(m.layers[0].mixer.left.freq, torch.tensor([100.0 ** (-2 * i / 8) / 3 for i in range(4)])) and m.layers[2].mixer.left.freq.numel() == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_parameters_in_kernel_layout_hold_the_checkpoint(tmp_path, dtype):
    cfg = config()
    t = P.make_tensors(cfg, 3)
    T.save_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(P.file_config(cfg)))
    model = registry.load_model(str(tmp_path), dtype=dtype, device="cpu")
    f = lambda name: t[name].float()
    g = torch.Generator().manual_seed(1)
    W, w = model.hidden_size, cfg["width"]
    h = torch.zeros(4, W)
    h[:, :w] = torch.randn(4, w, generator=g)
    hs = h[:, :w]
    close = lambda a, b: torch.allclose(a, b, atol=3e-5)

    def heads(y, n, padded, dim):
        y = y.reshape(*y.shape[:-1], n, padded)
        assert float(y[..., dim:].abs().sum()) == 0
        return y[..., :dim].reshape(*y.shape[:-2], -1)

    def into(out_proj, n, padded, dim, name):
        z = torch.zeros(4, n, padded)
        z[..., :dim] = torch.randn(4, n, dim, generator=g)
        assert close((z.view(4, -1) @ out_proj.float().T)[:, :w], z[..., :dim].reshape(4, -1) @ f(name).T)
    assert torch.equal(model.embed[:83, :w].float(), f("embed")) and torch.equal(model.bigram[:, :w].float(), f("bigram")) and model.head.data_ptr() == model.embed.data_ptr()
    for i, ly in enumerate(cfg["layers"]):
        blk, m, p = model.layers[i], ly["mixer"], f"l{i}."
        at = blk.mixer
        y = h @ at.in_proj.float().T
        if isinstance(at, StateSpace):
            H, dim, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            want = (hs @ f(p + "mix.in").T).split([H * dim, H * dim, G * N, G * N, H], 1)
            parts = y.split([at.inner, at.inner, G * at.dk, G * at.dk, at.in_proj.shape[0] - at.tail], 1)
            for got, ref, n, pad, d in zip(parts, want, (H, H, G, G), (at.dv, at.dv, at.dk, at.dk), (dim, dim, N, N)):
                assert close(heads(got, n, pad, d), ref)
            assert close(parts[4][:, :H], want[4]) and float(parts[4][:, H:].abs().sum()) == 0
            for got, ref in zip(at.conv_w.float().split([at.inner, G * at.dk, G * at.dk], 1), f(p + "mix.conv").split([H * dim, G * N, G * N])):
                n, pad, d = (H, at.dv, dim) if got.shape[1] == at.inner and ref.shape[0] == H * dim else (G, at.dk, N)
                assert torch.equal(heads(got, n, pad, d), ref.T)
            for got, name in ((at.dt_bias, "dt_bias"), (at.a_log, "A_log"), (at.skip, "D")):
                assert got.dtype == torch.float32 and torch.equal(got, f(p + "mix." + name))
            assert torch.equal(heads(at.norm.float(), H, at.dv, dim), f(p + "mix.norm"))
            into(at.out_proj, H, at.dv, dim, p + "mix.o")
        else:
            a, r, L, R = m["left"], m["right"], at.left, at.right
            y = y + at.bias.float()
            q, k = y[:, :L.columns].split([L.heads * L.dk, L.kv_heads * L.dk], 1)
            for got, name, n in ((q, "q", a["heads"]), (k, "k", a["kv_heads"])):
                assert close(heads(got, n, L.dk, a["dim"]), hs @ f(f"{p}mix.left.{name}").T + f(f"{p}mix.left.{name}.b"))
            for got, name, pad, d in zip(y[:, L.columns:].split(R.splits, 1), "qkvg", (R.dk, R.dk, R.dv, R.dv), (r["dim"], r["dim"], r["vdim"], r["vdim"])):
                assert close(heads(got, r["heads"], pad, d), hs @ f(f"{p}mix.right.{name}").T)
            low = y[:, L.columns:].split(R.splits, 1)[4]
            assert close(heads(low @ R.a2.float().T + R.a2_bias.float(), r["heads"], R.dk, r["dim"]),
                         (hs @ f(p + "mix.right.a1").T) @ f(p + "mix.right.a2").T + f(p + "mix.right.a2.b"))
            assert torch.equal(L.sinks, f(p + "mix.left.sink")) and torch.equal(L.q_norm[:a["dim"]].float(), f(p + "mix.left.q.norm"))
            assert torch.equal(heads(R.norm.float(), r["heads"], R.dv, r["vdim"]), f(p + "mix.right.norm").repeat(r["heads"]))
            for got, name in ((at.left_out, "left"), (at.right_out, "right")):
                assert got.dtype == torch.float32 and torch.equal(got[:w] * 2, f(f"{p}mix.{name}.out"))
            into(at.left_proj, a["heads"], L.dk, a["dim"], p + "mix.left.o")
            into(at.right_proj, r["heads"], R.dv, r["vdim"], p + "mix.right.o")
        f_ = ly["mlp"]
        if f_ is None:
            assert blk.mlp is None and blk.norm2 is None
        elif f_["kind"] == "dense":
            u = (h @ blk.mlp.gate_up.float().T).view(4, -1, 2, 8)
            for j, name in enumerate(("gate", "up")):
                assert close(u[:, :, j].reshape(4, -1)[:, :f_["ff"]], hs @ f(f"{p}mlp.{name}").T)
            into(blk.mlp.down, 1, blk.mlp.ff_padded, f_["ff"], p + "mlp.down")
        else:
            n, E = blk.mlp.choices, blk.mlp.experts
            z = h @ blk.mlp.router.float().T
            assert close(z[:, :n], hs @ f(p + "mlp.router").T) and torch.equal(blk.mlp.correction, f(p + "mlp.correction"))
            if blk.mlp.gated:
                assert close(z[:, n:n + 1], hs @ f(p + "mlp.shared.sg").T) and close((h @ blk.mlp.shared_up.float().T)[:, :12], hs @ f(p + "mlp.shared.up").T)
                into(blk.mlp.shared_down, 1, blk.mlp.shared_padded, 12, p + "mlp.shared.down")
            for e in range(E):
                assert close((h @ blk.mlp.up[e].float().T)[:, :blk.mlp.ff], hs @ f(f"{p}mlp.e{e}.up").T)
                into(blk.mlp.down[e], 1, blk.mlp.ff_padded, blk.mlp.ff, f"{p}mlp.e{e}.down")


def test_checkpoint_conversion_complains_about_missing_surplus_and_misshapen_tensors():
    cfg = config()
    t = P.make_tensors(cfg, 3)
    model = registry.build_model("Moponex", config_dict=P.with_ranks(cfg), dtype=torch.float32)
    processing_Moponex(t, model)
    for name in ("bigram", "l0.mix.left.sink", "l1.mix.conv.b", "l1.mlp.shared.sg", "l2.mlp.e4.down", "l0.mix.right.a2.b"):
        with pytest.raises(KeyError, match="lacks"):
            processing_Moponex({k: v for k, v in t.items() if k != name}, model)
    with pytest.raises(KeyError, match="l3.norm2"):
        processing_Moponex(dict(t, **{"l3.norm2": t["l0.norm1"]}), model)
    with pytest.raises(ValueError, match="l1.mix.in"):
        processing_Moponex(dict(t, **{"l1.mix.in": t["l1.mix.in"][:-1]}), model)


def test_state_of_every_kind_is_prepared_kept_and_forked():
    m = registry.build_model("Moponex", config_dict=P.with_ranks(config()), dtype=torch.float32)
    s = m.new_state()
    assert isinstance(s, SequenceState)
    kinds = {k: type(c) for k, c in s.caches.items()}
    assert kinds == {(0, "keys"): RingCache, (0, "state"): RecurrentState, (1, "conv"): RingCache, (1, "state"): RecurrentState, (2, "keys"): RingCache,
                     (2, "state"): RecurrentState, (3, "conv"): RingCache, (3, "state"): RecurrentState, "last token": RecurrentState}
    assert (s.caches[0, "keys"].window, s.caches[2, "keys"].window, s.caches[1, "conv"].window, s.caches[1, "conv"].width) == (9, 0, 3, 6 * 16 + 2 * 3 * 16)
    dev = torch.device("cpu")
    s.begin([2, 0, 1], 20, 5, torch.float32, dev)
    assert s.caches[0, "keys"].buf.shape[1] == 9 and s.caches[1, "conv"].buf.shape[1] == 3 and s.capacity() == 25
    last = s.caches["last token"].tensors[0]
    assert last.dtype == torch.int64 and last.shape == (3,)
    last.copy_(torch.tensor([5, 6, 7]))
    two = s.fork([1])
    s.keep([0, 2])
    assert two.caches["last token"].tensors[0].tolist() == [6] and s.caches["last token"].tensors[0].tolist() == [5, 7]
    two.caches["last token"].tensors[0].fill_(9)
    assert s.caches["last token"].tensors[0].tolist() == [5, 7]
    s.begin([0], 2, 0, torch.float32, dev)                   # shorter than the rings: they grow
    assert s.caches[1, "conv"].buf.shape[1] == 2 and s.capacity() == 2
    s.ensure(3)
    assert s.caches[1, "conv"].buf.shape[1] == 3 and s.capacity() >= 3


def test_units():
    assert unit_code(None, None) == (0, 0.0, 0.0, 1) and unit_code(None, (7.0, 1.7)) == (1, 7.0, 1.7, 2)
    assert unit_code("geglu", None)[::3] == (2, 2) and unit_code("gelu", None)[::3] == (3, 1)


def test_plain_restatement_on_known_answers():
    """The equations by other means: closed forms, torch's own functions, step-by-step sums."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    z = r(50)
    assert torch.allclose(P.gelu_erf(z), torch.nn.functional.gelu(z)) and torch.allclose(P.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert P.bigram_rows([3, 5, 0], 10, 3, 7) == [7, (30 + 15) % 7, 50 % 7]
    x, w, b = r(9, 4), r(4, 3), r(4)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T[None], (2, 0)), w[:, None], b, groups=4)[0].T
    assert torch.allclose(P.short_conv(x, w, b), ref)
    # one step size and decay for all: a geometric sum
    n, H, N, V = 6, 2, 3, 4
    xx, B, C, dt = r(n, H, V), r(n, 1, N), r(n, 1, N), torch.full((n, H), 0.5, dtype=torch.float64)
    y, S = P.ssm_scan(xx, B, C, dt, torch.zeros(H, dtype=torch.float64), torch.ones(H, dtype=torch.float64))
    want = xx[-1] + sum(torch.exp(torch.tensor(-0.5 * (n - 1 - s))) * 0.5 * (B[s, 0] @ C[-1, 0]) * xx[s] for s in range(n))
    assert torch.allclose(y[-1], want)
    o, _ = P.gla_scan(r(4, 1, N), k := r(4, 1, N), v := r(4, 1, V), torch.zeros(4, 1, N, dtype=torch.float64))
    assert torch.allclose(P.gla_scan(torch.ones(4, 1, N, dtype=torch.float64), k, v, torch.zeros(4, 1, N, dtype=torch.float64))[0][-1],
                          (k.sum(-1, keepdim=True) * v).sum(0))
    # rotations keep lengths and depend on distances alone
    q, k = r(1, 1, 8).expand(10, 1, 8), r(1, 1, 8).expand(10, 1, 8)
    a, c = P.rotate(q, range(10), 6, 50.0, 2.0), P.rotate(k, range(10), 6, 50.0, 2.0)
    assert torch.allclose(a.norm(dim=-1), q.norm(dim=-1)) and torch.allclose((a[7] * c[4]).sum(), (a[5] * c[2]).sum()) and torch.equal(a[..., 6:], q[..., 6:])
    seen = P.chunk_mask(7, 3)
    assert [int(v) for v in seen.sum(-1)] == [1, 2, 3, 1, 2, 3, 1] and bool(seen[5, 3]) and not bool(seen[3, 2])
    # a sink of minus infinity is none; of the size of the only score it takes half
    one = P.sink_attention(q[:1], k[:1], k[:1], 0.3, torch.tensor([float((q[0] * k[0]).sum()) * 0.3], dtype=torch.float64), P.chunk_mask(1, None))
    assert torch.allclose(one, k[:1] / 2)
    # choices: a group whose best is hidden by the correction stays closed; negative choice scores compete
    zz = torch.log(torch.tensor([[0.4, 0.1, 0.3, 0.2]], dtype=torch.float64))
    idx, w = P.choose(zz, torch.tensor([-1.0, -1.0, -1.0, -0.5], dtype=torch.float64), 2, 2, 1)
    assert idx == [[3, 2]] and torch.allclose(w[0], torch.tensor([0.4, 0.6], dtype=torch.float64))


def test_kernels_validate_before_any_cuda_call():
    L = _lib.lib()
    buf = ctypes.create_string_buffer(64)
    a = (ctypes.addressof(buf) + 15) & ~15
    B16, F16, F32 = _lib.BF16, _lib.F16, _lib.F32
    err = _lib.last_error
    conv = lambda C=8, taps=4, ring=a: L.eb_short_conv(a, 8, a, a, a, 8, 1, 4, C, taps, None, ring, 32, 8, 4, B16, None)
    assert conv(C=12) == -1 and conv(taps=0) == -1 and conv(ring=None) == -1
    scan = lambda fn, dk=64, dv=8, groups=1, dtype=B16: fn(a, 1 << 12, a, 2, a, a, a, None, a, 1 << 12, a, 1, 1, 2, groups, dk, dv, dtype, None)
    assert scan(L.eb_ssm_scan, dk=12) == -1 and scan(L.eb_ssm_scan, groups=3) == -1 and "share" in err()
    assert scan(L.eb_ssm_chunks, dk=96) == -1 and "64 or 128" in err() and scan(L.eb_ssm_chunks, dtype=F16) == -1 and "bf16" in err()
    gla = lambda dk=64, tau=1.0, dtype=B16, ws=None: L.eb_gla_chunks(a, a, a, 64, a, 128, tau, 1.0, None, a, 16, a, 1, 1, 2, dk, 8, dtype, ws, 0, None)
    assert gla(dk=32) == -1 and gla(tau=0.0) == -1 and "tau" in err() and gla(dtype=F32) == -1 and gla() == -1 and "workspace" in err()
    assert L.eb_gla_chunks_workspace_bytes(2, 130, 3, 64) == 260 * 3 * (192 + 128) * 2 + 2 * 2 * 3 * 64 * 4 + 16
    assert L.eb_gla_scan(a, a, a, 64, a, 128, 0.0, 1.0, None, a, 16, a, 1, 1, 2, 64, 8, F32, None) == -1
    step = lambda taps=4, groups=1, dk=8: L.eb_ssm_step(a, 64, a, a, taps, a, 256, 64, 4, a, None, a, 2, a, a, a, a, 16, a, 1, 2, groups, dk, 8, B16, None)
    assert step(taps=0) == -1 and step(groups=3) == -1 and step(dk=12) == -1
    gstep = lambda rank=8, tau=1.0, count=8: L.eb_gla_step(a, a, a, a, a, 64, a, a, rank, tau, 1.0, a, count, 1e-5, a, 8, a, 1, 1, 8, 8, B16, None)
    assert gstep(rank=12) == -1 and gstep(tau=0.0) == -1 and gstep(count=9) == -1
    norm = lambda dv=8, pad=8, parts=1: L.eb_gate_group_norm(a, 64, a, 64, a, 1e-5, a, 64, 1, 3, dv, pad, parts, B16, None)
    assert norm(dv=9) == -1 and norm(pad=12) == -1 and norm(parts=5) == -1 and "equal parts" in err()
    rot = lambda dk=8, count=8, pairs=4, freq=a: L.eb_attention_rotary(a, 32, 1, 1, dk, count, a, a, 1e-5, freq, pairs, a, 8, None, 0, a, 64, 8, a, 64, 8, 4, 1, 1, None, None, B16, None)
    assert rot(dk=12) == -1 and rot(count=6) == -1 and rot(freq=None) == -1
    pre = lambda group=1, chunk=4, scale=0.1: L.eb_attention_prefill_chunk_tc(a, a, a, a, *[64] * 8, 1, 2, group, 8, 64, chunk, None, a, scale, B16, None)
    assert pre(group=3) == -1 and pre(chunk=-1) == -1 and pre(scale=0.0) == -1
    dec = lambda chunk=4, kv=2, nsplit=1: L.eb_attention_group_decode_chunk(a, a, a, a, 256, 640, 128, 640, 128, 256, 1, 4, kv, 64, 5, chunk, a, None, a, 1.0, B16, nsplit, None, 0, None)
    assert dec(chunk=-1) == -1 and dec(kv=3) == -1 and dec(nsplit=2) == -1
    assert L.eb_attention_plain_chunk(a, a, a, a, *[8] * 12, 1, 2, 1, 1, 8, 8, -1, 4, None, None, None, 1.0, F32, None) == -1
    route = lambda n=9, E=8, top=2, groups=3, keep=2, ld=16: L.eb_moe_route_rule(a, ld, 1, n, E, top, None, groups, keep, None, 0, a, a, None, None, a, None)
    assert route(groups=2) == -1 and route(keep=4) == -1 and route(top=7) == -1 and "open choices" in err() and route(E=10) == -1 and route(ld=9) == -1
    add = lambda **k: L.eb_stream_add(k.get("src"), 8, k.get("src2"), 8, k.get("y"), 8, k.get("w"), k.get("y2"), 8, k.get("w2"), k.get("idx"), None, a, 1, 2, k.get("ident"), 8,
                                      k.get("shared"), 8, k.get("gate"), 1.0, a, 8, k.get("wn"), 1.0, k.get("h"), 8, 1e-5, 1, k.get("n2", 8), 8, k.get("router"), 4, 4, 1, None,
                                      1, 1, None, None, None, B16, None)
    assert add() == -1 and add(src2=a, y=a) == -1 and add(y=a, y2=a) == -1 and add(y=a, w=a) == -1 and add(y=a, idx=a) == -1 and "mixture" in err()
    assert add(y=a, idx=a, ident=a, shared=a) == -1 and "gate" in err() and add(wn=a) == -1 and add(src=a, n2=12) == -1 and add(y=a, router=a) == -1
    assert L.eb_gemm_gated(a, 8, a, 8, a, 8, 4, 24, 8, 2, 0.0, 0.0, B16, 0, None, 0, None) == -1 and "multiple of 16" in err()
    assert L.eb_gemm_gated(a, 8, a, 8, a, 8, 4, 16, 8, 3, 0.0, 0.0, B16, 0, None, 0, None) == -1 and L.eb_unit_act(a, 16, a, 8, 1, 8, 4, 0.0, 0.0, F32, None) == -1
    assert L.eb_gemm_grouped(a, 8, a, 8, a, 8, 128, 16, 8, 1, a, a, 4, 0.0, 0.0, B16, None) == -1
    assert L.eb_grouped_skinny(a, 8, 0, 1, a, 128, 8, a, 16, 0, None, 1, 1, 16, 8, 4, 0.0, 0.0, B16, None) == -1
    big = lambda **k: L.eb_greedy_step_bigram(a, 8, 1, 8, F32, a, 4, 4, None, a, k.get("emb", a), 0, 8, None, 0, 0, 8, B16, a, 8, a, k.get("pair", a), k.get("rows", 5), 3, 7,
                                              k.get("out", a), 8, None)
    assert big(pair=None) == -1 and big(out=None) == -1 and big(rows=0) == -1 and big(emb=None) == -1
