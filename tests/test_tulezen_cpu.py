"""Host-side logic of the latent-attention decoder: configuration, registry, checkpoint reader and
parameter layouts, cache and sequence state, trace sessions, argument validation of its kernels."""
import json

import pytest
import torch

import tulezen_plain as P
from energonai_b200 import _lib, registry
from energonai_b200.attention import pick_latent_nsplit
from energonai_b200.model import GenerationModel, LatentDecoder, LatentDecoderConfig, PipelineModel, RingCache, SequenceState
from energonai_b200.trace import TraceSession
from energonai_b200.utils import load_checkpoint, load_safetensors, load_state_dict, processing_Tulezen

LAYERS = [dict(heads=3, dim=20, vdim=28, rank=40, window=9, scale=0.3, moe=(5, 2, 12, 0.7)),
          dict(heads=2, dim=8, vdim=8, rank=24, window=33, scale=0.5, moe=None),
          dict(heads=5, dim=12, vdim=4, rank=40, window=70, scale=0.2, kv_from=0, moe=(3, 3, 20, 1.5))]


def config():
    return P.make_config(LAYERS, width=76, vocab=101)


def test_configuration_reads_every_size_and_rejects_what_it_does_not_know():
    c = LatentDecoderConfig.from_dict(config())
    assert (c.vocab, c.width, c.eps, len(c.layers)) == (101, 76, 3e-5, 3)
    m = c.layers[2].mixer
    assert (m.heads, m.dim, m.vdim, m.kv_rank, m.window, m.scale, m.kv_from) == (5, 12, 4, 40, 70, 0.2, 0)
    f = c.layers[2].mlp
    assert (f.experts, f.top, f.ff, f.limit, f.alpha) == (3, 3, 20, 1.5, 1.702)
    assert c.layers[1].mlp is None
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="dense"),
                   lambda d: d["layers"][2]["mixer"].update(kv_from=2), lambda d: d["layers"][2]["mixer"].update(kv_from=1),
                   lambda d: d["layers"][0]["mixer"]["mask"].update(size=0)):
        d = json.loads(json.dumps(config()))
        change(d)
        with pytest.raises(ValueError):
            LatentDecoderConfig.from_dict(d)
    d = config()
    del d["layers"][0]["mixer"]["scale"]
    with pytest.raises(KeyError):
        LatentDecoderConfig.from_dict(d)


def test_registry_knows_the_design_and_the_other_models():
    assert "Tulezen" in registry.architectures() and {"opt_125M", "gpt2_small", "bert_small", "Tulezen"} <= set(registry.models())
    model = registry.build_model("Tulezen", config_dict=config(), dtype=torch.float32)
    assert isinstance(model, LatentDecoder) and isinstance(model, GenerationModel) and issubclass(PipelineModel, GenerationModel)
    with pytest.raises(KeyError):
        registry.build_model("nothing")


def test_load_model_refuses_an_unknown_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Elsewhere"}))
    with pytest.raises(ValueError, match="not registered"):
        registry.load_model(str(tmp_path), device="cpu")


def test_safetensors_reader(tmp_path):
    t = {"a": torch.arange(6, dtype=torch.int32).view(2, 3), "b": torch.randn(3, 5).bfloat16(), "c": torch.randn(7), "e": torch.empty(0, 4)}
    path = str(tmp_path / "x.safetensors")
    P.save_safetensors(path, t)
    got = load_safetensors(path)
    assert got.keys() == t.keys() and all(torch.equal(got[k], t[k]) and got[k].dtype == t[k].dtype for k in t)
    (tmp_path / "config.json").write_text("{}")
    assert load_state_dict(str(tmp_path)).keys() == t.keys()          # a folder: its *.safetensors
    with open(path, "r+b") as f:
        f.truncate(40)
    with pytest.raises(ValueError):
        load_safetensors(path)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_parameters_in_kernel_layout_hold_the_checkpoint(tmp_path, dtype):
    """Every projection applied through the packed, padded parameters equals the checkpoint's."""
    cfg = config()
    t = P.make_tensors(cfg, 3)
    P.save_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    model = registry.load_model(str(tmp_path), dtype=dtype, device="cpu")
    g = torch.Generator().manual_seed(1)
    h = torch.zeros(4, model.hidden_size)
    h[:, :76] = torch.randn(4, 76, generator=g)
    f = lambda name: t[name].float()
    for i, ly in enumerate(LAYERS):
        at, p = model.layers[i].mixer, f"l{i}.mix."
        H, d, dv, r = ly["heads"], ly["dim"], ly["vdim"], ly["rank"]
        y = h @ at.in_proj.float().T
        q = y[:, :at.q_rows].view(4, H, at.dk)
        assert torch.allclose(q[..., :d].reshape(4, -1), h[:, :76] @ f(p + "q").T, atol=1e-5) and float(q[..., d:].abs().sum()) == 0
        if ly.get("kv_from") is None:
            c = y[:, at.q_rows:]
            assert torch.allclose(c[:, :r], h[:, :76] @ f(p + "dkv").T, atol=1e-5) and float(c[:, r:].abs().sum()) == 0
        c = torch.zeros(4, at.rank)
        c[:, :r] = torch.randn(4, r, generator=g)
        kv = c @ at.kv_up.float().T
        k, v = kv[:, :at.q_rows].view(4, H, at.dk), kv[:, at.q_rows:].view(4, H, at.dv)
        assert torch.allclose(k[..., :d].reshape(4, -1), c[:, :r] @ f(p + "uk").T, atol=1e-5)
        assert torch.allclose(v[..., :dv].reshape(4, -1), c[:, :r] @ f(p + "uv").T, atol=1e-5)
        # absorbed keys: (W_uk^T q) . c = q . (W_uk c)
        qa = torch.einsum("thd,hrd->thr", q, at.k_absorb.float())
        assert torch.allclose(torch.einsum("thr,tr->th", qa, c), torch.einsum("thd,thd->th", q, k), atol=1e-4)
        o = torch.zeros(4, H, at.dv)
        o[..., :dv] = torch.randn(4, H, dv, generator=g)
        z = o.view(4, -1) @ at.out_proj.float().T
        assert torch.allclose(z[:, :76], o[..., :dv].reshape(4, -1) @ f(p + "o").T, atol=1e-5) and float(z[:, 76:].abs().sum()) == 0
        mlp = model.layers[i].mlp
        assert (mlp is None) == (ly["moe"] is None)
        for e in range(ly["moe"][0] if ly["moe"] else 0):
            gu = (h @ mlp.gate_up[e].float().T).view(4, -1, 2, 8)
            for n, name in enumerate(("gate", "up")):
                x = gu[:, :, n].reshape(4, -1)
                assert torch.allclose(x[:, :ly["moe"][2]], h[:, :76] @ f(f"l{i}.mlp.e{e}.{name}").T, atol=1e-5)
                assert float(x[:, ly["moe"][2]:].abs().sum()) == 0


def test_checkpoint_conversion_complains_about_missing_surplus_and_misshapen_tensors():
    cfg = config()
    t = P.make_tensors(cfg, 3)
    model = registry.build_model("Tulezen", config_dict=cfg, dtype=torch.float32)
    processing_Tulezen(t, model)
    with pytest.raises(KeyError, match="lacks"):
        processing_Tulezen({k: v for k, v in t.items() if k != "l0.mix.uv"}, model)
    with pytest.raises(KeyError, match="l2.mix.dkv"):
        processing_Tulezen(dict(t, **{"l2.mix.dkv": t["l0.mix.dkv"]}), model)
    with pytest.raises(ValueError, match="l1.mix.q"):
        processing_Tulezen(dict(t, **{"l1.mix.q": t["l1.mix.q"][:-1]}), model)


def test_left_padding_is_read_from_the_mask_and_other_masks_are_refused():
    assert LatentDecoder.left_padding(torch.tensor([[0, 0, 1, 1], [1, 1, 1, 1]])) == [2, 0]
    for bad in ([[1, 1, 0, 0]], [[0, 1, 0, 1]], [[0, 0, 0, 0]]):
        with pytest.raises(ValueError):
            LatentDecoder.left_padding(torch.tensor(bad))


def test_cache_is_a_ring_as_long_as_the_longest_window_of_its_readers():
    model = registry.build_model("Tulezen", config_dict=config(), dtype=torch.float32)
    caches = model.state.caches
    assert sorted(caches) == [0, 1] and caches[0].window == 70 and caches[1].window == 33
    s = model.new_state()
    s.begin([0, 3], 20, 5, torch.float32, torch.device("cpu"))
    assert [tuple(s.caches[i].buf.shape) for i in (0, 1)] == [(2, 25, 40), (2, 25, 24)]
    assert s.capacity() == 25 and s.padded and s.first.tolist() == [0, 3] and s.kv_state.tolist() == [20, 21]
    s.caches[0].buf[:, :20] = 1.0
    s.set_length(25)
    s.ensure(26)                                            # grows, never beyond the window
    assert s.caches[0].buf.shape[1] == 70 and s.caches[1].buf.shape[1] == 33 and s.capacity() is None
    assert float(s.caches[0].buf[:, :20].min()) == 1.0 and float(s.caches[0].buf[:, 25:].abs().sum()) == 0.0
    before = s.caches[1].buf.data_ptr()
    s.begin([0, 0], 40, 5, torch.float32, torch.device("cpu"))
    assert not s.padded and s.caches[1].buf.data_ptr() == before and s.caches[1].buf.shape[1] == 33    # memory used again


def test_state_keeps_and_forks_sequences():
    s = SequenceState({0: RingCache(8, 4)})
    s.begin([2, 0, 1], 6, 3, torch.float32, torch.device("cpu"))
    s.caches[0].buf.copy_(torch.arange(3.)[:, None, None].expand_as(s.caches[0].buf))
    two = s.fork([1])
    s.keep([0, 2])
    assert two.batch == 1 and two.first.tolist() == [0] and float(two.caches[0].buf.mean()) == 1.0
    assert s.batch == 2 and s.first.tolist() == [2, 1] and s.caches[0].buf[:, 0, 0].tolist() == [0.0, 2.0]
    s.advance()
    assert s.kv_state.tolist() == [7, 8] and two.kv_state.tolist() == [6, 7] and s.length == 7 and two.length == 6


class FakeModel:
    """Logits that name the sequence (sum of its tokens so far) and the place."""
    vocab = 50

    class State:
        def __init__(self):
            self.sums = []

        def keep(self, rows):
            self.sums = [self.sums[r] for r in rows]

        def fork(self, rows):
            out = FakeModel.State()
            out.sums = [self.sums[r] for r in rows]
            return out

    def new_state(self):
        return FakeModel.State()

    def prompt(self, ids, mask, reserve=0):
        run = (ids * mask).cumsum(1)
        self.state.sums = run[:, -1].tolist()
        return run.reshape(-1, 1).float()

    def step(self, tokens):
        self.state.sums = [s + int(t) for s, t in zip(self.state.sums, tokens)]
        return torch.tensor(self.state.sums, dtype=torch.float32)[:, None]

    def logits(self, x):
        return x


def test_trace_session_batches_splits_and_ends_requests():
    s = TraceSession(FakeModel(), torch.device("cpu"))
    run = lambda entries, end=(): s.run([dict(id=i, tokens=t, want=w) for i, t, w in entries], list(end))
    assert run([("x", [1, 2, 3], [0, 2]), ("y", [9], [0])]).flatten().tolist() == [1, 6, 9]
    assert run([("y", [4], [0]), ("x", [1], [0])]).flatten().tolist() == [13, 7]        # any order
    assert run([("z", [5, 5], [1])]).flatten().tolist() == [10]                        # another batch beside it
    assert run([("z", [1], [])]) is None
    assert run([("x", [2], [0])]).flatten().tolist() == [9]                             # part of a batch goes on
    assert run([("z", [1], [0]), ("x", [1], [0]), ("y", [1], [0])], ["x"]).flatten().tolist() == [12, 10, 14]
    assert run([("y", [1], [0])], ["y", "z"]).flatten().tolist() == [15]
    assert s.batches == []
    assert run([("x", [7], [0])]).flatten().tolist() == [7]                             # a name that is used again
    for entries in ([("x", [1, 1], [])], [("x", [1], []), ("new", [1], [])], [("n", [], [])], [("n", [50], [])], [("n", [1], [1])]):
        with pytest.raises(ValueError):
            run(entries)


def test_latent_split_rule():
    assert pick_latent_nsplit(16, 16, 4096) == 9 and pick_latent_nsplit(64, 16, 4096) == 2
    assert pick_latent_nsplit(1, 1, 64) == 1 and pick_latent_nsplit(200, 64, 4096) == 1
    assert pick_latent_nsplit(1, 16, 1 << 20) == 64


def test_kernels_validate_before_any_cuda_call():
    import ctypes
    L = _lib.lib()
    buf = ctypes.create_string_buffer(64)
    a = (ctypes.addressof(buf) + 15) & ~15
    B16, F32 = _lib.BF16, _lib.F32
    assert L.eb_rms_norm(a, 8, F32, a, 0.0, 1e-5, a, 8, B16, 0, 8, 8, None, 0, 0, 0, 1, None, None) == 0
    assert L.eb_rms_norm(a, 8, F32, a, 0.0, 1e-5, a, 8, B16, 2, 12, 8, None, 0, 0, 0, 1, None, None) == -1 and "multiple of 8" in _lib.last_error()
    assert L.eb_rms_norm(a, 8, _lib.F16, a, 0.0, 1e-5, a, 8, B16, 2, 8, 8, None, 0, 0, 0, 1, None, None) == -1
    assert L.eb_rms_residual(a, 8, B16, a, None, None, 0, a, 1.0, 1e-5, a, 8, None, 0, 1, 8, 8, None, 0, 0, None, None, None) == -1
    assert "weights" in _lib.last_error()
    assert L.eb_moe_route(a, 4, 1, 4, 5, None, 0, a, a, None, None, None) == -1
    assert L.eb_moe_plan(None, 4, a, a, 1, a, None) == -1
    assert L.eb_gemm_grouped(a, 8, a, 8, a, 8, 64, 16, 8, 1, a, a, 0, 0.0, 0.0, B16, None) == -1 and "whole tiles" in _lib.last_error()
    assert L.eb_gemm_grouped(a, 8, a, 8, a, 8, 128, 24, 8, 1, a, a, 1, 1.0, 1.0, B16, None) == -1
    assert L.eb_grouped_skinny(a, 8, 0, 1, a, 8, 8, a, 8, 0, None, 1, 1, 8, 12, 0, 0.0, 0.0, B16, None) == -1
    assert L.eb_gemm_f32(a, 4, 0, a, 8, 0, a, 8, 0, 1, 8, 8, 1, None, None, None, 0, None, None) == -1
    latent = lambda rank=64, dtype=B16, nsplit=1: L.eb_latent_decode(a, 64, a, 640, 64, 10, a, 64, 1, 1, rank, 4, a, None, 1.0, dtype, nsplit,
                                                                     None, 0, None)
    assert latent(rank=96) == -1 and "latent width" in _lib.last_error()
    assert latent(dtype=F32) == -1 and latent(nsplit=3) == -1 and "scratch" in _lib.last_error()
    assert L.eb_latent_decode_scratch_bytes(2, 3, 64, 4) == 0 and L.eb_latent_decode_scratch_bytes(2, 3, 64, 3) == 2 * 3 * 3 * 66 * 4
    assert L.eb_attention_plain(a, a, a, None, *[8] * 12, 1, 1, 1, 1, 8, 8, 0, 4, None, None, None, None, 0, 1.0, F32, None) == -1
    args = [a, a, a, a, None, 64, 64, 64, 64, 64, 64, 64, 64, 0, 1, 1, 8, 8, 64]
    assert L.eb_attention_prefill_window_tc(*args, -1, 0.1, B16, None) == -1 and "window" in _lib.last_error()
