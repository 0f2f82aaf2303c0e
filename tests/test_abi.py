"""The C-ABI library loads and exports every symbol include/ferrite_b200.h declares (no GPU needed)."""
import os
import re

from conftest import ROOT
from ferrite_b200 import _lib


def declared():
    text = open(os.path.join(ROOT, "include", "ferrite_b200.h")).read()
    text = re.sub(r"/\*.*?\*/", "", text, flags=re.S)
    return sorted(set(re.findall(r"\b(fb_[a-z0-9_]+)\s*\(", text)))


def test_every_declared_symbol_is_exported_and_bound():
    lib = _lib.lib()
    names = declared()
    assert "fb_linear" in names and "fb_quantize" in names
    for name in names:
        assert hasattr(lib, name), f"{name} is declared in the header but not exported"
        assert name in _lib.SIGNATURES, f"{name} has no ctypes signature"
    assert sorted(_lib.SIGNATURES) == names, "ctypes signatures without a declaration"


def test_host_side_calls():
    lib = _lib.lib()
    assert lib.fb_version() >= 1
    # ferrite's footprint, 1088 / 576 bytes per 1024 values (ferrite/compiler.py:19-20), in units of 64 x 64
    assert lib.fb_packed_bytes(_lib.BFP8, 64, 64) == 4 * 1088 and lib.fb_packed_bytes(_lib.BFP4, 128, 64) == 8 * 576
    assert lib.fb_packed_bytes(_lib.BFP8, 32, 48) == 4 * 1088, "rows and columns pad to whole units"
    assert lib.fb_packed_bytes(_lib.BFP8, 32, 40) == 0, "columns come in runs of 16"
    # fb_linear's workspace: a zeroed head of 18 KB (arrival words, row scales, counters), then partial tiles and the
    # normalised activations; one row also leaves room for the streaming GEMV's partial sums, a slot per column group
    # and sharing CTA
    head = 18432
    assert lib.fb_linear_workspace_bytes(32, 4096, 4096) >= head + 32 * 4096 * 2
    assert lib.fb_linear_workspace_bytes(1, 4096, 128256) >= head + (128256 // 64) * 2 * 64 * 4


def test_bad_arguments_are_refused_without_a_gpu():
    lib = _lib.lib()
    rc = lib.fb_quantize(_lib.BF16, None, 1, 32, 32, None, None)
    assert rc == -1 and b"block float" in lib.fb_last_error()
    rc = lib.fb_linear(_lib.BFP8, 16, 1, 30, 32, 16, 32, 16, _lib.BF16, 32, None, 1e-5, 0, None, 0, None, 0, None)
    assert rc == -1 and b"multiple of 4" in lib.fb_last_error()
    rc = lib.fb_linear_prefer(7)
    assert rc == -1 and b"unknown kernel" in lib.fb_last_error()
    assert lib.fb_linear_prefer(_lib.LINEAR_AUTO) == 0


def test_new_entry_points_refuse_bad_arguments_without_a_gpu():
    import ctypes
    lib = _lib.lib()
    two = (ctypes.c_void_p * 2)(16, 32)
    rc = lib.fb_peer_reduce_add(two, two, 0, 9, 16, 64, None, 16, None)
    assert rc == -1 and b"up to 8 ranks" in lib.fb_last_error()
    rc = lib.fb_peer_reduce_add(two, two, 0, 2, 16, 60, None, 16, None)
    assert rc == -1 and b"16-byte pieces" in lib.fb_last_error()
    rc = lib.fb_rope_kv_write_packed(_lib.BF16, 16, 1, 256, 2, 1, 64, 16, 16, 64, 8, 16, 16, None, 1e-5, 16, 128, 16, 64, None)
    assert rc == -1 and b"bfp8 or bfp4 cache" in lib.fb_last_error()
    rc = lib.fb_decode_attention_packed(_lib.BFP8, 16, 1, 128, 2, 1, 96, 16, 64, 16, 16, 64, 0, 16, 128, None, 0, None)
    assert rc == -1 and b"64 or 128" in lib.fb_last_error()
    rc = lib.fb_touched(16, 16, 4, 40, 8, 0, 16, 16, None)
    assert rc == -1 and b"up to 32 choices" in lib.fb_last_error()


def test_empty_shapes_need_no_workspace_and_static_attention_refuses_them():
    lib = _lib.lib()
    assert lib.fb_decode_attention_workspace_bytes(0, 8, 2, 128, 64) == 0 and lib.fb_decode_attention_workspace_bytes(4, 8, 0, 128, 64) == 0
    assert lib.fb_attend_workspace_bytes(0, 4, 128, 64) == 0
    rc = lib.fb_decode_attention_static(16, 0, 1024, 8, 2, 128, 16, 64, 8192, 16, 16, 64, 0, 16, 1024, None)
    assert rc == -1 and b"at least one token" in lib.fb_last_error()
    rc = lib.fb_rope_kv_write(16, 1, 256, 2, 1, 48, 16, 16, 48, 8, 16, 16, 16, 1e-5, 16, 96, 16, 64, 64 * 48, None)
    assert rc == -1 and b"multiple of 64" in lib.fb_last_error()


def test_dense_latent_and_decay_entry_points_refuse_bad_arguments_without_a_gpu():
    import ctypes
    lib = _lib.lib()
    rc = lib.fb_dense(16, 4, 60, 64, 0, 16, 32, 64, 0, 1, 16, _lib.BF16, 32, 0, None, 0, None)
    assert rc == -1 and b"multiple of 8" in lib.fb_last_error()
    e = _lib.DenseEpilogue(kind=9)
    rc = lib.fb_dense(16, 4, 64, 64, 0, 16, 32, 64, 0, 1, 16, _lib.BF16, 32, 0, ctypes.byref(e), 0, None)
    assert rc == -1 and b"unknown epilogue" in lib.fb_last_error()
    e = _lib.DenseEpilogue(kind=_lib.DENSE_DYT_ADD)
    rc = lib.fb_dense(16, 4, 64, 64, 0, 16, 32, 64, 0, 1, 16, _lib.FP32, 32, 0, ctypes.byref(e), 0, None)
    assert rc == -1 and b"its vectors" in lib.fb_last_error()
    assert lib.fb_dense_supports(8, 64, 0, 16, 64, 0, 64, 32, _lib.DENSE_NONE) == 0, "a row of x that is not 16-byte aligned"
    rc = lib.fb_latent_put(_lib.FP32, 16, 2, 100, 40, 40, 21, 8, 16, 16, 1e-5, 16, 1.0, 16, 16, _lib.BF16, 16, 40, 0, 0, None, 0, 0, 16, 64, None)
    assert rc == -1 and b"within the key part" in lib.fb_last_error()
    rc = lib.fb_rotate_pairs(_lib.BF16, 16, 2, 4, 64, 16, 16, 5, 16, 1.0, 16, 16, 64, 16, None)
    assert rc == -1 and b"even number" in lib.fb_last_error()
    rc = lib.fb_latent_attention(_lib.BF16, 16, 2, 100, 4, 32, 8, 16, 64, 16, 0, 16, 64, 0, 0, 1.0, None, 16, 128, None, 0, None)
    assert rc == -1 and b"row strides too small" in lib.fb_last_error()
    rc = lib.fb_decay_scan(_lib.BF16, 16, 4096, 2, 600, 64, 16, 16, -1, 1, 4, 16, 2 * 600 * 64, 16, 128, None)
    assert rc == -1 and b"up to 512" in lib.fb_last_error()
    rc = lib.fb_gated_rmsnorm(16, 2, 64, 32, _lib.BF16, 16, 64, 0, 16, 1e-5, 1, _lib.BF16, 16, 64, None)
    assert rc == -1


def test_heads_and_experts_entry_points_refuse_bad_arguments_without_a_gpu():
    import ctypes
    lib = _lib.lib()
    h = _lib.Heads(heads=5, kv_heads=2, dim=8, vdim=8)
    rc = lib.fb_heads_put(ctypes.byref(h), _lib.FP32, 16, 4, 64, 16, _lib.BF16, 16, 40, 16, 64, 64 * 16, None)
    assert rc == -1 and b"whole groups" in lib.fb_last_error()
    rc = lib.fb_heads_put(ctypes.byref(_lib.Heads(heads=4, kv_heads=2, dim=8, vdim=8)), _lib.BF16, 16, 4, 64, 16, _lib.FP32, 16, 32, 16, 64, 64 * 16, None)
    assert rc == -1 and b"fp32 results come from fp32" in lib.fb_last_error()
    attend = lambda heads, dim, span, chunk=0, base=16: lib.fb_heads_attention(_lib.BF16, 16, 2, heads * dim, heads, 2, dim, 64, 16, 64, 64 * (dim + 64), base, 0, 16, 64, chunk, span, 0, 1.0, 0.0, None, None, 1.0, 0,
                                                                               None, 0, 16, heads * 64, None)
    assert attend(3, 64, 0) == -1 and b"whole groups" in lib.fb_last_error()
    assert attend(4, 2048, 0) == -1 and b"up to 1024" in lib.fb_last_error()
    assert attend(4, 64, -1) == -1 and attend(4, 64, 8, chunk=1) == -1 and b"one sequence's" in lib.fb_last_error()
    assert lib.fb_route_tiles(5, 10, 3, 16, 1) == 10 and lib.fb_route_tiles(1, 10, 3, 16, 1) == 3 and lib.fb_route_tiles(100, 10, 3, 32, 0) == 300 // 32 + 10
    rc = lib.fb_route(ctypes.byref(_lib.Router(10, 3, 0, None, 0, 1.0)), 16, 100, 10, 64, 1, 16, 16, 16, 16, 16, None, None)
    assert rc == -1 and b"all the tokens in one" in lib.fb_last_error()
    rc = lib.fb_route(ctypes.byref(_lib.Router(70, 65, 0, None, 0, 1.0)), 16, 4, 70, 16, 1, 16, 16, 16, 16, 16, None, None)
    assert rc == -1 and b"up to 64 choices" in lib.fb_last_error()
    e = _lib.DenseEpilogue(kind=_lib.DENSE_DYT_ADD)
    rc = lib.fb_dense_grouped(16, 64, 64, 64, 0, 16, 64, 64, 4096, 2, 16, 16, 2, 32, 16, _lib.BF16, 64, ctypes.byref(e), None)
    assert rc == -1 and b"a gated unit" in lib.fb_last_error()
    rc = lib.fb_dense_grouped(16, 64, 64, 64, 0, 16, 64, 64, 4096, 2, 16, 16, 3, 32, 16, _lib.BF16, 64, None, None)
    assert rc == -1 and b"all of them there" in lib.fb_last_error()
    rc = lib.fb_grouped_matmul(_lib.FP32, 16, 8, 64, 0, _lib.FP32, 16, (ctypes.c_int64 * 3)(4096, 1, 64), 2, 64, 64, 16, 16, 1, 16, None, _lib.FP32, 16, 64, None)
    assert rc == -1 and b"rows there" in lib.fb_last_error()
    rc = lib.fb_add_norm(ctypes.byref(_lib.Branches(x=16)), 2, 64, _lib.BF16, _lib.BF16, None)
    assert rc == -1 and b"no result" in lib.fb_last_error()
    rc = lib.fb_embed(_lib.BF16, 16, 8, 64, 16, 16, 0, None, 2, 1.0, 16, None)
    assert rc == -1 and b"takes the places" in lib.fb_last_error()


def test_turned_heads_windows_and_scored_routes_refuse_bad_arguments_without_a_gpu():
    import ctypes
    lib = _lib.lib()
    put = lambda **h: lib.fb_heads_put(ctypes.byref(_lib.Heads(**dict(heads=4, kv_heads=2, dim=8, vdim=8) | h)), _lib.FP32, 16, 6, 64, 16, _lib.BF16, 16, 32, 16, 64, 64 * 16, None)
    for h, what in ((dict(turned=10, freq=16, places=16), b"even number"), (dict(turned=4, freq=16), b"even number"), (dict(keys_are_values=1, vdim=4), b"as wide"), (dict(norm_all=1, q_norm=16), b"its weights"),
                    (dict(conv=16, taps=3, places=16, sequences=1), b"its state"), (dict(conv=16, taps=3, state=16, places=16, sequences=4, state_stride=999), b"as many rows"),
                    (dict(conv=16, taps=3, state=16, places=16, sequences=2, state_stride=64), b"as many rows"), (dict(norm_all=1, q_norm=16, k_norm=16, first=16, ld_first=16, share=16), b"plain heads")):
        assert put(**h) == -1 and what in lib.fb_last_error(), h
    put = lambda **a: lib.fb_latent_put(_lib.FP32, 16, 2, 200, a.get("q_rank", 0), 40, 8, 8, None, 16, 1e-5, 16, 1.0, 16, 16, _lib.BF16, 16, a.get("ld_q", 40), 5, 8, a.get("turned", 16), 240, 48, 16, 64, None)
    assert put(turned=None) == -1 and b"both their parts" in lib.fb_last_error()
    assert put(ld_q=39) == -1 and put(q_rank=8) == -1
    attend = lambda window, cap: lib.fb_heads_attention(_lib.BF16, 16, 2, 128, 2, 2, 64, 64, 16, 64, 64 * 128, 16, 0, 16, 64, 0, 0, window, 1.0, cap, None, None, 1.0, 0, None, 0, 16, 128, None)
    assert attend(-1, 0.0) == -1 and attend(4, -1.0) == -1 and b"a cap of scores" in lib.fb_last_error()
    rc = lib.fb_route(ctypes.byref(_lib.Router(10, 3, 10, None, 1, 1.0)), 16, 4, 10, 16, 1, 16, 16, 16, 16, 16, None, None)
    assert rc == -1 and b"at least one expert" in lib.fb_last_error()
    e = _lib.DenseEpilogue(kind=_lib.DENSE_GEGLU)
    rc = lib.fb_dense(16, 4, 64, 64, 0, 16, 40, 64, 0, 1, 16, _lib.BF16, 32, 0, ctypes.byref(e), 0, None)
    assert rc == -1 and b"whole runs of 16" in lib.fb_last_error()
    rc = lib.fb_dense_grouped(16, 64, 64, 64, 0, 16, 64, 64, 4096, 2, 16, 16, 2, 32, 16, _lib.BF16, 64, ctypes.byref(e), None)
    assert rc == -1 and b"a gated unit" in lib.fb_last_error()


def test_state_spaces_convolutions_and_sigmoid_weights_refuse_bad_arguments_without_a_gpu():
    import ctypes
    lib = _lib.lib()
    scan = lambda heads=4, groups=2, dim=8, ld=64, stride=256, **a: lib.fb_selective_scan(_lib.BF16, 16, ld, heads, groups, dim, 8, 16, a.get("ld_step", 4), 16, 16, 16, 16, -1, 2, 3, 16, stride, 16, 32, None)
    assert scan(groups=3) == -1 and b"whole groups of heads" in lib.fb_last_error()
    assert scan(dim=600, ld=9999, stride=99999) == -1 and b"up to 512" in lib.fb_last_error()
    assert scan(ld=63) == -1 and b"row strides" in lib.fb_last_error()
    assert scan(ld_step=3) == -1 and scan(stride=255) == -1 and b"row strides" in lib.fb_last_error()
    rc = lib.fb_gated_rmsnorm(16, 2, 60, 60, _lib.FP32, 16, 60, 1, 16, 1e-5, 7, _lib.BF16, 16, 60, None)
    assert rc == -1 and b"equal parts" in lib.fb_last_error()
    rc = lib.fb_gated_rmsnorm(16, 2, 60, 60, _lib.BF16, 16, 60, 1, 16, 1e-5, 2, _lib.FP32, 16, 60, None)
    assert rc == -1 and b"take fp32 gates" in lib.fb_last_error()
    conv = lambda **c: lib.fb_short_conv(ctypes.byref(_lib.Conv(**dict(cols=8, taps=4, w=16, places=16, dead=-1, sequences=2, tokens=3, state=16, state_stride=24) | c)), _lib.FP32, 16, 8, _lib.BF16, 16, 8, None)
    assert conv(state=None) == -1 and b"taps - 1 rows" in lib.fb_last_error()
    assert conv(state_stride=23) == -1 and conv(taps=0) == -1 and conv(cols=9, state_stride=99) == -1 and b"row strides" in lib.fb_last_error()
    lru = lambda ld_g=16, dtype=_lib.BF16, y=_lib.FP32, **c: lib.fb_lru_scan(ctypes.byref(_lib.Lru(**dict(width=8, blocks=2, lam=16, rate=-8.0, scale=1.0, places=16, dead=-1, sequences=2, tokens=3, state=16,
                                                                                                  state_stride=8) | c)), dtype, 16, 8, 16, ld_g, y, 16, 8, 16, 8, None)
    assert lru(blocks=3) == -1 and b"equal blocks" in lib.fb_last_error()
    assert lru(ld_g=15) == -1 and lru(state_stride=7) == -1 and lru(dtype=_lib.FP32, y=_lib.BF16) == -1 and b"come from fp32" in lib.fb_last_error()
    put = lambda **h: lib.fb_heads_put(ctypes.byref(_lib.Heads(**dict(heads=4, kv_heads=2, dim=8, vdim=8) | h)), _lib.FP32, 16, 6, 64, 16, _lib.BF16, 16, 32, 16, 64, 64 * 16, None)
    assert put(temp_coef=0.5, temp_every=8.0) == -1 and put(temp_coef=0.5, temp_every=0.0, places=16) == -1 and b"temperature" in lib.fb_last_error()
    rc = lib.fb_heads_attention(_lib.BF16, 16, 2, 128, 2, 2, 64, 64, 16, 64, 64 * 128, 16, 0, 16, 64, 0, 0, 0, 1.0, 0.0, 16, 16, 1.0, 0, None, 0, 16, 128, None)
    assert rc == -1 and b"a softmax's denominator" in lib.fb_last_error()
    rc = lib.fb_route(ctypes.byref(_lib.Router(10, 3, 0, None, 3, 1.0)), 16, 4, 10, 16, 1, 16, 16, 16, 16, 16, None, None)
    assert rc == -1 and b"softmax or sigmoid" in lib.fb_last_error()
    e = _lib.DenseEpilogue(kind=_lib.DENSE_NONE, row_scale=16)
    rc = lib.fb_dense_grouped(16, 64, 64, 64, 0, 16, 64, 64, 4096, 2, 16, 16, 2, 32, 16, _lib.BF16, 64, ctypes.byref(e), None)
    assert rc == -1 and b"take one" in lib.fb_last_error()
    rc = lib.fb_add_norm(ctypes.byref(_lib.Branches(x=16, x_out=16, ld_x=64, ld_x_out=64, gate=16, ld_gate=60)), 2, 64, _lib.BF16, _lib.BF16, None)
    assert rc == -1 and b"a gate a column" in lib.fb_last_error()
