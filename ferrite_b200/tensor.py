"""Lazy tensors on a B200: the drop-in for `ferrite.tensor` (Tensor, jit) on the decode path.

The operator surface is ferrite's (ferrite/tensor.py:14-817): batch x rows x cols tensors of bf16, fp32, int32, bfp8 or
bfp4 whose ops build a tree; `realize` turns the tree into kernel launches.  Below the method signatures nothing is
ferrite's: storage is a torch CUDA tensor (ownership and views only), every computation is one of this package's
sm_100a kernels reached through the C ABI (ferrite_b200/_lib.py), launched on torch's current stream, and the planner
maps the trees a Llama block builds onto the fused kernels:

    x * rsqrt(mean(x*x) + eps) * w  feeding a block-float matmul   -> RMSNorm prologue of fb_linear
    silu(mm[:, :m]) * mm[:, m:]                                      -> SwiGLU epilogue of fb_linear (bf16 weights: fb_dense)
    x + mm                                                           -> residual epilogue of fb_linear
    any other elementwise tree                                       -> one fb_elementwise launch (postfix program)

There is no CPU path: without the CUDA library the import of `_lib` raises.
`jit` replays a recorded step as one CUDA graph (ferrite/tensor.py:788-810 replays a recorded block of launches).
"""
import array
import gc
import math

import numpy as np
import torch

from . import _lib, ops
from ._lib import check, lib

BFP = ("bfp8", "bfp4")
_TORCH = {"bf16": torch.bfloat16, "fp32": torch.float32, "int32": torch.int32}
_NAME = {v: k for k, v in _TORCH.items()}
# Whether the planner hands an RMSNorm from the matmul that makes its input to the matmul that consumes it
# (fb_linear_chained) instead of running the norm's preparation as a kernel of its own.  Off: measured on the 8B-shape
# step it saves 64 launches and still costs time (5.21 ms against 5.01): the preparation kernel hides behind the next
# matmul's set-up, while the hand-over adds a pass at the end of the producing matmul and a sum over its 128 parts.
CHAIN_NORMS = False
FIDELITY = 4  # accepted and ignored, as the numpy reference ignores it (models/llama.py:33): products are exact here

# elementwise opcodes of fb_elementwise (include/ferrite_b200.h)
_BINARY = {"add": 10, "sub": 11, "mul": 12, "max": 13, "cmplt": 14, "cmpne": 15, "keep": 16, "drop": 17, "div": 18, "min": 19}
_UNARY = {"exp": 30, "log": 31, "sin": 32, "cos": 33, "sqrt": 34, "recip": 35, "relu": 36, "exp2": 37, "log2": 38, "round_bf16": 39,
          "trunc": 40, "neg": 41, "tanh": 42}
_ELEMENTWISE = set(_BINARY) | set(_UNARY) | {"cast"}
_MAX_OPS, _MAX_INPUTS, _MAX_STACK = 48, 8, 12


class Runtime:
    """What ferrite's Runtime is to its Tensors (ferrite/runtime.py:304-505), on a CUDA device: launches are queued on
    a stream in order and only reading back waits; `wait` has a timeout in the sense that every device-side wait of the
    kernels is bounded and reports through the status word."""

    def __init__(self, device=0):
        assert torch.cuda.is_available(), "ferrite_b200 needs a CUDA device: there is no CPU path"
        self.device = torch.device("cuda", device) if not isinstance(device, torch.device) else device
        torch.cuda.set_device(self.device)
        lib()
        self.numbers, self.launches, self.names = {}, 0, []

    def launched(self, name, kernels=0):
        """One op queued; kernels: how many kernels it launched that no ops.* wrapper has counted already."""
        ops.count(kernels)
        self.launches += 1
        if len(self.names) < 4096:
            self.names.append(name)

    def wait(self, timeout=None):
        torch.cuda.synchronize(self.device)
        code = lib().fb_status_word()
        if code:
            raise TimeoutError(f"a device-side wait gave up (code {code})")

    def profile(self, since=0):
        """(name, launches) of the kernels launched after launch number `since`, most frequent first."""
        counts = {}
        for n in self.names[since:]:
            counts[n] = counts.get(n, 0) + 1
        return sorted(counts.items(), key=lambda kv: -kv[1])


def _strides3(buf):
    return [int(s) for s in buf.stride()]


class Tensor:
    """batch x rows x cols of bf16, fp32, int32, bfp8 or bfp4 (ferrite/tensor.py:15-29); realized (it has storage) or
    an op on other tensors not yet computed."""

    def __init__(self, rt, rows, cols, op=None, srcs=(), batch=1, dtype="bf16", buf=None, packed=None, owner=None, args=None):
        self.rt, self.rows, self.cols, self.batch, self.op, self.srcs, self.dtype = rt, rows, cols, batch, op, srcs, dtype
        self.args, self.owner, self.buf, self.packed = args or {}, owner, buf, packed
        self.requires_grad, self.grad = False, None
        if op is None and buf is None and packed is None:
            if dtype in BFP:
                n = lib().fb_packed_bytes(_lib.DTYPES[dtype], rows, cols)
                assert n, f"a block float's columns come in runs of 16, not {cols}"
                self.packed = ops.Packed(dtype, batch, rows, cols, torch.empty(batch * n, dtype=torch.uint8, device=rt.device))
            else:
                self.buf = torch.empty(batch, rows, cols, dtype=_TORCH[dtype], device=rt.device)

    @property
    def shape(self):
        return (self.batch, self.rows, self.cols)

    def __hash__(self):
        return id(self)

    # ---------------------------------------------------------------- in and out

    @classmethod
    def full(cls, rt, rows, cols, value, dtype="bf16"):
        return cls.of(rt, [[value] * cols for _ in range(rows)], dtype)

    @classmethod
    def of(cls, rt, data, dtype="bf16"):
        """From a list of rows of numbers, or a list of those (a batch), rounded to dtype (bf16: to nearest even)."""
        a = np.asarray(data, dtype=np.int32 if dtype == "int32" else np.float32)
        a = a.reshape((1,) * (3 - a.ndim) + a.shape)
        host = torch.from_numpy(np.ascontiguousarray(a))
        return cls(rt, a.shape[1], a.shape[2], batch=a.shape[0], dtype=dtype, buf=host.to(_TORCH[dtype]).to(rt.device))

    @classmethod
    def frombytes(cls, rt, rows, cols, data, batch=1, dtype="bf16"):
        """From dtype's values in row-major order (little-endian), matrix after matrix (ferrite/tensor.py:60-80)."""
        assert dtype not in BFP, "a block float is made on the chip, by cast"
        raw = np.frombuffer(memoryview(data).cast("B"), dtype=np.uint8)
        size = {"bf16": 2, "fp32": 4, "int32": 4}[dtype]
        assert len(raw) == size * batch * rows * cols, f"{len(raw)} bytes for {batch} x {rows} x {cols} of {dtype}"
        view = {"bf16": np.int16, "fp32": np.float32, "int32": np.int32}[dtype]
        host = torch.from_numpy(raw.view(view).reshape(batch, rows, cols).copy())
        if dtype == "bf16":
            host = host.view(torch.bfloat16)
        return cls(rt, rows, cols, batch=batch, dtype=dtype, buf=host.to(rt.device))

    def tobytes(self):
        """dtype's values in row-major order, a block float's as bf16 (ferrite/tensor.py:82-107).  Waits."""
        t = self.realize()
        buf = ops.dequantize(t.packed) if t.dtype in BFP else t.buf
        host = buf.contiguous().cpu()
        code = lib().fb_status_word()
        if code:
            raise TimeoutError(f"a device-side wait gave up (code {code})")
        if host.dtype == torch.bfloat16:
            host = host.view(torch.int16)
        return host.numpy().tobytes()

    def tolist(self):
        raw = self.tobytes()
        if self.dtype == "bf16" or self.dtype in BFP:
            raw = array.array("I", [b << 16 for b in array.array("H", raw)]).tobytes()
        values = array.array("i" if self.dtype == "int32" else "f", raw).tolist()
        m = [[values[(b * self.rows + r) * self.cols:(b * self.rows + r + 1) * self.cols] for r in range(self.rows)] for b in range(self.batch)]
        return m if self.batch > 1 else m[0]

    def numpy(self):
        """The values as a numpy array of shape (batch, rows, cols): float32 (bf16 and block floats widened) or int32."""
        kind = np.int32 if self.dtype == "int32" else np.float32
        raw = self.tobytes()
        if self.dtype == "bf16" or self.dtype in BFP:
            return (np.frombuffer(raw, np.uint16).astype(np.uint32) << 16).view(np.float32).reshape(self.shape)
        return np.frombuffer(raw, kind).reshape(self.shape)

    # ---------------------------------------------------------------- building the tree

    def _lazy(self, op, srcs, shape, dtype, **args):
        return Tensor(self.rt, shape[1], shape[2], op, tuple(srcs), shape[0], dtype, args=args)

    def _view(self, buf):
        """A realized tensor over `buf`, a torch view of this one's storage (shares it; writes go through)."""
        return Tensor(self.rt, buf.shape[1], buf.shape[2], batch=buf.shape[0], dtype=self.dtype, buf=buf, owner=self.owner or self)

    def _unary(self, op):
        if self.dtype == "int32" and op != "relu":
            return self.float()._unary(op)
        return self._lazy(op, (self,), self.shape, self.dtype)

    def _binop(self, op, x, reverse=False):
        """numpy's broadcasting: shapes match, or one side has 1 where the other does not; different dtypes meet in
        fp32 (ferrite/tensor.py:305-314).  A Python number is a constant of the expression."""
        if isinstance(x, Tensor):
            assert all(n == m or 1 in (n, m) for n, m in zip(self.shape, x.shape)), f"cannot broadcast {self.shape} with {x.shape}"
            shape = tuple(map(max, self.shape, x.shape))
            dtype = self.dtype if self.dtype == x.dtype else "fp32"
        else:
            shape, dtype = self.shape, "fp32" if self.dtype == "int32" and isinstance(x, float) else self.dtype
        if dtype == "int32" and op in ("mul", "div"):
            dtype = "int32"  # computed through fp32, exact below 2^24 (as ferrite's)
        a, b = (x, self) if reverse else (self, x)
        return self._lazy(op, (a, b), shape, dtype)

    def cast(self, dtype):
        if dtype == self.dtype:
            return self
        return self._lazy("cast", (self,), self.shape, dtype)

    def float(self): return self.cast("fp32")
    def bfloat16(self): return self.cast("bf16")
    def exp2(self): return self._unary("exp2")
    def log2(self): return self._unary("log2")
    def sin(self): return self._unary("sin")
    def cos(self): return self._unary("cos")
    def sqrt(self): return self._unary("sqrt")
    def reciprocal(self): return self._unary("recip")
    def exp(self): return self._unary("exp")
    def log(self): return self._unary("log")
    def tanh(self): return self._unary("tanh")
    def relu(self): return self._unary("relu")
    def rsqrt(self): return self.sqrt().reciprocal()
    def maximum(self, x): return self._binop("max", x)
    def minimum(self, x): return self._binop("min", x)
    def __add__(self, x): return self._binop("add", x)
    def __sub__(self, x): return self._binop("sub", x)
    def __mul__(self, x): return self._binop("mul", x)
    def __rsub__(self, x): return self._binop("sub", x, True)
    __radd__, __rmul__ = __add__, __mul__
    def __truediv__(self, x): return self * (1 / x) if isinstance(x, (int, float)) else self * x.reciprocal()
    def __rtruediv__(self, x): return self.reciprocal() * x
    def __neg__(self): return 0 - self if self.dtype == "int32" else self * -1
    def __lt__(self, x): return self._binop("cmplt", x)
    def __gt__(self, x): return self._binop("cmplt", x, True)
    def __ge__(self, x): return 1 - (self < x)
    def __le__(self, x): return 1 - (self > x)
    def ne(self, x): return self._binop("cmpne", x)
    def eq(self, x): return 1 - self.ne(x)
    __ne__, __eq__ = ne, eq
    def sigmoid(self): return (1 + (-self).exp()).reciprocal()
    def silu(self): return self * self.sigmoid()

    def where(self, x, y):
        """x where self is not 0, else y (ferrite/tensor.py:343-346)."""
        return self._binop("keep", x) + self._binop("drop", y)

    def gelu(self):  # GPT-2's tanh form (ferrite/tensor.py:355-357)
        k = 2 * math.sqrt(2 / math.pi)
        return self * (1 + (self * (self * self * (-0.044715 * k) - k)).exp()).reciprocal()

    def delta(self, *args, **kwargs):
        """Gated DeltaNet's recurrence (ferrite/tensor.py): on the reference's surface, not on the decode path built here."""
        raise NotImplementedError("Tensor.delta (Gated DeltaNet) is outside the decode path this library covers")

    def sum(self, axis=None): return self._reduce("sum", axis)
    def max(self, axis=None): return self._reduce("max", axis)

    def _reduce(self, f, axis):
        """numpy's, keeping the axis as 1 (ferrite/tensor.py:361-368)."""
        if axis is None:
            return self._reduce(f, 0)._reduce(f, 1)._reduce(f, 2)
        axis %= 3
        shape = tuple(1 if ax == axis else s for ax, s in enumerate(self.shape))
        return self if shape == self.shape else self._lazy("reduce_" + f, (self,), shape, self.dtype, axis=axis)

    def mean(self, axis=None):
        s = self.sum(axis)
        return s * (math.prod(s.shape) / math.prod(self.shape))

    def softmax(self, axis=-1):
        e = (self - self.max(axis)).exp()
        return e / e.sum(axis)

    def log_softmax(self, axis=-1):
        m = self - self.max(axis)
        return m - m.exp().sum(axis).log()

    def layernorm(self, axis=-1, eps=1e-5):
        c = self - self.mean(axis)
        return c * ((c * c).mean(axis) + eps).rsqrt()

    # ---------------------------------------------------------------- movement: views of the storage where torch has one

    def __getitem__(self, key):
        """x[b]; x[rows, cols] of every matrix; x[batch, rows, cols], with slices (ferrite/tensor.py:149-165).  A slice
        of a matmul not yet computed stays part of the tree, so that SwiGLU's halves fuse into the matmul."""
        if isinstance(key, int):
            return self.realize()._view(self.buf[key:key + 1])
        assert isinstance(key, tuple) and len(key) in (2, 3) and all(isinstance(k, slice) for k in key), "x[b], x[rows, cols] or x[batch, rows, cols]"
        key = (slice(None),) * (3 - len(key)) + tuple(key)
        ranges = [range(*k.indices(n)) for k, n in zip(key, self.shape)]
        assert all(len(r) for r in ranges), f"an empty slice of {self.shape}"
        if self.op == "matmul" and all(r.step == 1 for r in ranges) and len(ranges[0]) == self.batch and len(ranges[1]) == self.rows:
            return self._lazy("cols", (self,), (self.batch, self.rows, len(ranges[2])), self.dtype, start=ranges[2].start)
        t = self.realize()
        if any(r.step < 0 for r in ranges):  # torch has no negative strides: flip through a gather of indices
            buf = t.buf
            for ax, r in enumerate(ranges):
                buf = buf.index_select(ax, torch.tensor(list(r), device=buf.device))
            return t._view(buf)
        return t._view(t.buf[key])

    def reshape(self, *shape):
        shape = (1,) * (3 - len(shape)) + tuple(shape)
        assert math.prod(shape) == math.prod(self.shape), f"cannot reshape {self.shape} to {shape}"
        if shape == self.shape:
            return self
        t = self.realize()
        try:
            return t._view(t.buf.view(shape))
        except RuntimeError:  # not expressible by strides: a copy, made by the elementwise kernel
            return (t + 0).realize().reshape(*shape)

    def permute(self, *order):
        assert sorted(order) == [0, 1, 2]
        t = self.realize()
        return t._view(t.buf.permute(*order))

    @property
    def T(self):
        return self.permute(0, 2, 1)

    def expand(self, *shape):
        shape = (1,) * (3 - len(shape)) + tuple(shape)
        assert all(n in (m, 1) for n, m in zip(self.shape, shape)), f"cannot expand {self.shape} to {shape}"
        t = self.realize()
        return t._view(t.buf.expand(*shape))

    def pad(self, widths):
        """Zeros around: (before, after) for each of the last len(widths) axes (ferrite/tensor.py:194-199)."""
        widths = ((0, 0),) * (3 - len(widths)) + tuple(widths)
        t = self.realize()
        shape = [n + w[0] + w[1] for n, w in zip(self.shape, widths)]
        out = Tensor(self.rt, shape[1], shape[2], batch=shape[0], dtype=self.dtype)
        _fill(out, 0)
        out[tuple(slice(w[0], w[0] + n) for n, w in zip(self.shape, widths))].assign(t)
        return out

    def cat(self, *xs, axis=0):
        ts, axis = [t.realize() for t in (self, *xs)], axis % 3
        shape = list(self.shape)
        shape[axis] = sum(t.shape[axis] for t in ts)
        out, at = Tensor(self.rt, shape[1], shape[2], batch=shape[0], dtype=self.dtype), 0
        for t in ts:
            key = [slice(None)] * 3
            key[axis] = slice(at, at + t.shape[axis])
            out[tuple(key)].assign(t)
            at += t.shape[axis]
        return out

    def repeat_interleave(self, n):
        """Each matrix n times over along the batch (ferrite/tensor.py:210-217).  Attention reads the repeat in place
        (entry b uses matrix b // n); anything else that needs its values gets a copy."""
        t = self.realize()
        return self._lazy("repeat", (t,), (t.batch * n, t.rows, t.cols), t.dtype, n=n)

    def split(self, n, axis=2):
        """The matrix cut into n equal parts along axis as a batch of n, in place (ferrite/tensor.py:219-232)."""
        assert axis in (1, 2)
        t = self.realize()
        if axis == 2:
            assert t.batch == 1 and t.cols % n == 0, "equal parts of one matrix"
            return t._view(t.buf.view(t.rows, n, t.cols // n).permute(1, 0, 2))
        assert t.rows % n == 0, "equal parts"
        if t.batch == 1:
            return t._view(t.buf.view(n, t.rows // n, t.cols))
        return t._view(t.buf.unflatten(1, (n, t.rows // n)).flatten(0, 1))

    def merge(self):
        """The batch side by side as one matrix, the inverse of split (ferrite/tensor.py:234-240)."""
        t = self.realize()
        out = Tensor(self.rt, t.rows, t.batch * t.cols, dtype=t.dtype)
        out.split(t.batch).assign(t)
        return out

    def assign(self, x):
        """x's value into this tensor's storage, in place (ferrite/tensor.py:273-283)."""
        assert self.op is None and (x.shape, x.dtype) == (self.shape, self.dtype), "a tensor or view, its own shape and dtype"
        if x.op is not None and x.op in _ELEMENTWISE:
            _run_elementwise(x, into=self)
            x.op, x.srcs, x.buf = None, (), self.buf
        else:
            _copy(x.realize(), self)
        return self

    # ---------------------------------------------------------------- rows by index

    def gather(self, ids):
        """Rows ids of this matrix: an embedding lookup (ferrite/tensor.py:116-126)."""
        if not isinstance(ids, Tensor):  # a list of rows: a constant of the program, uploaded once (a recorded step meets it again)
            key = ("rows", tuple(int(i) for i in ids))
            assert all(0 <= i < self.rows for i in key[1])
            if key not in self.rt.numbers:
                self.rt.numbers[key] = Tensor.of(self.rt, [list(key[1])], "int32")
            ids = self.rt.numbers[key]
        assert self.batch == 1 and ids.dtype == "int32" and ids.shape[:2] == (1, 1), "rows of a matrix, by a row of int32"
        t, ids = self.realize(), ids.realize()
        table = t.buf[0] if t.buf[0].is_contiguous() else t.buf[0].contiguous()
        out = Tensor(self.rt, ids.cols, self.cols, dtype=self.dtype)
        ops.gather_rows(table, ids.buf.reshape(-1), out.buf[0])
        self.rt.launched("gather")
        return out

    def put(self, ids, x):
        """x's rows into rows ids of each matrix of this tensor, in place (ferrite/tensor.py:128-140); a later
        duplicate wins."""
        assert ids.dtype == "int32" and ids.shape[:2] == (1, 1) and ids.cols == x.rows, "rows of x, by a row of int32 places"
        assert (x.batch, x.cols) == (self.batch, self.cols) and x.dtype == self.dtype, f"{x.shape} {x.dtype} into {self.shape} {self.dtype}"
        t, x, ids = self.realize(), x.realize(), ids.realize()
        check(lib().fb_put_rows(t.buf.data_ptr(), *_strides3(t.buf), x.buf.data_ptr(), *_strides3(x.buf), ids.buf.data_ptr(), t.batch, x.rows, t.cols,
                                t.rows, t.buf.element_size(), ops._stream()))
        self.rt.launched("put", 1)
        return self

    # ---------------------------------------------------------------- matmul, attention, the router

    def __matmul__(self, x):
        return self.matmul(x)

    def matmul(self, x, dtype=None, fidelity=None, index=None):
        """Matrix by matrix through a batch, summed in fp32 and written as dtype: bf16, or fp32 if either operand is,
        unless said (ferrite/tensor.py:443-485).  x may be a block float when self is bf16.  index: an int32 (rows, k)
        tensor picking, for batch entry b of the result, which of x's matrices to multiply by (a mixture of experts'
        choice); an entry picking none (x.batch or more) is zeros."""
        assert "int32" not in (self.dtype, x.dtype), "the FPU multiplies floats"
        assert self.cols == x.rows, f"{self.shape} @ {x.shape}"
        if index is not None:
            assert index.dtype == "int32" and self.dtype == "bf16" and self.batch in (1, index.rows * index.cols), \
                f"{self.shape} @ {x.shape} picked by {index.shape} {index.dtype}"
            return self._lazy("matmul", (self, x, index), (index.rows * index.cols, self.rows, x.cols), dtype or "bf16")
        assert self.batch == x.batch or 1 in (self.batch, x.batch), f"{self.shape} @ {x.shape}"
        dtype = dtype or ("fp32" if "fp32" in (self.dtype, x.dtype) else "bf16")
        return self._lazy("matmul", (self, x), (max(self.batch, x.batch), self.rows, x.cols), dtype)

    def attend(self, k, v, places, window=0, fidelity=None, parts=None):
        """softmax(self @ k^T + mask) @ v in one kernel (ferrite/tensor.py:487-516): self a batch of queries, k and v
        the keys and values for each (a repeat is read in place), places (int32, a column per entry or one for all):
        each row's last key; with a window, only the last `window` keys.  bf16 keys and values."""
        rep = k.args.get("n", 1) if k.op == "repeat" else 1
        assert (v.args.get("n", 1) if v.op == "repeat" else 1) == rep and self.batch == k.batch == v.batch
        assert self.dtype == "bf16" and k.dtype == v.dtype == "bf16", "bf16 queries, keys and values (a block-float cache is read by attend_cache)"
        assert self.cols == k.cols == v.cols and self.cols in (64, 128) and k.rows == v.rows, "heads of 64 or 128 columns"
        assert places.rows == self.rows and places.batch in (1, self.batch) and places.cols == 1 and places.dtype == "int32", \
            f"{self.shape} by {k.shape}, {places.shape}"
        q, places = self.realize(), places.realize()
        kb = (k.srcs[0] if k.op == "repeat" else k).realize().buf
        vb = (v.srcs[0] if v.op == "repeat" else v).realize().buf
        if q.buf.stride(2) != 1 or q.buf.stride(1) % 8 or q.buf.stride(0) % 8:
            q = (q + 0).realize()
        kb, vb = (b if b.stride(2) == 1 and b.stride(1) == self.cols else b.contiguous() for b in (kb, vb))
        assert kb.stride(0) == vb.stride(0), "keys and values laid out alike"
        out = Tensor(self.rt, self.rows, self.cols, batch=self.batch)
        need = lib().fb_attend_workspace_bytes(self.batch, self.rows, self.cols, k.rows)
        ws = ops.attention_workspace(self.rt.device, need)
        check(lib().fb_attend(q.buf.data_ptr(), self.batch, self.rows, self.cols, q.buf.stride(0), q.buf.stride(1), kb.data_ptr(), vb.data_ptr(),
                              kb.stride(0), rep, k.rows, places.buf.data_ptr(), places.buf.stride(0) if places.batch > 1 else 0,
                              places.buf.stride(1), window or 0, 1.0, out.buf.data_ptr(), ops._ptr(ws), ws.numel() if ws is not None else 0,
                              ops._stream()))
        self.rt.launched("attention", 2 if need else 1)
        return out

    def topk(self, k, parts=1, labels=None):
        """Along each row, largest first: (values, int32 indices), the first column of equals first
        (ferrite/tensor.py:373-388).  parts: each row cut into so many parts, each part's k best side by side."""
        cols = self.cols // parts
        assert self.dtype in ("bf16", "fp32") and k <= min(cols, 64) and parts * cols == self.cols, "bf16 or fp32, k of at most 64, whole parts"
        assert labels is None or (labels.dtype == "int32" and labels.shape == self.shape and parts == 1), "labels: int32, x's shape"
        x = self.realize()
        if not x.buf.is_contiguous():
            x = (x + 0).realize()
        labels = None if labels is None else labels.realize()
        if labels is not None and not labels.buf.is_contiguous():
            labels = (labels + 0).realize()
        values = Tensor(self.rt, x.rows, parts * k, batch=x.batch, dtype=x.dtype)
        ids = Tensor(self.rt, x.rows, parts * k, batch=x.batch, dtype="int32")
        # a row of `parts` parts is `parts` rows of one part each: one launch for all of them
        check(lib().fb_topk(_lib.DTYPES[x.dtype], x.buf.data_ptr(), x.batch * x.rows * parts, cols, cols, k, ops._ptr(labels.buf) if labels is not None else None,
                            values.buf.data_ptr(), ids.buf.data_ptr(), None, k, ops._stream()))
        if parts > 1:  # (the parts' first columns: a constant, uploaded once - a recorded step meets it again)
            key = ("topk parts", parts, cols, k)
            if key not in self.rt.numbers:
                self.rt.numbers[key] = Tensor.of(self.rt, [[p * cols for p in range(parts) for _ in range(k)]], "int32")
            ids = (ids + self.rt.numbers[key]).realize()
        self.rt.launched("topk", 1)
        return values, ids

    def group(self, n):
        """A mixture of experts' tokens grouped by expert, from int32 choices (rows x k, values below n), as three int32
        tensors (ferrite/tensor.py:389-402): order, a row of 32 t slots in which each value's choices have a run of whole
        tiles of 32, each slot the row it holds (0 for none); tiles, a column of t, each tile's value (n past those
        used); places, a row of k runs of the rows rounded up to 32, run j holding the slot of each row's choice j."""
        assert self.dtype == "int32" and self.batch == 1 and self.cols <= 32, "a matrix of int32 choices, at most 32 a row"
        x = self.realize()
        x = x if x.buf.is_contiguous() else (x + 0).realize()
        rows, k = self.rows, self.cols
        t, rp = -(-rows * k // 32) + min(n, rows * k), -(-rows // 32) * 32
        order, tiles, places = Tensor(self.rt, 1, 32 * t, dtype="int32"), Tensor(self.rt, t, 1, dtype="int32"), Tensor(self.rt, 1, k * rp, dtype="int32")
        check(lib().fb_group(x.buf.data_ptr(), rows, k, n, order.buf.data_ptr(), tiles.buf.data_ptr(), places.buf.data_ptr(), ops._stream()))
        self.rt.launched("group", 1)
        return order, tiles, places

    def touched(self, n, weights, first=0):
        """The experts some row picks by a weight that is not 0, each once, ascending, then n (none); and each entry's
        weight from each row (ferrite/tensor.py:403-416).  first: count the experts from it (a rank's run of a mixture's
        experts: only those are listed, numbered from 0)."""
        assert self.dtype == "int32" and weights.dtype == "bf16" and self.shape == weights.shape and self.batch == 1 and self.cols <= 32
        x, w = self.realize(), weights.realize()
        x = x if x.buf.is_contiguous() else (x + 0).realize()
        w = w if w.buf.is_contiguous() else (w + 0).realize()
        slots = min(self.rows * self.cols, n)
        experts, out = Tensor(self.rt, slots, 1, dtype="int32"), Tensor(self.rt, self.rows, 1, batch=slots)
        check(lib().fb_touched(x.buf.data_ptr(), w.buf.data_ptr(), self.rows, self.cols, n, first, experts.buf.data_ptr(), out.buf.data_ptr(), ops._stream()))
        self.rt.launched("touched", 1)
        return experts, out

    def gelu_gated(self, bias=None, dtype=None):
        """gelu(gate) * up of self's two halves, bias (fp32, a number a column of self) added before; fuses into a matmul."""
        assert self.cols % 2 == 0 and (bias is None or (bias.dtype == "fp32" and bias.shape == (1, 1, self.cols)))
        return self._lazy("gelu_gated", (self,) if bias is None else (self, bias), (self.batch, self.rows, self.cols // 2), dtype or self.dtype)

    def silu_columns(self, n):
        """self with its first n columns through SiLU (a joint projection of activated and plain parts); fuses into a matmul."""
        return self._lazy("silu_columns", (self,), self.shape, self.dtype, n=n)

    # ---------------------------------------------------------------- a decode step's two fused kernels

    def rope_put(self, cos, sin, places, rows, cache, heads, kv, qk_norm=None, eps=1e-5):
        """self: a fused q, k, v projection [1, tokens, (heads + 2 kv) hd].  One kernel does what models/llama.py:119-128
        spells as split, (Qwen3's norm of each q and k head,) rope, merge and put: q's heads turned by RoPE come back as
        [1, tokens, heads hd]; k's (turned) and v's go into `cache` ([2 kv, size, hd]) at `rows`.  cos / sin: tables with
        a row for each place, one head wide or as wide as self; places, rows: int32 rows read on the device."""
        hd = cache.cols
        qkv = self.realize()
        assert qkv.batch == 1 and qkv.cols == (heads + 2 * kv) * hd and cache.batch == 2 * kv and cache.dtype in ("bf16",) + tuple(BFP), \
            f"{qkv.shape} into a cache {cache.shape}"
        assert places.dtype == rows.dtype == "int32" and places.cols == rows.cols == qkv.rows, "a place and a cache row per token"
        cos, sin, places, rows = (t.realize() for t in (cos, sin, places, rows))
        qb = qkv.buf[0] if qkv.buf.stride(2) == 1 else (qkv + 0).realize().buf[0]
        out = Tensor(self.rt, qkv.rows, heads * hd)
        assert cache.dtype in BFP or (cache.buf.stride(2) == 1 and cache.buf.stride(1) == hd), "a cache's rows lie one after another"
        ops.rope_kv_write(qb, cos.buf[0], sin.buf[0], places.buf.reshape(-1), rows.buf.reshape(-1), cache.packed if cache.dtype in BFP else cache.buf, heads, kv, hd, q_out=out.buf[0],
                          qk_norm=None if qk_norm is None else qk_norm.realize().buf, eps=eps)
        self.rt.launched("rope put")
        return out

    def attend_cache(self, cache, base, last, kv, length=None, window=0, chunk=False):
        """self: [1, tokens, heads hd], each token's query heads.  Token t attends the cache rows base[t] .. base[t] +
        last[t] of every kv head (the last `window` of them, if any), its heads / kv query heads sharing each key row
        read: attention as models/llama.py:129-146 runs it on the chip (Tensor.attend with places), without the views,
        the repeat and the regrouping moves in between.  length: the most keys a token can see (it sizes the split of
        the keys over the GPU).  chunk: the tokens are one sequence's (a prompt's chunk, its first cache row 0): a query
        head's tokens then share each key row read, 16 at a time, instead of every token reading the keys anew."""
        hd = cache.cols
        q = self.realize()
        heads = q.cols // hd
        assert q.batch == 1 and q.cols % hd == 0 and heads % kv == 0 and cache.batch == 2 * kv, f"{q.shape} over a cache {cache.shape}"
        base, last = base.realize(), last.realize()
        out = Tensor(self.rt, q.rows, q.cols)
        if chunk:
            ops.prefill_attention(q.buf[0], cache.packed if cache.dtype in BFP else cache.buf, 0, last.buf.reshape(-1), heads, kv, hd,
                                  max_keys=min(length or cache.rows, cache.rows), window=window or 0, out=out.buf[0])
            self.rt.launched("attention")
            return out
        ops.decode_attention(q.buf[0], cache.packed if cache.dtype in BFP else cache.buf, base.buf.reshape(-1), last.buf.reshape(-1), heads, kv, hd,
                             max_keys=min(length or cache.rows, cache.rows),
                             window=window or 0, out=out.buf[0])
        self.rt.launched("attention")
        return out

    # ---------------------------------------------------------------- latent attention and decaying linear attention

    def latent_heads_put(self, rotation, places, rows, cache, heads, dim, turned, kv_norm, eps):
        """self: a joint projection [1, tokens, queries (heads x (dim | rot)) | key-value latent | shared key part].  As latent_put for a
        design without a query latent: the queries' first parts come back side by side, as the cache is stored, the others go,
        turned, into `turned` (a view [heads, tokens, rot])."""
        x, places, rows = self.realize(), places.realize(), rows.realize()
        rank = kv_norm.cols
        rot = cache.cols - rank
        assert x.batch == 1 and x.buf.stride(2) == 1 and x.cols >= heads * (dim + rot) + cache.cols and cache.buf.is_contiguous(), f"{self.shape} into a cache {cache.shape}"
        assert turned.shape == (heads, x.rows, rot) and turned.dtype == cache.dtype and turned.buf.stride(2) == 1 and kv_norm.dtype == "fp32" and places.cols == rows.cols == x.rows
        freq, dims, mag = rotation
        out = Tensor(self.rt, x.rows, heads * dim, dtype=cache.dtype)
        ops.latent_put(x.buf[0], 0, rank, rot, dims, None, kv_norm.buf, eps, freq, mag, places.buf.reshape(-1), rows.buf.reshape(-1), cache.buf[0], out.buf[0], heads, dim, turned.buf)
        self.rt.launched("latent put")
        return out

    def latent_put(self, rotation, places, rows, cache, q_rank, q_norm, kv_norm, eps):
        """self: a joint down-projection [1, tokens, query latent | key-value latent | shared key part | ...].  One kernel norms
        both latents, turns the key part and puts (key-value latent | key part) into `cache` ([1, size, kv_rank + rot]) at
        `rows`; returns the normed query latent, as the cache is stored.  rotation: (frequencies on the device, their
        number of columns, factor) of mixers.rotation; places, rows: int32 rows read on the device."""
        x, places, rows = self.realize(), places.realize(), rows.realize()
        kv_rank = kv_norm.cols
        rot = cache.cols - kv_rank
        assert x.batch == 1 and x.buf.stride(2) == 1 and x.cols >= q_rank + cache.cols and cache.buf.is_contiguous(), f"{self.shape} into a cache {cache.shape}"
        assert q_norm is None or (q_norm.cols == q_rank and q_norm.dtype == "fp32") and kv_norm.dtype == "fp32" and places.cols == rows.cols == x.rows
        freq, dims, mag = rotation
        out = Tensor(self.rt, x.rows, q_rank, dtype=cache.dtype) if q_rank else None
        ops.latent_put(x.buf[0], q_rank, kv_rank, rot, dims, None if q_norm is None else q_norm.buf, kv_norm.buf, eps, freq, mag, places.buf.reshape(-1),
                       rows.buf.reshape(-1), cache.buf[0], None if out is None else out.buf[0])
        self.rt.launched("latent put")
        return out

    def rotate_pairs(self, rotation, places, into=None):
        """self: [heads, tokens, width], each head's first columns turned pair by pair by its token's angle (the rest as they
        are), into `into` (a view of the same shape) or a tensor of its own."""
        x, places = self.realize(), places.realize()
        into = into if into is not None else Tensor(self.rt, x.rows, x.cols, batch=x.batch, dtype=x.dtype)
        assert into.shape == x.shape and into.dtype == x.dtype and x.buf.stride(2) == into.buf.stride(2) == 1 and places.cols == x.rows
        ops.rotate_pairs(x.buf, rotation, places.buf.reshape(-1), into.buf)
        self.rt.launched("rotate pairs")
        return into

    def attend_latent(self, cache, base, last, rank, scale, sink=None, length=None, chunk=False, window=0):
        """self: [1, tokens, heads (rank + rot)], each head's query in the latents' space and its turned part.  Token t attends
        the cache rows base[t] .. base[t] + last[t] (the last `window` of them, if any): one row is key (all of it) and value (its
        first `rank` columns) of every head.  sink: a number per head that joins the softmax's denominator.  chunk: the tokens are one sequence's, its first
        cache row 0.  Returns [1, tokens, heads rank]: weighted sums of latents."""
        q, last = self.realize(), last.realize()
        heads = q.cols // cache.cols
        assert q.batch == cache.batch == 1 and q.cols % cache.cols == 0 and q.dtype == cache.dtype and q.buf.stride(2) == 1, f"{q.shape} over a cache {cache.shape}"
        out = Tensor(self.rt, q.rows, heads * rank, dtype=q.dtype)
        ops.latent_attention(q.buf[0], cache.buf[0], None if chunk else base.realize().buf.reshape(-1), last.buf.reshape(-1), heads, rank, scale,
                             None if sink is None else sink.buf, min(length or cache.rows, cache.rows), chunk, out=out.buf[0], window=window)
        self.rt.launched("latent attention")
        return out

    def decay_scan(self, heads, dim, vdim, decay, places, state, dead=-1):
        """self: rows of q | k | v (| more) of one sequence, or one row of each of state.batch sequences; state: fp32 [sequences,
        heads dim, vdim], read and written.  S = decay S + k v^T, o = S^T q per head; a sequence at place 0 starts from
        zeros, one at place `dead` is left alone.  Returns fp32 [1, tokens, heads vdim]."""
        x, places = self.realize(), places.realize()
        assert x.batch == 1 and x.buf.stride(2) == 1 and state.dtype == "fp32" and state.shape[1:] == (heads * dim, vdim) and x.rows % state.batch == 0
        out = Tensor(self.rt, x.rows, heads * vdim, dtype="fp32")
        ops.decay_scan(x.buf[0], heads, dim, vdim, decay.buf, places.buf.reshape(-1), dead, state.buf, out.buf[0])
        self.rt.launched("decay scan")
        return out

    def selective_scan(self, heads, groups, dim, vdim, step, step_bias, a_log, skip, places, state, dead=-1):
        """self: rows of values (heads x vdim) | keys (groups x dim) | queries (groups x dim), as decay_scan's sequences; step: fp32, a number a row and
        head.  With d = softplus(step + step_bias): S = exp(-exp(a_log) d) S + d k v^T, o = S^T q + skip v per head.  Returns fp32 [1, tokens, heads vdim]."""
        x, step, places = self.realize(), step.realize(), places.realize()
        assert x.batch == 1 and x.buf.stride(2) == 1 and state.dtype == "fp32" and state.shape[1:] == (heads * dim, vdim) and x.rows % state.batch == 0
        assert step.dtype == "fp32" and step.shape == (1, x.rows, heads) and all(t.dtype == "fp32" and t.cols == heads for t in (step_bias, a_log, skip))
        out = Tensor(self.rt, x.rows, heads * vdim, dtype="fp32")
        ops.selective_scan(x.buf[0], heads, groups, dim, vdim, step.buf[0], step_bias.buf, a_log.buf, skip.buf, places.buf.reshape(-1), dead, state.buf, out.buf[0])
        self.rt.launched("selective scan")
        return out

    def short_conv(self, w, places, state, dead=-1, bias=None, in_bias=None, silu=False, dtype="bf16"):
        """self: rows of one sequence, or one row of each of state.batch sequences.  A causal convolution over time of every column by w ([taps,
        columns], fp32; in_bias joins before it, bias after), then SiLU; state ([sequences, >= taps - 1, columns], fp32, read and written): the inputs
        of earlier tokens - zeros at place 0; a sequence at place `dead` leaves it alone."""
        x, places = self.realize(), places.realize()
        assert x.batch == 1 and x.buf.stride(2) == 1 and all(t is None or (t.dtype == "fp32" and t.cols == x.cols) for t in (w, bias, in_bias, state)) and x.rows % state.batch == 0
        out = Tensor(self.rt, x.rows, x.cols, dtype=dtype)
        buf = lambda t: None if t is None else t.buf
        ops.short_conv(x.buf[0], w.buf[0], out.buf[0], places.buf.reshape(-1), dead, state.buf, buf(bias), buf(in_bias), silu)
        self.rt.launched("short conv")
        return out

    def lru_scan(self, gates, y, lam, rate, blocks, places, state, dead=-1, gate_bias=None, y_bias=None, scale=1.0, into=None):
        """self: rows as short_conv's; gates: fp32, a block's r columns and then its i columns, block after block.  With r and i their sigmoids and
        log a = rate r softplus(lam): S = a S + sqrt(1 - a^2) i self per column, and the result is scale S gelu(y); state: fp32 [sequences, 1, columns]."""
        x, gates, y, places = self.realize(), gates.realize(), y.realize(), places.realize()
        out = into if into is not None else Tensor(self.rt, x.rows, x.cols, dtype=x.dtype)
        assert x.batch == 1 and x.buf.stride(2) == gates.buf.stride(2) == y.buf.stride(2) == out.buf.stride(2) == 1 and y.shape == x.shape == out.shape and gates.shape == (1, x.rows, 2 * x.cols)
        assert all(t is None or t.dtype == "fp32" for t in (lam, gate_bias, y_bias, state)) and (gate_bias is None or gate_bias.buf.is_contiguous()) and x.rows % state.batch == 0
        buf = lambda t: None if t is None else t.buf
        ops.lru_scan(x.buf[0], gates.buf[0], y.buf[0], out.buf[0], lam.buf, rate, blocks, places.buf.reshape(-1), dead, state.buf, buf(gate_bias), buf(y_bias), scale)
        self.rt.launched("lru scan")
        return out

    def gated_rms(self, gate, w, eps, before=False, parts=1, dtype=None):
        """RMSNorm of self (fp32 rows), each of its equal parts by its own root mean square, by w, times the sigmoid of gate; before: self times the
        SiLU of gate is what is normed.  As gate is stored, or as dtype."""
        x, gate = self.realize(), gate.realize()
        out = Tensor(self.rt, x.rows, x.cols, dtype=dtype or gate.dtype)
        ops.gated_rmsnorm(x.buf[0], gate.buf[0], w.buf, eps, out.buf[0], before, parts)
        self.rt.launched("gated rmsnorm")
        return out

    # ---------------------------------------------------------------- an fp32 residual stream with grouped-query heads and experts

    def embed(self, ids, places_table=None, places=None, scale=1.0):
        """Rows ids of this table times scale, plus rows `places` of another where given, as an fp32 matrix: a residual stream's start."""
        ids, places = ids.realize(), None if places is None else places.realize()
        out = Tensor(self.rt, ids.cols, self.cols, dtype="fp32")
        assert places_table is None or (places_table.cols == self.cols and places_table.dtype == self.dtype and places.cols == ids.cols)
        ops.embed(self.realize().buf[0], ids.buf.reshape(-1), None if places_table is None else places_table.realize().buf[0], None if places is None else places.buf.reshape(-1), out.buf[0], scale)
        self.rt.launched("embed")
        return out

    def heads_put(self, heads, dim, vdim, rows, cache, bias=None, q_norm=None, k_norm=None, eps=0.0, mix=None, norm_all=False,
                  keys_are_values=False, rotation=None, places=None, conv=None, state=None, dead=-1, temperature=None):
        """self: a joint projection [1, tokens, q (heads x dim) | k | v (| more)]; its keys and values go into `cache` ([key
        heads, size, dim + vdim]) at `rows`, its queries come back, as the cache is stored.  bias: a number a column of q | k | v;
        q_norm, k_norm: RMSNorm of each head (norm_all: of all of them together); mix: (other values of the tokens, their bias or
        None, share): the values become (1 - share) own + share other; keys_are_values: there is no v, the keys as projected are the
        values; rotation: mixers.rotation's, by `places`; conv ([taps, columns]): a short convolution over time of every column, state
        ([sequences, taps - 1, columns], fp32, read and written) what it needs of earlier tokens - nothing at place 0, and a sequence
        at place `dead` leaves it alone; temperature: (coef, every): queries, after their norm, times 1 + coef ln(floor((place + 1) / every) + 1)."""
        x, rows = self.realize(), rows.realize()
        wide = (heads + cache.batch) * dim + (0 if keys_are_values else cache.batch * vdim)
        assert x.batch == 1 and x.buf.stride(2) == 1 and rows.cols == x.rows and x.cols >= wide, f"{self.shape} into a cache {cache.shape}"
        assert all(t is None or t.dtype == "fp32" for t in (bias, q_norm, k_norm, conv, state)) and all(t is None or t.cols == wide for t in (bias, conv, state))
        assert q_norm is None or (q_norm.cols, k_norm.cols) == ((heads * dim, cache.batch * dim) if norm_all else (dim, dim))
        buf = lambda t: None if t is None else t.realize().buf
        first, first_bias, share = mix or (None, None, None)
        assert first is None or (first.dtype == x.dtype and first.shape == (1, x.rows, cache.batch * vdim) and first.buf.stride(2) == 1), "the other layer's values, a column each of this one's"
        out = Tensor(self.rt, x.rows, heads * dim, dtype=cache.dtype)
        ops.heads_put(x.buf[0], heads, cache.batch, dim, vdim, rows.buf.reshape(-1), cache.buf, out.buf[0], buf(bias), buf(q_norm), buf(k_norm), eps,
                      None if first is None else first.buf[0], buf(first_bias), buf(share), norm_all, keys_are_values, rotation, None if places is None else places.realize().buf.reshape(-1),
                      None if conv is None else conv.realize().buf[0], buf(state), dead, temperature or (0.0, 1.0))
        self.rt.launched("heads put")
        return out

    def attend_heads(self, cache, base, last, vdim, scale, length=None, span=0, sink=None, gate=None, chunk=False, window=0, softcap=0.0, key_bias=None,
                     out_scale=1.0, into=None):
        """self: [1, tokens, heads x dim] over such a cache.  Token t, which stands at place last[t], attends the rows from base[t]
        on up to its own; with span, only those of its own span of that many places, with window, only the last so many.  softcap: c
        > 0 makes a scaled score s c tanh(s / c).  sink: a number per head that joins the
        softmax's denominator; key_bias: a number per head, no softmax: a key's weight is the sigmoid of its score and that; gate: the result is multiplied by
        its sigmoid, column by column; chunk: one sequence's tokens, its first cache row 0.  Returns [1, tokens, heads x vdim] times out_scale (into: there)."""
        q, last = self.realize(), last.realize()
        dim = cache.cols - vdim
        assert q.batch == 1 and q.cols % dim == 0 and q.dtype == cache.dtype and (q.cols // dim) % cache.batch == 0, f"{q.shape} over a cache {cache.shape}"
        heads = q.cols // dim
        out = into if into is not None else Tensor(self.rt, q.rows, heads * vdim, dtype=q.dtype)
        assert (gate is None or gate.shape == out.shape) and out.shape == (1, q.rows, heads * vdim) and out.dtype == q.dtype and out.buf.stride(2) == 1
        ops.heads_attention(q.buf[0], cache.buf, None if chunk else base.realize().buf.reshape(-1), last.buf.reshape(-1), heads, vdim, scale, min(length or cache.rows, cache.rows), chunk, span,
                            None if sink is None else sink.realize().buf, None if gate is None else gate.realize().buf[0], out=out.buf[0], window=window, softcap=softcap,
                            key_bias=None if key_bias is None else key_bias.realize().buf, out_scale=out_scale)
        self.rt.launched("attention")
        return out

    def route(self, n, k, bias=None, scored=False, identity=0, scale=1.0, as_scored=False, on_input=False):
        """self: fp32 router logits, n a token: each token's k experts, their weights and where their rows go (ops.Routes).  scored ("softmax",
        "sigmoid"): chosen by score + bias, weighted by the scores, over their sum unless as_scored; identity: the last so many give back their input; scale: of
        the weights; on_input: they go on the experts' inputs."""
        x = self.realize()
        assert x.dtype == "fp32" and x.batch == 1 and x.cols == n and x.buf.stride(2) == 1 and (bias is None or (bias.dtype == "fp32" and bias.cols == n))
        self.rt.launched("route")
        return ops.route(x.buf[0], n, k, None if bias is None else bias.realize().buf, scored, identity, scale, as_scored, on_input)

    def experts(self, routes, gate_up, down, clamp=None, relu2=False):
        """self: rows of tokens.  Every chosen expert's down(silu(gate) * up) of its tokens' rows, a row a choice where `routes`
        puts it; gate and up side by side in gate_up [n, K, 2 m], down [n, m, N].  clamp: (limit, slope) of clamped_glu in the
        unit's place; relu2: max(up, 0)^2, and gate_up [n, K, m] is up alone.  A weight on an input scales the products of its row before the unit."""
        rt, h, m = self.rt, self.realize(), down.rows
        assert h.batch == 1 and gate_up.cols == (m if relu2 else 2 * m) and gate_up.batch == down.batch == routes.n and h.rows == routes.T
        if not routes.shared:
            x = Tensor(rt, routes.tiles * routes.tile, h.cols, dtype=h.dtype)
            ops.spread_rows(h.buf[0], routes, x.buf[0])
            rt.launched("spread rows")
            h = x
        act = Tensor(rt, routes.tiles * routes.tile, m, dtype=h.dtype)
        out = Tensor(rt, routes.tiles * routes.tile, down.cols, dtype=h.dtype)
        weights = routes.row_weights
        unit = dict(kind=_lib.DENSE_RELU2) if relu2 else dict(kind=_lib.DENSE_GLU, limit=clamp[0], slope=clamp[1]) if clamp else dict(kind=_lib.DENSE_SWIGLU)
        if ops.grouped(h.buf[0], gate_up.buf, routes, act.buf[0], shared=routes.shared, row_scale=None if weights is None else weights.data_ptr(), **unit):
            rt.launched("experts relu2" if relu2 else "experts glu" if clamp else "experts swiglu")
        else:
            both = Tensor(rt, act.rows, gate_up.cols, dtype="fp32")
            ops.grouped_matmul(h.buf[0], gate_up.buf, routes, both.buf[0], routes.shared, weights)
            rt.launched("experts matmul")
            if relu2:
                up = both.relu()
                (up * up).cast(h.dtype).realize(into=act)
            else:
                gate, up = both[:, :m], both[:, m:]
                (clamped_glu(gate, up, *clamp) if clamp else gate.silu() * up).cast(h.dtype).realize(into=act)
        if ops.grouped(act.buf[0], down.buf, routes, out.buf[0]):
            rt.launched("experts")
        else:
            ops.grouped_matmul(act.buf[0], down.buf, routes, out.buf[0])
            rt.launched("experts matmul")
        return out

    def add_norm(self, w, eps, plus=0.0, dtype="bf16", mixer=None, mixer_scale=None, other=None, other_scale=None, experts=None,
                 mixer_bias=None, own=None, into=None, gate=None, gate_bias=None, post=None):
        """self: an fp32 residual stream.  (self + (mixer + mixer_bias) * mixer_scale + (other + the experts' rows by their weights) *
        other_scale, and that as RMSNorm by w + plus leaves it, or, w None, as it is); experts: (rows, routes), own: the row that an
        identity expert gives back.  gate (fp32, with gate_bias): the branches' sum is multiplied by its sigmoid, and post: goes through RMSNorm by it, before it joins
        the stream.  Without branches: (self, its norm).  into: where the second goes."""
        x = self.realize()
        get = lambda t: None if t is None else t.realize().buf[0]
        assert x.dtype == "fp32" and x.batch == 1 and all(t is None or (t.shape == x.shape and t.buf.stride(2) == 1) for t in (mixer and mixer.realize(), other and other.realize(), gate and gate.realize()))
        assert gate is None or gate.dtype == "fp32"
        bare = mixer is other is experts is mixer_bias is None
        out, h = x if bare else Tensor(self.rt, x.rows, x.cols, dtype="fp32"), into if into is not None else Tensor(self.rt, x.rows, x.cols, dtype=dtype)
        assert h.shape == x.shape and h.dtype == dtype and h.buf.stride(2) == 1
        scale = lambda t: None if t is None else t.realize().buf
        rows, routes = experts or (None, None)
        ops.add_norm(x.buf[0], None if bare else out.buf[0], get(mixer), scale(mixer_scale), get(other), scale(other_scale), get(rows), routes, scale(w), plus, eps, h.buf[0], scale(mixer_bias), get(own),
                     get(gate), scale(gate_bias), scale(post))
        self.rt.launched("norm" if bare else "add norm")
        return out, h

    def greedy(self, values=None):
        """Each row's first largest logit's column, int32 [1, 1, rows], picked on the device (the reference reads the
        logits back and takes numpy's argmax, models/llama.py:787-795): fp32 logits of one matrix."""
        x = self.realize()
        assert x.dtype == "fp32" and x.batch == 1 and x.buf.stride(2) == 1, "a matrix of fp32 logits"
        out = Tensor(self.rt, 1, x.rows, dtype="int32")
        ops.argmax(x.buf[0], out.buf.reshape(-1), None if values is None else values.buf.reshape(-1))
        self.rt.launched("argmax")
        return out

    # ---------------------------------------------------------------- computing the tree

    def realize(self, into=None):
        """Compute it now, into storage of its own or into `into`'s (ferrite/tensor.py:247-272).  Returns it, realized."""
        if self.op is None:
            if into is not None:
                _copy(self, into)
            return self
        _realize(self, into)
        return self


def clamped_glu(gate, up, limit, slope):
    """g sigmoid(slope g) (u + 1) with the gate's half cut at limit and the other within -limit .. limit."""
    g, u = gate.minimum(limit), up.maximum(-limit).minimum(limit)
    return g * (g * slope).sigmoid() * (u + 1)


# -------------------------------------------------------------------- the planner

def _done(t, buf=None, packed=None):
    """t is computed: it now owns storage and forgets how it was made."""
    t.buf, t.packed, t.op, t.srcs = buf, packed, None, ()


def _realize(t, into=None):
    op = t.op
    if op in _ELEMENTWISE:
        if op == "cast" and t.dtype in BFP:
            src = t.srcs[0].cast("bf16").realize()
            buf = src.buf if src.buf.is_contiguous() else (src + 0).realize().buf
            _done(t, packed=ops.quantize(buf if t.batch > 1 else buf[0], t.dtype))
            t.rt.launched("cast " + t.dtype)
            return
        if op == "cast" and t.srcs[0].dtype in BFP:
            src = t.srcs[0].realize()
            bf = Tensor(t.rt, t.rows, t.cols, batch=t.batch, buf=ops.dequantize(src.packed))
            _done(t, buf=bf.buf if t.dtype == "bf16" else bf.cast(t.dtype).realize().buf)
            return
        if _fused_linear(t, into) or _fused_dense(t, into):
            return
        if _run_rmsnorm(t, into):
            return
        found = _match_dyt(t)
        if found:  # (what it stands on is read by others too - the residual stream: computed once, not inside this expression)
            found[0].realize()
        _run_elementwise(t, into)
    elif op == "reduce_sum" and t.args["axis"] == 0 and _match_experts(t.srcs[0]):
        _run_experts(t, _match_experts(t.srcs[0]), None, into)
    elif op in ("reduce_sum", "reduce_max"):
        src, axis = t.srcs[0].realize(), t.args["axis"]
        out = into or Tensor(t.rt, t.rows, t.cols, batch=t.batch, dtype=t.dtype)
        i64 = lambda v: (ctypes_i64 * 3)(*v)
        check(lib().fb_reduce(int(op == "reduce_max"), src.buf.data_ptr(), i64(_strides3(src.buf)), _lib.DTYPES[src.dtype], *src.shape, axis,
                              out.buf.data_ptr(), i64(_strides3(out.buf)), _lib.DTYPES[out.dtype], ops._stream()))
        t.rt.launched(f"{op}{axis}", 1)
        _done(t, buf=out.buf)
    elif op == "matmul":
        _run_matmul(t, into)
    elif op == "cols":  # a run of columns of a matmul, read on its own: the whole matmul, then a view
        mm = t.srcs[0].realize()
        start = t.args["start"]
        _done(t, buf=mm.buf[:, :, start:start + t.cols])
        t.owner = mm
        if into is not None:
            _copy(t, into)
    elif op == "silu_columns":
        if _dense(t, t.srcs[0], into, _lib.DENSE_SILU, act_cols=t.args["n"]):
            return
        src = t.srcs[0].realize()
        out = (src + 0).realize()
        part = out[:, :, :t.args["n"]]
        part.assign(part.silu())
        _done(t, buf=out.buf)
    elif op == "gelu_gated":
        mm, m = t.srcs[0], t.cols
        bias = t.srcs[1].realize() if len(t.srcs) > 1 else None
        half = lambda x, i: x[:, :, i * m:(i + 1) * m]
        if mm.batch == 1 and _dense(t, mm, into, _lib.DENSE_GEGLU, gate_bias=bias and half(bias, 0), up_bias=bias and half(bias, 1)):
            return
        mm = mm.realize()
        gate, up = (half(mm, i) + half(bias, i) if bias is not None else half(mm, i) for i in (0, 1))
        out = (gate.gelu() * up).cast(t.dtype).realize(into=into)
        return _done(t, buf=out.buf)
    elif op == "repeat":
        src, n = t.srcs[0].realize(), t.args["n"]
        out = Tensor(t.rt, t.rows, t.cols, batch=t.batch, dtype=t.dtype)
        for b in range(src.batch):
            _copy(src._view(src.buf[b:b + 1].expand(n, src.rows, src.cols)), out._view(out.buf[b * n:(b + 1) * n]))
        _done(t, buf=out.buf)
    else:
        raise NotImplementedError(f"no kernel for {op}")
    if into is not None and t.buf is not into.buf and op not in ("cols",):
        _copy(t, into)


import ctypes  # noqa: E402

ctypes_i64 = ctypes.c_int64


def _is_const(x, value=None):
    return isinstance(x, (int, float)) and (value is None or x == value)


def _match_rms(t):
    """(x, w, eps) if t is x * rsqrt(mean(x * x) + eps) * w as models/llama.py:82-85 writes RMSNorm, else None."""
    if not isinstance(t, Tensor) or t.op != "mul":
        return None
    for n, w in (t.srcs, t.srcs[::-1]):
        if not (isinstance(w, Tensor) and w.op is None and w.shape == (1, 1, t.cols) and isinstance(n, Tensor) and n.op == "mul"):
            continue
        for x, r in (n.srcs, n.srcs[::-1]):
            if not (isinstance(r, Tensor) and r.op == "recip" and isinstance(x, Tensor)):
                continue
            root = r.srcs[0]
            if root.op != "sqrt" or root.srcs[0].op != "add":
                continue
            mean, eps = root.srcs[0].srcs
            if not (_is_const(eps) and isinstance(mean, Tensor) and mean.op == "mul" and _is_const(mean.srcs[1])):
                continue
            total = mean.srcs[0]
            if not (isinstance(total, Tensor) and total.op == "reduce_sum" and total.args["axis"] == 2 and abs(mean.srcs[1] * x.cols - 1) < 1e-6):
                continue
            sq = total.srcs[0]
            if sq.op == "mul" and sq.srcs[0] is x and sq.srcs[1] is x:
                return x, w, float(eps)
    return None


def _run_rmsnorm(t, into):
    """t as one fb_rmsnorm call where its tree is an RMSNorm of bf16 rows that no matmul takes in as its prologue (a
    mixture's router and experts both read the normed rows; the output layer of a single sequence reads its last)."""
    found = _match_rms(t) if t.dtype == "bf16" and t.batch == 1 else None
    if not found or found[0].dtype != "bf16" or found[0].shape != t.shape:
        return False
    x, w, eps = found
    x = x.realize()
    if x.buf.stride(2) != 1 or (into is not None and into.buf.stride(2) != 1):
        return False
    out = into if into is not None else Tensor(t.rt, t.rows, t.cols)
    ops.rmsnorm(x.buf[0], w.realize().buf.reshape(-1), eps, out=out.buf[0])
    t.rt.launched("rmsnorm")
    _done(t, buf=out.buf)
    return True


def _match_dyt(t):
    """(x, alpha, w, b) if t is tanh(alpha x) w + b as mixers.dyt writes it, or a cast of it, else None."""
    if isinstance(t, Tensor) and t.op == "cast":
        t = t.srcs[0]
    if not (isinstance(t, Tensor) and t.op == "add" and isinstance(t.srcs[0], Tensor) and t.srcs[0].op == "mul"):
        return None
    (th, w), b = t.srcs[0].srcs, t.srcs[1]
    vector = lambda v: isinstance(v, Tensor) and v.op is None and v.dtype == "fp32" and v.shape == (1, 1, t.cols)
    if not (isinstance(th, Tensor) and th.op == "tanh" and th.srcs[0].op == "mul" and vector(w) and vector(b)):
        return None
    x, alpha = th.srcs[0].srcs
    return (x, alpha, w, b) if isinstance(alpha, Tensor) and alpha.op is None and alpha.dtype == "fp32" and alpha.shape == (1, 1, 1) else None


def _match_clamped_glu(t):
    """(matmul, limit, slope) if t is clamped_glu over the halves of one matmul not yet computed, else None."""
    if not (t.op == "mul" and all(isinstance(s, Tensor) for s in t.srcs)):
        return None
    act, plus = t.srcs
    if not (act.op == "mul" and isinstance(act.srcs[1], Tensor) and act.srcs[1].op == "recip" and plus.op == "add" and _is_const(plus.srcs[1], 1)):
        return None
    g, u = act.srcs[0], plus.srcs[0]
    one = act.srcs[1].srcs[0]
    if not (one.op == "add" and _is_const(one.srcs[1], 1) and one.srcs[0].op == "exp"):
        return None
    neg = one.srcs[0].srcs[0]
    if not (neg.op == "mul" and _is_const(neg.srcs[1], -1) and neg.srcs[0].op == "mul" and neg.srcs[0].srcs[0] is g and _is_const(neg.srcs[0].srcs[1])):
        return None
    if not (isinstance(u, Tensor) and g.op == "min" and u.op == "min" and isinstance(u.srcs[0], Tensor) and u.srcs[0].op == "max"):
        return None
    limit, gate, up = g.srcs[1], g.srcs[0], u.srcs[0].srcs[0]
    if not (_is_const(limit) and _is_const(u.srcs[1], limit) and _is_const(u.srcs[0].srcs[1], -limit) and gate.op == up.op == "cols" and gate.srcs[0] is up.srcs[0]):
        return None
    mm = gate.srcs[0]
    if gate.args["start"] != 0 or up.args["start"] != gate.cols or 2 * gate.cols != mm.cols:
        return None
    return mm, float(limit), float(neg.srcs[0].srcs[1])


def _match_swiglu(t):
    """The matmul if t is silu(mm[:, :m]) * mm[:, m:] over the halves of one matmul not yet computed, else None."""
    for g, u in (t.srcs, t.srcs[::-1]):
        gate = _match_silu_of(g)
        if gate is not None and isinstance(u, Tensor) and gate.op == u.op == "cols" and gate.srcs[0] is u.srcs[0]:
            mm = gate.srcs[0]
            if gate.args["start"] == 0 and u.args["start"] == gate.cols and 2 * gate.cols == mm.cols and mm.batch == 1:
                return mm
    return None


def _match_gated(t):
    """(matmul, gate) if t is matmul * gate.sigmoid(), a number a row of each of the matmul's batch, else None."""
    if t.op != "mul" or not all(isinstance(s, Tensor) for s in t.srcs):
        return None
    mm, s = t.srcs
    if mm.op != "matmul" or s.op != "recip" or s.srcs[0].op != "add" or not _is_const(s.srcs[0].srcs[1], 1) or s.srcs[0].srcs[0].op != "exp":
        return None
    neg = s.srcs[0].srcs[0].srcs[0]
    if not (neg.op == "mul" and _is_const(neg.srcs[1], -1) and isinstance(neg.srcs[0], Tensor) and neg.srcs[0].op is None):
        return None
    gate = neg.srcs[0]
    return (mm, gate) if gate.dtype == "fp32" and gate.shape == (mm.batch, mm.rows, 1) and (mm.batch == 1 or gate.buf.stride(0) == 1) else None


def _dense(t, mm, into, kind, **extra):
    """t by fb_dense where mm is a matmul, not yet computed, by bf16 weights whose columns each lie together (a turned matrix as
    a checkpoint stores it), with an epilogue; else False.  extra: the epilogue's fields, tensors by name."""
    if mm.op != "matmul" or len(mm.srcs) != 2:
        return False
    a, w = mm.srcs
    if not (a.dtype == "bf16" and w.dtype == "bf16" and w.op is None and a.batch == w.batch and w.buf.stride(1) == 1 and w.rows % 8 == 0 and w.buf.stride(2) % 8 == 0):
        return False
    if kind in (_lib.DENSE_GLU, _lib.DENSE_SWIGLU, _lib.DENSE_GEGLU) and w.cols % 32:
        return False
    x = a.realize()
    if not ops.dense_supports(x.buf, w.buf, kind):
        x = (x + 0).realize()
        if not ops.dense_supports(x.buf, w.buf, kind):
            return False
    out = into if into is not None and into.buf.stride(2) == 1 and into.dtype == t.dtype else Tensor(t.rt, t.rows, t.cols, batch=t.batch, dtype=t.dtype)
    fields, keep = {}, []
    for name, v in extra.items():
        if isinstance(v, Tensor):
            v = v.realize()
            keep.append(v)
            fields[name] = v.buf.data_ptr()
            if name in ("residual", "gate", "h_out"):
                fields["ld_" + name.removesuffix("_out")] = v.buf.stride(1)
        elif v is not None:
            fields[name] = v
    ops.dense(x.buf, w.buf, out.buf, getattr(w, "settled", False), kind=kind, **fields)
    t.rt.launched("dense" + ("", " silu", " glu", " gate", " dyt add", " swiglu", " geglu")[kind])
    _done(t, buf=out.buf)
    if into is not None and out is not into:
        _copy(t, into)
    return True


def _fused_dense(t, into, hand_on=None):
    """t as one fb_dense call with an epilogue, where its tree is a gated unit, a gated output, or a branch's end - the Dynamic
    Tanh over a matmul, added to the residual stream; else False.  hand_on: the Dynamic Tanh (its tensors, and where its
    result goes) that the next branch starts with: the same kernel computes it."""
    inner = t.srcs[0] if t.op == "cast" and t.dtype == "bf16" else t
    if not isinstance(inner, Tensor) or inner.op is None:
        return False
    if inner.op == "mul" and t.dtype == "bf16":
        found = _match_clamped_glu(inner)
        if found:
            return _dense(t, found[0], into, _lib.DENSE_GLU, limit=found[1], slope=found[2])
        found = _match_gated(inner)
        if found:
            return _dense(t, found[0], into, _lib.DENSE_GATE, gate=found[1])
        found = _match_swiglu(inner)
        if found:
            return _dense(t, found, into, _lib.DENSE_SWIGLU)
    if t.op == "cast" and t.dtype == "bf16" and t.batch == 1:
        found = _match_dyt(inner)
        if found and found[0].op == "add" and found[0].dtype == "fp32":
            h = into if into is not None and into.buf.stride(2) == 1 else Tensor(t.rt, t.rows, t.cols)
            if _fused_dense(found[0], None, (h, *found[1:])):
                _done(t, buf=h.buf)
                if into is not None and h is not into:
                    _copy(t, into)
                return True
    if t.op == "add" and t.dtype == "fp32" and t.batch == 1:
        for x, y in (t.srcs, t.srcs[::-1]):
            found = _match_dyt(y) if isinstance(y, Tensor) and y.op == "add" else None
            if found and isinstance(x, Tensor) and x.dtype == "fp32" and x.shape == t.shape and found[0].op == "matmul" and found[0].dtype == "fp32":
                mm, alpha, w, b = found
                mm.srcs[0].realize()  # (it may stand on x itself: then x is computed by now, and not once more)
                x = x.realize()
                x = x if x.buf.stride(2) == 1 else (x + 0).realize()
                extra = dict(residual=x, alpha=alpha, w=w, b=b)
                if hand_on:
                    extra |= dict(h_out=hand_on[0], alpha2=hand_on[1], w2=hand_on[2], b2=hand_on[3])
                return _dense(t, mm, into, _lib.DENSE_DYT_ADD, **extra)
    return False


def _match_silu_of(g):
    """The tensor a if g is a * sigmoid(a) as Tensor.silu builds it, else None."""
    if not isinstance(g, Tensor) or g.op != "mul":
        return None
    for a, s in (g.srcs, g.srcs[::-1]):
        if not (isinstance(s, Tensor) and s.op == "recip" and isinstance(a, Tensor)):
            continue
        plus = s.srcs[0]
        if plus.op != "add":
            continue
        for e, one in (plus.srcs, plus.srcs[::-1]):
            if _is_const(one, 1) and isinstance(e, Tensor) and e.op == "exp":
                neg = e.srcs[0]
                if neg.op == "mul" and neg.srcs[0] is a and _is_const(neg.srcs[1], -1):
                    return a
    return None


def _packed_matmul(t):
    """(a, w) if t is a matmul, not yet computed, of one bf16 matrix by one block-float matrix, else None."""
    if isinstance(t, Tensor) and t.op == "matmul" and len(t.srcs) == 2 and t.srcs[1].dtype in BFP and t.srcs[1].batch == 1 and t.srcs[0].batch == 1 \
            and t.srcs[0].dtype == "bf16":
        return t.srcs
    return None


def _fused_linear(t, into, hand_on=None):
    """t as one fb_linear call with an epilogue, where its tree is a block's SwiGLU or residual add; else False.
    hand_on: the weight of the RMSNorm the result goes through next (see _linear): only a residual add takes it."""
    if t.op == "mul" and t.dtype == "bf16":  # silu(mm[:, :m]) * mm[:, m:]
        for g, u in (t.srcs, t.srcs[::-1]):
            gate = _match_silu_of(g)
            if gate is None or not isinstance(u, Tensor) or gate.op != "cols" or u.op != "cols":
                continue
            mm = gate.srcs[0]
            if u.srcs[0] is mm and _packed_matmul(mm) and mm.dtype == "bf16" and gate.args["start"] == 0 and u.args["start"] == gate.cols \
                    and 2 * gate.cols == mm.cols and mm.cols % 32 == 0:
                _linear(t, mm, "swiglu", None, into)
                return True
    if t.op == "add" and t.dtype == "bf16":  # x + the experts' sum
        for x, y in (t.srcs, t.srcs[::-1]):
            if isinstance(x, Tensor) and isinstance(y, Tensor) and y.op == "reduce_sum" and y.args["axis"] == 0 and x.shape == t.shape:
                found = _match_experts(y.srcs[0])
                if found:
                    _run_experts(t, found, x, into)
                    return True
    if t.op == "add" and t.dtype == "bf16":  # x + mm
        for x, mm in (t.srcs, t.srcs[::-1]):
            if isinstance(x, Tensor) and _packed_matmul(mm) and x.shape == mm.shape == t.shape and x.dtype == "bf16" and mm.dtype == "bf16":
                _linear(t, mm, "residual", x, into, hand_on)
                return True
    return False


def _linear(t, mm, epilogue, residual, into, hand_on=None):
    """fb_linear for the matmul mm (with its RMSNorm prologue, if its A is one) and the epilogue, into t.

    An RMSNorm between two block-float matmuls costs no kernel of its own where the first can hand it to the second
    (fb_linear_chained): when mm's A is rms(x) and x is a residual add of a block-float matmul not yet computed, that
    matmul is run with this norm's weight (hand_on) and leaves, beside x, x * g in bf16 and the rows' sums of squares;
    mm then reads those.  x is computed either way, for whoever else reads it (the next residual add)."""
    a, w = mm.srcs
    rms = _match_rms(a)
    x, norm_w, eps = rms if rms else (a, None, 0.0)
    w = w.realize()
    taken = None  # (x * g, sums of squares, parts) left by the matmul that made x
    # (9 rows and more: fewer go to the register-fed kernel, which takes no norm over)
    if CHAIN_NORMS and rms and x.op == "add" and x.dtype == "bf16" and x.batch == 1 and 9 <= x.rows <= 128:
        norm_w = norm_w.realize()
        if norm_w.buf.is_contiguous() and _fused_linear(x, None, hand_on=norm_w):
            taken = x.args.pop("handed", {}).get(id(norm_w))
    x = x.realize()
    res = None
    if residual is not None:
        residual = residual.realize()
        res = residual.buf[0] if residual.buf.stride(2) == 1 else (residual + 0).realize().buf[0]
    out = into if into is not None and into.buf.stride(2) == 1 else Tensor(t.rt, t.rows, t.cols, dtype=t.dtype)
    name = "linear " + w.dtype + (" rms" if rms else "") + ("" if epilogue == "none" else " " + epilogue)
    give = hand_on is not None and epilogue == "residual" and t.dtype == "bf16" and 9 <= t.rows <= 128 and ops.chain_parts(w.packed, t.rows, epilogue)
    if taken or give:
        xb = taken[0] if taken else (x.buf[0] if x.buf.stride(2) == 1 and x.buf.stride(1) % 8 == 0 else (x + 0).realize().buf[0])
        if rms and not taken:  # (a norm that nobody handed over: computed on its own, then the chained call reads plain rows)
            xb = ops.rmsnorm(xb, norm_w.buf.reshape(-1), eps)
        got = ops.linear_chained(xb, w.packed, out=out.buf[0], out_dtype=t.dtype, eps=eps, epilogue=epilogue, residual=res,
                                 norm_in=taken[1:] if taken else None, next_norm_w=hand_on.buf if give else None)
        if give:
            t.args = dict(t.args, handed={id(hand_on): (got[1], got[2], got[3])})
        t.rt.launched(name + " chained")
        _done(t, buf=out.buf)
        return
    xb = x.buf[0] if x.buf.stride(2) == 1 and x.buf.stride(1) % 8 == 0 else (x + 0).realize().buf[0]
    ops.linear(xb, w.packed, out=out.buf[0], out_dtype=t.dtype, norm_w=None if norm_w is None else norm_w.realize().buf, eps=eps, epilogue=epilogue, residual=res)
    t.rt.launched(name)
    _done(t, buf=out.buf)


def _run_matmul(t, into):
    if _packed_matmul(t):
        return _linear(t, t, "none", None, into)
    if len(t.srcs) == 3:
        return _run_indexed_matmul(t, into)
    if _dense(t, t, into, _lib.DENSE_NONE):
        return
    a, b = t.srcs[0].realize(), t.srcs[1]
    if b.dtype in BFP:  # a batch of block floats, or an fp32 A: by the values, through the general kernel
        b = b.cast("bf16")
    b = b.realize()
    out = into or Tensor(t.rt, t.rows, t.cols, batch=t.batch, dtype=t.dtype)
    i64 = lambda buf, batch: (ctypes_i64 * 3)(*([0] + _strides3(buf)[1:] if batch == 1 and t.batch > 1 else _strides3(buf)))
    check(lib().fb_matmul(a.buf.data_ptr(), i64(a.buf, a.batch), _lib.DTYPES[a.dtype], b.buf.data_ptr(), i64(b.buf, b.batch), _lib.DTYPES[b.dtype],
                          out.buf.data_ptr(), i64(out.buf, t.batch), _lib.DTYPES[out.dtype], t.batch, t.rows, t.cols, a.cols, ops._stream()))
    t.rt.launched("matmul", 1)
    _done(t, buf=out.buf)


def _indexed_packed(t):
    """(a, w, index) if t is a matmul, not yet computed, picking block-float matrices by an index, else None."""
    if isinstance(t, Tensor) and t.op == "matmul" and len(t.srcs) == 3 and t.srcs[1].dtype in BFP and t.srcs[0].dtype == "bf16":
        return t.srcs
    return None


def _match_experts(t):
    """A mixture's touched experts as models/llama.py:317-324 writes them for a decode step:
    (glu(x[:, :, :m], x[:, :, m:]) * weights).matmul(down, index=picks) with x = h.matmul(gate_up, index=picks).
    Returns (h, gate_up, down, picks, weights or None), else None."""
    found = _indexed_packed(t)
    if not found:
        return None
    a, down, picks = found
    weights = None
    if isinstance(a, Tensor) and a.op == "mul":
        for g, w in (a.srcs, a.srcs[::-1]):
            if isinstance(w, Tensor) and w.op is None and w.shape == (t.batch, t.rows, 1) and w.dtype == "bf16" and isinstance(g, Tensor) and g.op == "mul":
                a, weights = g, w
                break
    if not (isinstance(a, Tensor) and a.op == "mul"):
        return None
    for g, u in (a.srcs, a.srcs[::-1]):
        gate = _match_silu_of(g)
        if gate is None or not isinstance(u, Tensor) or gate.op != "cols" or u.op != "cols" or u.srcs[0] is not gate.srcs[0]:
            continue
        first = _indexed_packed(gate.srcs[0])
        if first and first[2] is picks and first[0].batch == 1 and gate.args["start"] == 0 and u.args["start"] == gate.cols \
                and 2 * gate.cols == first[1].cols and first[1].cols % 128 == 0 and gate.cols == down.rows and gate.cols % 64 == 0 and t.rows <= 128:
            return first[0], first[1], down, picks, weights
    return None


def _run_experts(t, found, residual, into):
    """Two kernels for a mixture's decode step: every touched expert's gate_up with SwiGLU and its tokens' weights into
    act [tokens, entries * m]; then the experts' downs summed over the entries in the accumulators (+ the residual)."""
    h, gate_up, down, picks, weights = found
    rms = _match_rms(h)
    x, norm_w, eps = rms if rms else (h, None, 0.0)
    x, picks = x.realize(), picks.realize()
    xb = x.buf[0] if x.buf.stride(2) == 1 and x.buf.stride(1) % 8 == 0 else (x + 0).realize().buf[0]
    slots, m, rows = picks.rows * picks.cols, down.rows, x.rows
    idx = picks.buf.reshape(-1) if picks.buf.is_contiguous() else (picks + 0).realize().buf.reshape(-1)
    act = Tensor(t.rt, rows, slots * m)
    scale = None
    if weights is not None:
        scale = weights.buf if weights.buf.is_contiguous() else (weights + 0).realize().buf
    ops.linear_indexed(xb, gate_up.realize().packed, idx, act.buf[0], out_slot_stride=m, norm_w=None if norm_w is None else norm_w.buf, eps=eps,
                       epilogue="swiglu", row_scale=scale)
    res = None
    if residual is not None:
        residual = residual.realize()
        res = residual.buf[0] if residual.buf.stride(2) == 1 else (residual + 0).realize().buf[0]
    out = into if into is not None and into.buf.stride(2) == 1 else Tensor(t.rt, t.rows, t.cols, dtype=t.dtype)
    ops.linear_indexed(act.buf[0], down.realize().packed, idx, out.buf[0], sum_slots=True, out_dtype=t.dtype,
                       epilogue="residual" if res is not None else "none", residual=res)
    t.rt.launched("experts " + gate_up.dtype)
    _done(t, buf=out.buf)


def _run_indexed_matmul(t, into):
    """Tensor.matmul(index=) on its own: one result per entry (ferrite/tensor.py:450-460); block-float matrices."""
    a, w, picks = t.srcs
    assert w.dtype in BFP and t.rows <= 128, "picked matrices are block floats here, for up to 128 rows"
    rms = _match_rms(a) if a.batch == 1 else None
    x, norm_w, eps = rms if rms else (a, None, 0.0)
    x, picks = x.realize(), picks.realize()
    if not (x.buf.is_contiguous() and x.cols % 8 == 0):
        x = (x + 0).realize()
    idx = picks.buf.reshape(-1) if picks.buf.is_contiguous() else (picks + 0).realize().buf.reshape(-1)
    out = into if into is not None and into.buf.is_contiguous() else Tensor(t.rt, t.rows, t.cols, batch=t.batch, dtype=t.dtype)
    ops.linear_indexed(x.buf.reshape(-1, x.cols), w.realize().packed, idx, out.buf, M=t.rows, x_slot_rows=0 if x.batch == 1 else t.rows,
                       out_slot_stride=t.rows * t.cols, out_dtype=t.dtype, norm_w=None if norm_w is None else norm_w.buf, eps=eps)
    t.rt.launched("matmul index " + w.dtype)
    _done(t, buf=out.buf)


def _program(t, inputs, code, consts, depth=1):
    """Append the postfix program of the elementwise tree under t; realized tensors become inputs."""
    if not isinstance(t, Tensor):
        code.append((1, 0)), consts.append(float(t))
        return depth
    if t.op not in _ELEMENTWISE or (t.op == "cast" and (t.dtype in BFP or t.srcs[0].dtype in BFP)) or len(code) > _MAX_OPS - 8 \
            or (len(inputs) >= _MAX_INPUTS - 1 and t.op is not None) or depth > _MAX_STACK - 2:
        leaf = t.realize()
        for i, u in enumerate(inputs):
            if u is leaf:
                break
        else:
            inputs.append(leaf)
            i = len(inputs) - 1
        code.append((0, i)), consts.append(0.0)
        return depth
    if t.op == "cast":
        most = _program(t.srcs[0], inputs, code, consts, depth)
        if t.dtype == "bf16":
            code.append((_UNARY["round_bf16"], 0)), consts.append(0.0)
        elif t.dtype == "int32":
            code.append((_UNARY["trunc"], 0)), consts.append(0.0)
        return most
    if t.op in _UNARY:
        most = _program(t.srcs[0], inputs, code, consts, depth)
        code.append((_UNARY[t.op], 0)), consts.append(0.0)
        return most
    most = max(_program(t.srcs[0], inputs, code, consts, depth), _program(t.srcs[1], inputs, code, consts, depth + 1))
    code.append((_BINARY[t.op], 0)), consts.append(0.0)
    return most


def _realize_leaves(t, seen):
    """Compute what the elementwise tree under t reads before the tree is looked at: a leaf's own inputs may be part of the
    tree as well (a residual stream under the branch that is added to it), and are then realized instead of inlined."""
    if not isinstance(t, Tensor) or t.op is None or id(t) in seen:
        return
    seen.add(id(t))
    if t.op not in _ELEMENTWISE:
        t.realize()
        return
    for src in reversed(t.srcs):
        _realize_leaves(src, seen)


def _run_elementwise(t, into=None):
    inputs, code, consts = [], [], []
    _realize_leaves(t, set())
    _program(t, inputs, code, consts)
    assert len(code) <= _MAX_OPS and len(inputs) <= _MAX_INPUTS, "an expression too large for one kernel even after splitting"
    out = into if into is not None else Tensor(t.rt, t.rows, t.cols, batch=t.batch, dtype=t.dtype)
    n = len(inputs)
    prog = (ctypes.c_int32 * (2 * len(code)))(*[v for pair in code for v in pair])
    cst = (ctypes.c_float * len(code))(*consts)
    ptrs = (ctypes.c_void_p * max(n, 1))(*[u.buf.data_ptr() for u in inputs])
    strides = (ctypes_i64 * (3 * max(n, 1)))(*[s for u in inputs for s in _strides3(u.buf.expand(t.shape))])
    dtypes = (ctypes.c_int32 * max(n, 1))(*[_lib.DTYPES[u.dtype] for u in inputs])
    check(lib().fb_elementwise(len(code), prog, cst, n, ptrs, strides, dtypes, out.buf.data_ptr(), (ctypes_i64 * 3)(*_strides3(out.buf)),
                               _lib.DTYPES[out.dtype], *t.shape, ops._stream()))
    t.rt.launched("elementwise", 1)
    _done(t, buf=out.buf)


def _copy(src, dst):
    """src's values into dst's storage (same shape; strides free), by the elementwise kernel."""
    assert src.shape == dst.shape, f"{src.shape} into {dst.shape}"
    _run_elementwise(src._lazy("add", (src, 0), src.shape, dst.dtype), into=dst)


def _fill(t, value):
    _run_elementwise(t._lazy("add", (value, 0), t.shape, t.dtype), into=t)


def jit(f):
    """f, a function of tensors that returns one, run from a recording (ferrite/tensor.py:788-810): its first call runs
    as any would, its second is recorded as a CUDA graph (the storage it takes kept from then on), and each later call
    copies its inputs into the second call's and replays the graph: nothing is planned, launched one by one or
    allocated again.  Its inputs keep their shapes and dtypes; it may not read back; its result is the same tensor
    every call, written again by the next."""
    state = {"calls": 0}

    def run(*xs):
        state["calls"] += 1
        if state["calls"] == 1:
            return f(*xs).realize()
        if state["calls"] == 2:
            inputs = [x.realize() for x in xs]
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            collects = gc.isenabled()
            gc.collect()
            gc.disable()  # (a recording that nobody holds any more may not be taken down while another is made)
            try:
                with torch.cuda.graph(graph, capture_error_mode="thread_local"):  # (other threads, NCCL's watchdog, may touch CUDA meanwhile)
                    out = f(*inputs).realize()
            finally:
                if collects:
                    gc.enable()
            graph.replay()
            state.update(inputs=inputs, graph=graph, out=out)
            return out
        for x, to in zip(xs, state["inputs"]):
            assert (x.shape, x.dtype) == (to.shape, to.dtype), f"{x.shape} {x.dtype} where the recording had {to.shape} {to.dtype}"
            if x is not to:
                to.buf.copy_(x.realize().buf, non_blocking=True)
        state["graph"].replay()
        return state["out"]

    return run
