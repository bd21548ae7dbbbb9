"""What the operator tests share: uploads that stay alive for a test, zeroed outputs, the storage types."""
import numpy as np

from safolorn_fixture import bf16_round

BF16, F32 = 30, 0
_ALIVE = []


def release():
    _ALIVE.clear()


def dev(G, a):
    _ALIVE.append(G.DeviceBuffer.from_numpy(np.ascontiguousarray(a)))
    return _ALIVE[-1]


def zeros(G, nbytes):
    b = G.DeviceBuffer(max(int(nbytes), 16))
    b.zero()
    _ALIVE.append(b)
    return b


def f32(a):
    return np.ascontiguousarray(a, dtype=np.float32)


def i32(a):
    return np.ascontiguousarray(a, dtype=np.int32)


def size_of(dt):
    return 2 if dt == BF16 else 4


def as_dt(dt, a):
    """(values as float64 after rounding into dt, the array to upload)"""
    if dt == BF16:
        return bf16_round(a)
    a32 = f32(a)
    return a32.astype(np.float64), a32


def from_dt(dt, buf, shape):
    n = int(np.prod(shape))
    if dt == BF16:
        return (buf.download(np.uint16, n).astype(np.uint32) << 16).view(np.float32).reshape(shape).astype(np.float64)
    return buf.download(np.float32, n).reshape(shape).astype(np.float64)


def ptr(b):
    return b.ptr if b is not None else None


def at(buf, byte_offset):
    return buf.ptr.value + byte_offset
