// Shared by the two extern "C" files (capi.cu, capi_bitnet.cu): no exception crosses them; failures become the
// reference's status codes and a message retrievable through tenzo_ext_last_error().
#pragma once
#include <new>
#include <stdexcept>
#include <string>

#include "engine_core.h"
#include "model_registry.h"

namespace tz {

template <typename F>
inline tenzo_status_t guarded(F&& f) {
    try {
        tz::g_last_error.clear();
        return f();
    } catch (const std::bad_alloc&) {
        tz::set_error("host allocation failed");
        return TENZO_ERROR_OUT_OF_MEMORY;
    } catch (const std::invalid_argument& e) {
        tz::set_error(e.what());
        return TENZO_ERROR_INVALID_ARGUMENT;
    } catch (const std::out_of_range& e) {
        tz::set_error(e.what());
        return TENZO_ERROR_INVALID_ARGUMENT;
    } catch (const IoError& e) {
        set_error(e.what());
        return TENZO_ERROR_IO;
    } catch (const ParseError& e) {
        set_error(e.what());
        return TENZO_ERROR_MODEL_PARSE;
    } catch (const std::exception& e) {
        tz::set_error(e.what());
        const std::string m = e.what();
        if (m.find("out of memory") != std::string::npos) return TENZO_ERROR_OUT_OF_MEMORY;
        return TENZO_ERROR_UNSUPPORTED;
    } catch (...) {
        tz::set_error("unknown failure");
        return TENZO_ERROR_UNSUPPORTED;
    }
}

inline bool live(tenzo_engine_t e) { return e && e->impl; }

}  // namespace tz
