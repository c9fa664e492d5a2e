// A small JSON reader for model configurations and weight-file headers (host only).
#pragma once
#include <map>
#include <stdexcept>
#include <string>
#include <vector>

namespace tz {

struct Json {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> items;
    std::map<std::string, Json> fields;

    bool is_null() const { return kind == Null; }
    bool has(const std::string& k) const { return kind == Object && fields.count(k); }
    const Json& at(const std::string& k) const {
        if (kind == Object) {
            auto it = fields.find(k);
            if (it != fields.end()) return it->second;
        }
        throw std::invalid_argument("missing key '" + k + "'");
    }
    double number() const {
        if (kind != Number) throw std::invalid_argument("a number was expected");
        return num;
    }
    int integer() const {
        const double v = number();
        if (v != (double)(long long)v || v < -2147483648.0 || v > 2147483647.0) throw std::invalid_argument("an integer was expected");
        return (int)v;
    }
    const std::string& string() const {
        if (kind != String) throw std::invalid_argument("a string was expected");
        return str;
    }
    const std::vector<Json>& array() const {
        if (kind != Array) throw std::invalid_argument("a list was expected");
        return items;
    }
};

Json parse_json(const std::string& text);          // throws std::invalid_argument with the byte position

}  // namespace tz
